"""The Netusun design in the layer-list family (sandwich blocks of RMS norms with layer scales; grouped-query attention behind short
convolutions with weighted per-head query / key norm, score cap, sliding window and a one in the softmax denominator; latent attention
with YaRN-scaled half-split rotation, a sink per head and an output gate; the mLSTM matrix memory; dense and routed feed-forwards with
expert groups and a shared expert; a layer loop whose passes open with a product over [stream; embedding]) against the plain float64
statement in oracle/netusun_oracle.py.  Every test mints its own small random checkpoint."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4


def rel(a, b):
    return float(np.abs(np.asarray(a, np.float64) - b).max() / max(np.abs(b).max(), 1e-30))


def close_bf16(a, b, noise):
    """bfloat16 matrices against the float64 oracle, row by row.  noise: what rounding the activations alone does to the rows of
    the same sequence (a router's close call or a norm over a few entries can turn it into large errors, hence the quantiles)."""
    e = np.abs(np.asarray(a, np.float64) - b).max(-1) / max(np.abs(b).max(), 1e-30)
    q = lambda v, p: float(np.quantile(v, p))
    return q(e, 0.5) < 2.0 * q(noise, 0.5) + 2e-3 and q(e, 0.9) < 2.0 * q(noise, 0.9) + 5e-3 and q(e, 1.0) < 4.0 * q(noise, 1.0) + 1e-2


@pytest.fixture(scope="module")
def no():
    import netusun_oracle
    return netusun_oracle


@pytest.fixture(scope="module")
def mk(tmp_path_factory, no):
    """mk(cfg, seed, quant, chunk, context, edit) -> (dsk.Model, weights): mints the checkpoint, loads it through Model.from_dir."""
    import dsk
    root = tmp_path_factory.mktemp("net")
    made, n = [], [0]

    def get(cfg, seed=0, quant="fp32", chunk=8, context=512, edit=None):
        W = no.random_weights(cfg, seed)
        if edit:
            edit(W)
            W = {k: no.bf16_to_f64(no.to_bf16(v)).reshape(v.shape) for k, v in W.items()}
        n[0] += 1
        d = no.write(str(root / f"m{n[0]}"), cfg, W)
        m = dsk.Model.from_dir(d, quant=quant, chunk=chunk, context=context)
        made.append(m)
        m.dir = d
        return m, W

    yield get
    for m in made:
        m.close()


def tokens_for(cfg, n, seed=0):
    return np.random.RandomState(seed).randint(0, cfg["vocab"], n).astype(np.int32)


def in_portions(m, toks, sizes, state=None):
    """The sequence in portions of the given sizes, the rest token by token; logits of every token."""
    p, rows = 0, []
    for c in list(sizes) + [1] * (len(toks) - sum(sizes)):
        rows.append(m.forward_chunk(toks[p:p + c], p, range(c), state=state))
        p += c
    return np.concatenate(rows)


def check_all_schedules(m, no, cfg, W, toks, tol=F32_TOL):
    exp, exp_layers = no.run(cfg, W, toks)
    n = len(toks)
    got, got_layers = m.forward_chunk(toks, 0, range(n), layers=True)
    assert got_layers.shape == exp_layers.shape
    assert rel(got_layers, exp_layers) < tol
    assert rel(got, exp) < tol
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < tol       # without the recording: the fused closing kernels
    assert rel(in_portions(m, toks, [n // 2]), exp) < tol
    return exp


# ---- each mechanism alone -------------------------------------------------------------------------------------------------
def plain_att(no, **a):
    return no.att(**dict(dict(heads=3, kv_heads=3, size=None, softcap=0, conv=1), **a))


YARN = (4.0, 24, 8.0, 0.5)


@pytest.mark.parametrize("kind", ["attention", "window", "grouped", "one_key_head", "value_size", "softcap", "conv", "long_conv", "two_taps", "latent", "latent_yarn",
                                  "latent_sizes", "latent_sinks", "latent_one_head", "mlstm", "mlstm_sizes", "mlstm_strong_gates", "mlstm_weak_gates", "dense", "moe",
                                  "moe_no_shared", "moe_groups", "moe_one_group_kept", "moe_all", "moe_large_shared", "loop", "loop_once", "loop_all", "loop_last"])
def test_mechanism_alone(mk, no, kind):
    """One mechanism at a time (the oracle and the model read the same config.json keys, so a key left out switches the same thing
    off in both)."""
    kw, edit = {}, None
    if kind == "attention":
        layers = [plain_att(no)]
    elif kind == "window":
        layers = [plain_att(no, size=5), plain_att(no, size=1), plain_att(no, size=16), plain_att(no, size=33)]
    elif kind == "grouped":
        layers = [plain_att(no, heads=6, kv_heads=2), plain_att(no, heads=8, kv_heads=4)]
    elif kind == "one_key_head":
        layers = [plain_att(no, heads=4, kv_heads=1), plain_att(no, heads=1, kv_heads=1)]
    elif kind == "value_size":
        layers = [plain_att(no, vdim=5), plain_att(no, vdim=17)]
    elif kind == "softcap":
        layers = [plain_att(no, softcap=0.7, scale=2.0), plain_att(no, softcap=30.0)]
    elif kind == "conv":
        layers = [plain_att(no, conv=4), plain_att(no, conv=3, heads=4, kv_heads=2, vdim=5)]
    elif kind == "long_conv":
        layers = [plain_att(no, conv=11)]
    elif kind == "two_taps":
        layers = [plain_att(no, conv=2)]
    elif kind == "latent":
        layers = [no.lat()]
    elif kind == "latent_yarn":
        layers = [no.lat(rot_dim=8, scaling=YARN), no.lat(rot_dim=12, base=10000.0, scaling=(32.0, 64, 32.0, 1.0)), no.lat(rot_dim=4, scaling=(2.0, 7, 1.0, 1.0))]
    elif kind == "latent_sizes":
        layers = [no.lat(heads=5, dim=3, rot_dim=2, vdim=9, kv_rank=7, q_rank=5), no.lat(heads=2, dim=16, rot_dim=16, vdim=1, kv_rank=40, q_rank=33)]
    elif kind == "latent_sinks":
        layers = [no.lat(heads=4)]

        def edit(W):
            W["l0.mix.sink"][:] = [8.0, -30.0, 0.0, 3.0]
    elif kind == "latent_one_head":
        layers = [no.lat(heads=1)]
    elif kind == "mlstm":
        layers = [no.mem()]
    elif kind == "mlstm_sizes":
        layers = [no.mem(heads=1, dim=3, vdim=9), no.mem(heads=5, dim=36, vdim=2), no.mem(heads=2, dim=17, vdim=41)]
    elif kind == "mlstm_strong_gates":       # gates at the cap: forgetting by e^-40 next to keeping everything, writes of e^+-40, inside one block of tokens
        layers = [no.mem(heads=4, gate_cap=40.0)]

        def edit(W):
            W["l0.mix.i"][:] *= 20.0
            W["l0.mix.f"][:] *= 20.0
            W["l0.mix.f.b"][:] = [-60.0, 60.0, 0.0, 5.0]
            W["l0.mix.i.b"][:] = [0.0, -60.0, 60.0, 0.0]
    elif kind == "mlstm_weak_gates":         # writes far below 1: the normaliser stays at its floor e^-m
        layers = [no.mem(heads=3, gate_cap=15.0)]

        def edit(W):
            W["l0.mix.i.b"][:] = [-9.0, -4.0, -1.0]
    elif kind == "dense":
        layers = [no.mem(mlp=no.dense(24)), no.mem(mlp=no.dense(9))]
    elif kind == "moe":
        layers = [no.mem(mlp=no.moe())]
    elif kind == "moe_no_shared":
        layers = [no.mem(mlp=no.moe(count=0, shared=None)), no.mem(mlp=no.moe(experts=7, top=3, ff=5, scale=0.6, shared=None))]
    elif kind == "moe_groups":
        layers = [no.mem(mlp=no.moe(12, 3, 8, 4, 2, 2.2, 20)), no.mem(mlp=no.moe(10, 4, 6, 5, 3, 0.9, 3))]
    elif kind == "moe_one_group_kept":
        layers = [no.mem(mlp=no.moe(12, 4, 8, 3, 1, 2.0, 7)), no.mem(mlp=no.moe(8, 1, 8, 8, 1, 2.0, 7))]
    elif kind == "moe_all":
        layers = [no.mem(mlp=no.moe(4, 4, 8, 2, 2, 1.0, 5)), no.mem(mlp=no.moe(1, 1, 8, 1, 1, 1.3, 1))]
    elif kind == "moe_large_shared":         # shared experts wider and narrower than the routed ones, more than 64 router rows
        layers = [no.mem(mlp=no.moe(70, 5, 6, 7, 4, 3.0, 90)), no.mem(mlp=no.moe(3, 2, 50, 3, 2, 1.0, 2))]
    elif kind == "loop":
        layers, kw = [no.mem(), plain_att(no, mlp=no.dense(12)), no.mem(mlp=no.moe())], dict(loop=(1, 2, 4))
    elif kind == "loop_once":
        layers, kw = [no.mem(), no.lat(mlp=no.moe()), no.mem()], dict(loop=(1, 3, 1))
    elif kind == "loop_all":
        layers, kw = [plain_att(no), no.mem(mlp=no.moe())], dict(loop=(0, 2, 3))
    else:
        layers, kw = [no.mem(mlp=no.moe()), no.mem()], dict(loop=(1, 2, 2))
    cfg = no.model_config(layers, **kw)
    m, W = mk(cfg, seed=3, chunk=40, edit=edit)
    toks = tokens_for(cfg, 44, 1)
    exp = check_all_schedules(m, no, cfg, W, toks)
    assert rel(in_portions(m, toks, [3, 5, 16, 4, 2]), exp) < F32_TOL


def test_mechanisms_matter(no):
    """The parts are not no-ops in the oracle: the same weights with one of them changed give other logits."""
    full = no.model_config([no.att(heads=4, kv_heads=2, dim=12, size=5, scale=0.6, softcap=2.0, mlp=no.moe(8, 3, 12, 4, 2, 1.4, 9)), no.mem(gate_cap=3.0, mlp=no.dense(12)),
                            no.lat(rot_dim=8, scaling=YARN)], loop=(1, 3, 2))
    W = no.random_weights(full, 2)
    toks = tokens_for(full, 20, 2)
    base = no.run(full, W, toks)[0]

    def without(f):
        cfg = json.loads(json.dumps(full))
        f(cfg)
        return no.run(cfg, W, toks)[0]
    mx = lambda c, i=0: c["layers"][i]["mixer"]
    rt = lambda c: c["layers"][0]["mlp"]["router"]
    for f in (lambda c: mx(c).pop("mask"), lambda c: mx(c)["mask"].update(size=4), lambda c: mx(c).update(scale=0.3), lambda c: mx(c).pop("softcap"),
              lambda c: mx(c).update(softcap=1.0), lambda c: mx(c, 1).update(gate_cap=1.0), lambda c: mx(c, 2).pop("rot"), lambda c: mx(c, 2)["rot"].pop("scaling"),
              lambda c: mx(c, 2)["rot"]["scaling"].update(factor=2.0), lambda c: mx(c, 2)["rot"].update(base=30.0), lambda c: mx(c, 2).update(scale=0.2),
              lambda c: rt(c).pop("groups"), lambda c: rt(c)["groups"].update(keep=1), lambda c: rt(c).update(top=1), lambda c: rt(c).update(scale=1.0),
              lambda c: c["layers"][0]["mlp"].pop("shared"), lambda c: c["loop"].update(times=1), lambda c: c.pop("loop")):
        assert rel(without(f), base) > 1e-3
    for name in ("l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.ls1", "l0.ls2", "final.norm", "loop.step", "loop.in", "l0.mix.q.norm", "l0.mix.k.norm",
                 "l0.mix.v.conv", "l0.mlp.shared.sg", "l0.mlp.router", "l1.mix.i", "l1.mix.i.b", "l1.mix.f", "l1.mix.f.b", "l1.mix.norm", "l1.mix.g", "l2.mix.sink",
                 "l2.mix.g", "l2.mix.dq.norm", "l2.mix.dkv.norm"):
        W2 = dict(W, **{name: W[name] * 0.5})
        assert rel(no.run(full, W2, toks)[0], base) > 1e-5, name
    for name in ("l0.mix.q.conv", "l0.mix.k.conv"):      # a factor falls out of the norm behind them; the earlier taps do not
        w = W[name].copy()
        w[:, 0] = 0.0
        assert rel(no.run(full, dict(W, **{name: w}), toks)[0], base) > 1e-4, name


# ---- schedules: whole prompt, token by token, portions ------------------------------------------------------------------------
@pytest.fixture(scope="module")
def full(mk, no):
    cfg = no.small_config()
    m, W = mk(cfg, seed=11, chunk=8)
    toks = tokens_for(cfg, 70, 4)
    exp, exp_layers = no.run(cfg, W, toks)
    return cfg, m, W, toks, exp, exp_layers


def test_whole_prompt(full):
    cfg, m, W, toks, exp, exp_layers = full
    got, got_layers = m.forward_chunk(toks, 0, range(len(toks)), layers=True)   # 70 tokens = 9 internal steps of 8
    assert got_layers.shape[0] == 6 + 3 * 2                                     # three layers run three times
    assert rel(got_layers, exp_layers) < F32_TOL
    assert rel(got, exp) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(len(toks))), exp) < F32_TOL


def test_token_by_token_equals_prefill(full):
    cfg, m, W, toks, exp, _ = full
    rows = [m.forward(int(t), i)[0].copy() for i, t in enumerate(toks)]
    assert rel(np.array(rows), exp) < F32_TOL


@pytest.mark.parametrize("chunk", [8, 64])      # steps below 32 tokens: the decode-sized attention; 32 and more: matrix products
@pytest.mark.parametrize("sizes", [[2] * 35, [3, 2, 5, 2, 7, 1, 8, 9, 2, 16, 2, 13], [33, 2, 35], [1, 69], [32, 38], [4] * 10 + [5] * 6, [17, 15, 16, 22]])
def test_portions(mk, full, chunk, sizes):
    cfg, _, W, toks, exp, _ = full
    m, _ = mk(cfg, seed=11, chunk=chunk)
    assert sum(sizes) == len(toks)
    assert rel(in_portions(m, toks, sizes), exp) < F32_TOL


def test_first_tokens_and_single_token_sequence(full, no):
    cfg, m, W, toks, exp, _ = full
    for n in (1, 2, 3, 4, 5):
        assert rel(m.forward_chunk(toks[:n], 0, range(n)), exp[:n]) < F32_TOL
    one = no.run(cfg, W, [7])[0]
    assert rel(m.forward_chunk([7], 0, [0]), one) < F32_TOL
    assert rel(m.forward(7, 0)[0], one[0]) < F32_TOL


# ---- states: interleaved sequences, states given back and used again ---------------------------------------------------
def test_interleaved_sequences_and_state_reuse(full, no):
    cfg, m, W, toks, exp, _ = full
    other = tokens_for(cfg, 41, 9)
    exp_o = no.run(cfg, W, other)[0]
    sa, sb = m.new_state(), m.new_state()
    ra, rb, pa, pb = [], [], 0, 0
    for ca, cb in [(5, 2), (1, 9), (17, 3), (2, 11), (45, 16)]:
        ra.append(m.forward_chunk(toks[pa:pa + ca], pa, range(ca), state=sa)); pa += ca
        rb.append(m.forward_chunk(other[pb:pb + cb], pb, range(cb), state=sb)); pb += cb
    assert rel(np.concatenate(ra), exp) < F32_TOL
    assert rel(np.concatenate(rb), exp_o) < F32_TOL
    # give both back and run each request in the other's state: nothing of the previous owner may show (matrix memories, their
    # running maxima, convolution inputs, ring rows)
    m.reset(state=sa); m.reset(state=sb)
    assert rel(m.forward_chunk(other, 0, range(len(other)), state=sa), exp_o) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(len(toks)), state=sb), exp) < F32_TOL
    # position 0 starts a new sequence by itself; a shorter request after a longer one in the same state
    assert rel(m.forward_chunk(other[:9], 0, range(9), state=sb), exp_o[:9]) < F32_TOL
    assert rel(in_portions(m, other[:12], [], state=sa), exp_o[:12]) < F32_TOL       # and token by token over a used state


def test_results_do_not_depend_on_what_ran_before(full):
    cfg, m, W, toks, exp, _ = full
    a = in_portions(m, toks[:30], [9, 2])
    m.forward_chunk(toks[::-1].copy(), 0, [])
    assert np.array_equal(in_portions(m, toks[:30], [9, 2]), a)


# ---- window: edges --------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("chunk", [8, 64])
@pytest.mark.parametrize("size", [1, 2, 5, 16, 24])
def test_window_edge_sensitivity(mk, no, size, chunk):
    """One layer of attention without convolutions (one tap): the logits at position i depend on the tokens i - size + 1 .. i and on
    nothing else.  Changing the token just outside changes nothing, bit for bit; changing the first token inside must.  In prompts
    and in decoding."""
    cfg = no.model_config([plain_att(no, heads=4, kv_heads=2, size=size)])
    m, W = mk(cfg, seed=21, chunk=chunk)
    n = 50

    def logits_at(toks, i, decode):
        if decode:
            m.forward_chunk(toks[:max(1, i - 6)], 0, [])
            for p in range(max(1, i - 6), i):
                m.forward_chunk(toks[p:p + 1], p, [])
            return m.forward_chunk(toks[i:i + 1], i, [0])[0]
        return m.forward_chunk(toks[:i + 1], 0, [i])[0]

    base = tokens_for(cfg, n, 5)
    for i in sorted({size, size + 1, 31, 32, n - 1}):
        first_in = i - size + 1
        for decode in (False, True):
            ref = logits_at(base, i, decode)
            outside = base.copy()
            outside[first_in - 1] = (outside[first_in - 1] + 1) % cfg["vocab"]
            assert np.array_equal(logits_at(outside, i, decode), ref)
            inside = base.copy()
            inside[first_in] = (inside[first_in] + 1) % cfg["vocab"]
            assert np.abs(logits_at(inside, i, decode) - ref).max() > 1e-5


@pytest.mark.parametrize("chunk", [8, 64])
def test_window_edges_and_far_keys_vs_oracle(mk, no, chunk):
    """Sharp attention (unit-RMS queries and keys of 8 to 12 entries, scale 6, caps of 40 and 90) over windows of 23 and 150 positions
    and over everything, with memories beside and between, so dominant keys fall on every offset to step, ring and window borders.
    Prompt in uneven portions, then decoding while keys leave the windows."""
    cfg = no.model_config([no.att(heads=3, dim=8, size=23, scale=6.0, softcap=40.0), no.mem(heads=2, dim=6, vdim=5, mlp=no.dense(6)),
                           no.att(heads=4, kv_heads=2, dim=12, vdim=6, size=150, scale=6.0, softcap=90.0, conv=5, mlp=no.moe()),
                           no.lat(heads=3, dim=9, rot_dim=4, scale=1.5, base=1000.0, scaling=YARN)])
    m, W = mk(cfg, seed=23, chunk=chunk)
    n = 330
    toks = tokens_for(cfg, n, 6)
    exp = no.run(cfg, W, toks)[0]
    assert rel(in_portions(m, toks, [7, 16, 2, 31, 9, 64, 23, 40]), exp) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL


FAR, ASKS = 39, 38      # the token whose key is to be found, and the token whose query looks for it


def far_case(m, m2, no, cfg, W, n, at, decoded):
    toks = np.random.RandomState(1).randint(0, 38, n).astype(np.int32)
    toks[at], toks[-1] = FAR, ASKS
    rows = no.run(cfg, W, toks)[0]
    lost = toks.copy()
    lost[at] = 0
    assert rel(no.run(cfg, W, lost)[0][n - 1:], rows[n - 1:]) > 0.05          # the far key carries the result in the oracle
    got = in_portions(m, toks, [n - decoded])
    assert rel(got[n - decoded - 1:], rows[n - decoded - 1:]) < F32_TOL        # decoded, the step size far below the distance
    assert rel(m.forward_chunk(toks, 0, [n - 1]), rows[n - 1:]) < F32_TOL
    assert rel(m2.forward_chunk(toks, 0, [n - 1]), rows[n - 1:]) < F32_TOL     # in a prompt, through the matrix-product path


@pytest.mark.parametrize("size,at,n", [(300, 1, 299), (150, 150, 299), (None, 0, 301)])
def test_far_key_dominates(mk, no, size, at, n):
    """A single key far back, among hundreds, takes nearly all of the softmax.  The query matrix is the key matrix behind a map that
    sends the embedding of token ASKS to that of token FAR (one tap, plain norm weights, so a key is a function of its token alone):
    the query of ASKS equals the key of FAR (score 32 per head) and meets every other key at about 0 +- 6.  FAR stands once in the
    sequence, at or near the far edge of the asking token's window."""
    cfg = no.model_config([no.att(heads=2, dim=32, vdim=8, scale=1.0, softcap=80.0, size=size, conv=1)], vocab=40)

    def edit(W):
        ea, eb = W["embed"][FAR], W["embed"][ASKS]
        W["l0.mix.q"][:] = W["l0.mix.k"] @ (np.eye(len(ea)) + np.outer(ea - eb, eb) / (eb @ eb))
        W["l0.norm1"][:] = 1.0
        W["l0.ls1"][:] = 2.0
        for t in "qk":
            W[f"l0.mix.{t}.norm"][:] = 1.0
            W[f"l0.mix.{t}.conv"][:] = 1.0
    m, W = mk(cfg, seed=33, chunk=16, edit=edit)
    m2, _ = mk(cfg, seed=33, chunk=128, edit=edit)
    far_case(m, m2, no, cfg, W, n, at, 49)


@pytest.mark.parametrize("at,n", [(0, 300), (3, 299), (140, 301)])
def test_far_latent_dominates(mk, no, at, n):
    """The same for latent attention: the plain key of FAR meets the query of ASKS with a score far above all others (the rotated part
    is kept small), hundreds of tokens back, with sinks of 0 beside it."""
    D = 24
    cfg = no.model_config([no.lat(heads=2, dim=D, rot_dim=4, vdim=8, kv_rank=30, q_rank=30, scale=1.0)], vocab=40)

    def edit(W):
        ea, eb = W["embed"][FAR], W["embed"][ASKS]
        W["l0.mix.dkv"][30:] *= 0.05
        W["l0.mix.dq"][:] = W["l0.mix.dkv"][:30] @ (np.eye(len(ea)) + np.outer(ea - eb, eb) / (eb @ eb))     # the query latent of ASKS is the latent of FAR
        uq = W["l0.mix.uq"].reshape(2, D + 4, 30)
        uq[:, :D], uq[:, D:] = W["l0.mix.uk"].reshape(2, D, 30), 0.05 * uq[:, D:]
        W["l0.norm1"][:] = 1.0
        W["l0.ls1"][:] = 2.0
        W["l0.mix.sink"][:] = 0.0
        W["l0.mix.dq.norm"][:] = W["l0.mix.dkv.norm"][:] = 1.0
    m, W = mk(cfg, seed=35, chunk=16, edit=edit)
    m2, _ = mk(cfg, seed=35, chunk=128, edit=edit)
    far_case(m, m2, no, cfg, W, n, at, 49)


@pytest.mark.parametrize("decode", [False, True])
def test_sinks_take_their_share(mk, no, decode):
    """Scores near 0 over a few keys and large values: the one (windowed attention) and the learned sinks (latent attention) hold a
    large share of the weight at the first tokens, and a sink of 12 nearly all of it."""
    cfg = no.model_config([no.att(heads=2, size=3, scale=0.01), no.lat(heads=3, scale=0.01)])

    def edit(W):
        W["l1.mix.sink"][:] = [12.0, 0.0, -12.0]
        W["l0.ls1"][:] = W["l1.ls1"][:] = 2.0
    m, W = mk(cfg, seed=36, chunk=40, edit=edit)
    toks = tokens_for(cfg, 40, 4)
    exp = no.run(cfg, W, toks)[0]
    other = dict(W)
    other["l1.mix.sink"] = W["l1.mix.sink"] * 0.0 - 30.0
    assert rel(no.run(cfg, other, toks)[0], exp) > 1e-2
    assert rel(in_portions(m, toks, [] if decode else [40]), exp) < F32_TOL


def test_memories_remember_far_tokens(mk, no):
    """Forget gates close to 1: the memories still hold the first tokens after 320, so a state, a normaliser or a running maximum that
    was lost, reset or rounded along the way shows.  Whole prompt, portions, and decoding from a carried state; across loop passes,
    each with a state of its own.  One head writes token 3 with a gate far above all later ones, so its maximum stays for ever."""
    cfg = no.model_config([no.mem(heads=3, dim=6, vdim=10, gate_cap=30.0, mlp=no.dense(8)), no.mem(heads=2, dim=9, vdim=4, gate_cap=8.0)], loop=(0, 2, 2), vocab=60)

    def edit(W):
        W["l0.mix.f.b"][:] = 29.0
        W["l0.mix.f"][:] *= 0.1
        W["l1.mix.f.b"][:] = 9.0
        W["l0.mix.i.b"][:] = [1.0, -2.0, 0.0]
    m, W = mk(cfg, seed=37, chunk=32, edit=edit)
    n = 320
    toks = tokens_for(cfg, n, 2)
    exp = no.run(cfg, W, toks)[0]
    other = toks.copy()
    other[3] = (other[3] + 1) % cfg["vocab"]
    assert rel(no.run(cfg, W, other)[0][-1:], exp[-1:]) > 1e-3            # token 3 still matters at the end, in the oracle
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [70, 2, 33, 100, 5]), exp) < F32_TOL


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("taps", [2, 3, 6])
def test_convolution_reach(mk, no, decode, taps):
    """A window of one position: the logits at position i depend on the convolutions' taps alone, tokens i - taps + 1 .. i."""
    cfg = no.model_config([no.att(size=1, conv=taps)])
    m, W = mk(cfg, seed=39, chunk=16)
    base = tokens_for(cfg, 41, 3)
    i = 40

    def at(toks):
        return in_portions(m, toks, [29, 5] if decode else [len(toks)])[i]
    ref = at(base)
    assert rel(ref, no.run(cfg, W, base)[0][i]) < F32_TOL
    for off, matters in ((taps, False), (taps - 1, True), (1, True)):
        t = base.copy()
        t[i - off] = (t[i - off] + 1) % cfg["vocab"]
        assert np.array_equal(at(t), ref) != matters


def test_expert_groups_hide_experts(mk, no):
    """A router whose best expert's runner-up lies in another group: the second choice must come from the kept group although an
    expert outside it scores higher.  The oracle without groups gives other logits."""
    cfg = no.model_config([no.mem(mlp=no.moe(8, 2, 12, 4, 1, 2.0, 4)), no.mem(mlp=no.moe(9, 3, 12, 3, 1, 2.0, None))])
    m, W = mk(cfg, seed=43, chunk=40)
    toks = tokens_for(cfg, 60, 4)
    exp = no.run(cfg, W, toks)[0]
    free = json.loads(json.dumps(cfg))
    for lc in free["layers"]:
        lc["mlp"]["router"].pop("groups")
    assert (np.abs(no.run(free, W, toks)[0] - exp).max(-1) > 1e-3 * np.abs(exp).max()).sum() > 30
    assert rel(m.forward_chunk(toks, 0, range(60)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [20, 3, 2]), exp) < F32_TOL


def test_long_decoding_wraps_the_rings(mk, no):
    """Steps of 2 tokens and windows of 5 and 3: the key rings have 6 and 4 rows and the convolution rings 9 and 12, so 160 decoded
    tokens go round them many times, while the memories are carried all the way."""
    cfg = no.model_config([no.att(heads=2, size=5, conv=2, mlp=no.moe()), no.mem(mlp=no.dense(5)), no.lat(), no.att(heads=4, kv_heads=1, dim=6, vdim=16, size=3, conv=5)],
                          loop=(0, 2, 2))
    m, W = mk(cfg, seed=29, chunk=2)
    toks = tokens_for(cfg, 160, 8)
    exp = no.run(cfg, W, toks)[0]
    assert rel(in_portions(m, toks, []), exp) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(160)), exp) < F32_TOL


def test_context_limit_and_refused_configurations(mk, no):
    import dsk
    cfg = no.model_config([no.lat(), no.att(size=None)])
    m, W = mk(cfg, seed=1, context=20, chunk=8)
    toks = tokens_for(cfg, 21, 1)
    assert rel(m.forward_chunk(toks[:20], 0, range(20)), no.run(cfg, W, toks[:20])[0]) < F32_TOL
    with pytest.raises(dsk.DskError):
        m.forward_chunk(toks[20:], 20, [0])
    for edit in (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"].update(dim=300), lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0),
                 lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][0]["mlp"]["router"].update(top=5),
                 lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3),
                 lambda c: c.update(loop={"start": 1, "stop": 5, "times": 2})):
        cfg = no.model_config([no.att(mlp=no.moe(6, 3, 8, 2, 1, 1.0, 4)), no.mem(), no.lat()])
        hc, specs = dsk.netusun_from_config(cfg, max_seq_len=32, chunk=8)
        dsk.Model(hc, layers=specs).close()
        edit(cfg)
        hc, specs = dsk.netusun_from_config(cfg, max_seq_len=32, chunk=8)
        with pytest.raises(dsk.DskError):
            dsk.Model(hc, layers=specs)


def test_incomplete_checkpoints_are_refused(no, tmp_path):
    """Every tensor of the design is required: a checkpoint that misses one does not load."""
    import dsk
    cfg = no.model_config([no.att(mlp=no.moe(3, 1, 4, 1, 1, 1.0, 4)), no.mem(mlp=no.dense(4)), no.lat()], loop=(0, 1, 2), width=8, vocab=9)
    W = no.random_weights(cfg, 1)
    for name in W:
        hc, specs = dsk.netusun_from_config(cfg, quant="fp32", max_seq_len=16, chunk=4)
        m = dsk.Model(hc, layers=specs)
        for k, a in W.items():
            if k != name:
                m.upload(k, "F32", a.shape, a.astype(np.float32))
        with pytest.raises(dsk.DskError):
            m.finalize()
        m.close()


# ---- other sizes --------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("case", ["ones", "odd", "wide", "largest_heads", "many_key_heads", "memory_first", "attention_only", "latent_only", "memory_only"])
def test_other_sizes(mk, no, case):
    kw, tol = {}, F32_TOL
    if case == "ones":      # every count that can be 1 is 1 (norms over one value turn rounding into large relative errors)
        layers = [no.att(heads=1, dim=1, vdim=1, size=1, conv=1, mlp=no.dense(1)), no.mem(heads=1, dim=1, vdim=1, mlp=no.moe(1, 1, 1, 1, 1, 1.0, 1)),
                  no.lat(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, q_rank=1)]
        kw, tol = dict(width=3, vocab=3, loop=(0, 1, 1)), 2e-3
    elif case == "odd":     # nothing is a multiple of 4; three query heads per key head
        layers = [no.att(heads=9, kv_heads=3, dim=7, vdim=5, size=11, conv=4, mlp=no.moe(9, 2, 5, 3, 2, 1.0, 7)), no.mem(heads=3, dim=7, vdim=11, mlp=no.dense(9)),
                  no.lat(heads=5, dim=7, rot_dim=6, vdim=3, kv_rank=11, q_rank=13, scaling=YARN, mlp=no.moe(5, 3, 3, 1, 1, 0.5, 5)), no.att(heads=5, kv_heads=5, dim=9, vdim=3, size=7, conv=6)]
        kw = dict(width=42, vocab=97, loop=(1, 3, 2))
    elif case == "wide":    # larger sizes: 16 heads of 64 over 4 key heads, a window wider than the prompt, memories of 128 x 64
        layers = [no.att(heads=16, kv_heads=4, dim=64, vdim=32, size=128, scale=0.11, softcap=12.0, mlp=no.moe(16, 4, 96, 4, 2, 2.0, 200)), no.mem(heads=4, dim=128, vdim=64, mlp=no.dense(320)),
                  no.lat(heads=8, dim=32, rot_dim=16, vdim=32, kv_rank=128, q_rank=96, scale=0.14, base=50000.0, scaling=(8.0, 64, 32.0, 1.0)), no.mem(heads=2, dim=32, vdim=256),
                  no.att(heads=16, kv_heads=4, dim=64, vdim=32, size=16, scale=0.11)]
        kw = dict(width=192, vocab=300)
    elif case == "largest_heads":   # states too large for one CTA's registers: the block kernels serve decoding too
        layers = [no.att(heads=2, dim=160, vdim=96, scale=0.08), no.mem(heads=2, dim=256, vdim=132), no.mem(heads=2, dim=200, vdim=200), no.lat(heads=2, dim=40, rot_dim=64, vdim=40, kv_rank=300, q_rank=200)]
        kw = dict(width=96, vocab=120)
    elif case == "many_key_heads":  # key rows too long for one CTA: the heads are dealt over CTAs
        layers = [no.att(heads=24, kv_heads=24, dim=96, vdim=64, size=20, scale=0.1)]
        kw = dict(width=64, vocab=80)
    elif case == "memory_first":
        layers = [no.mem(mlp=no.dense(12)), no.att(), no.mem(heads=2, dim=6, vdim=2), no.lat(mlp=no.dense(10))]
        kw = dict(loop=(2, 4, 2))
    elif case == "attention_only":
        layers = [no.att(mlp=no.dense(8)), no.att(heads=2, kv_heads=1, vdim=12, size=4), no.att(size=30, conv=7, mlp=no.moe())]
    elif case == "latent_only":
        layers = [no.lat(mlp=no.dense(8)), no.lat(heads=6, scaling=YARN, mlp=no.moe())]
    else:
        layers = [no.mem(mlp=no.dense(8)), no.mem(heads=4, dim=2, vdim=3, mlp=no.dense(4))]
        kw = dict(loop=(0, 2, 2))
    cfg = no.model_config(layers, **kw)
    m, W = mk(cfg, seed=31, chunk=16)
    toks = tokens_for(cfg, 45, 3)
    exp = check_all_schedules(m, no, cfg, W, toks, tol)
    if case == "ones":      # a norm over one to three values turns rounding into sign flips: no bfloat16 comparison here
        return
    mb, _ = mk(cfg, seed=31, chunk=64, quant="bf16")            # the bfloat16 kernels on the same sizes, matrix-product attention
    noise = no.rounding_noise(cfg, W, toks)
    assert close_bf16(mb.forward_chunk(toks, 0, range(45)), exp, noise)
    assert close_bf16(in_portions(mb, toks, [20]), exp, noise)


def test_large_steps_and_many_wanted_rows(mk, no):
    """A step above 256 tokens with every row wanted: two blocks of queries in the matrix-product attention, the second seeing keys
    of the first; the LM head runs over the wanted rows in several groups; the memories run over many blocks of tokens, and a thread of
    the gate scan owns several."""
    cfg = no.model_config([no.att(heads=4, kv_heads=2, size=200, mlp=no.moe(6, 2, 24, 3, 2, 1.2, 30)), no.mem(heads=4, dim=12, vdim=20, mlp=no.dense(24)), no.lat(scaling=YARN),
                           no.att(heads=4, kv_heads=2, size=50)])
    toks = tokens_for(cfg, 330, 7)
    for quant in ("fp32", "bf16"):
        m, W = mk(cfg, seed=41, chunk=512, quant=quant)
        exp = no.run(cfg, W, toks)[0]
        noise = no.rounding_noise(cfg, W, toks) if quant == "bf16" else None
        ok = (lambda a, b: rel(a, b) < F32_TOL) if quant == "fp32" else (lambda a, b: close_bf16(a, b, noise[:len(a)]))
        assert ok(m.forward_chunk(toks, 0, range(330)), exp)
        if quant == "fp32":
            assert ok(m.forward_chunk(toks[:300], 0, [0, 150, 299]), exp[[0, 150, 299]])
            assert ok(m.forward_chunk(toks[300:], 300, range(30)), exp[300:])      # a portion that continues a long step


def test_bf16_matrices(mk, no):
    cfg = no.small_config()
    m, W = mk(cfg, seed=11, quant="bf16", chunk=8)
    toks = tokens_for(cfg, 50, 4)
    exp = no.run(cfg, W, toks)[0]
    noise = no.rounding_noise(cfg, W, toks)
    assert close_bf16(m.forward_chunk(toks, 0, range(50)), exp, noise)
    assert close_bf16(in_portions(m, toks, [30]), exp, noise)


# ---- generation through the framework's own entry points -------------------------------------------------------------------------
def oracle_greedy(no, cfg, W, prompt, steps):
    seq = no.Sequence(cfg, W)
    for t in prompt:
        lg = seq.feed(int(t))
    out, margins = [], []
    for _ in range(steps):
        top = np.sort(lg)[-2:]
        margins.append(top[1] - top[0])
        out.append(int(np.argmax(lg)))
        lg = seq.feed(out[-1])
    return out, min(margins)


def test_greedy_generation(full, no):
    cfg, m, W, toks, exp, _ = full
    prompt, steps = toks[:12], 24
    want, margin = oracle_greedy(no, cfg, W, prompt, steps)
    m.forward_chunk(prompt, 0, [len(prompt) - 1])
    dev, _ = m.decode_greedy(len(prompt), steps)                # device loop: a captured step, arg-max fed back without the host
    m.forward_chunk(prompt, 0, [len(prompt) - 1])
    host = []
    for i in range(steps):                                      # the samplers' loop: dsk_sample -> dsk_forward
        host.append(m.sample(temperature=0.0))
        m.forward(host[-1], len(prompt) + i)
    assert list(dev) == host
    if margin > 1e-3:                                           # no near-tie along the way: the oracle must agree token for token
        assert host == want


def test_device_loop_continues_and_hands_over(full, no):
    """The captured step carries positions, rings and states on the device: a second run of the loop and a host step continue it."""
    cfg, m, W, toks, exp, _ = full
    prompt = toks[:10]
    m.forward_chunk(prompt, 0, [9])
    a, _ = m.decode_greedy(10, 7)
    b, _ = m.decode_greedy(17, 6)
    got, _ = m.forward(int(m.sample(temperature=0.0)), 23)
    seq = np.concatenate([prompt, a, b])
    nxt = no.run(cfg, W, seq)[0]
    last = int(np.argmax(nxt[-1]))
    assert rel(got, no.run(cfg, W, np.append(seq, last))[0][-1]) < F32_TOL


def test_launch_count_of_a_decoded_token(full):
    """dsk_launches_per_forward against the launches of the layers: 12 runs, closing norms fused with what follows."""
    cfg, m, W, toks, exp, _ = full
    import dsk
    n = dsk.lib().dsk_launches_per_forward(m.h, dsk.OUTPUT_LOGITS)
    att, mem, lat, moe, dense = 5, 3, 10, 4, 2            # launches of a mixer / feed-forward without the norms around it
    runs = [(att, moe)] + [(mem, dense), (lat, moe), (att, moe)] * 3 + [(mem, moe), (lat, None)]
    want = 3 + 1 + sum(a + 1 + ((f + 1) if f else 0) for a, f in runs) + 3 * 2     # embed, head, arg-max; first norm; passes: product and norm
    assert n == want


def test_cli_completion(full, repo):
    cfg, m, W, toks, exp, _ = full
    exe = os.path.join(repo, "deepseek.cpp_b200", "main")
    if not os.path.exists(exe):
        subprocess.check_call(["make", "-C", os.path.join(repo, "deepseek.cpp_b200"), "main"], stdout=subprocess.DEVNULL)
    prompt, steps = [int(t) for t in toks[:9]], 10
    r = subprocess.run([exe, m.dir, "-I", ",".join(map(str, prompt)), "-q", "fp32", "-n", str(steps), "-t", "0", "-T", "128"], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    ids = [int(x) for x in r.stdout.split("generated ids:")[1].split()]
    m.forward_chunk(prompt, 0, [len(prompt) - 1])
    dev, _ = m.decode_greedy(len(prompt), steps)
    assert ids == prompt + list(dev)


def test_trace_runner(full, repo, tmp_path):
    """bin/trace_run end to end: two requests in turn, portions, decoded tokens, a state given back and used again."""
    cfg, m, W, toks, exp, _ = full
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [int(t) for t in toks[:33]], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [int(t) for t in toks[33:35]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [int(toks[35])], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": [int(t) for t in toks[:8]], "want": [7, 3]}], "end": ["b"]}]
    r = subprocess.run([sys.executable, os.path.join(repo, "bin", "trace_run"), "--model", m.dir, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    V = cfg["vocab"]
    g0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V)
    g2 = np.fromfile(out / "2.f32", dtype="<f4").reshape(-1, V)
    g3 = np.fromfile(out / "3.f32", dtype="<f4").reshape(-1, V)
    assert not (out / "1.f32").exists()
    assert rel(g0, exp[[0, 32]]) < F32_TOL and rel(g2, exp[[35]]) < F32_TOL and rel(g3, exp[[7, 3]]) < F32_TOL


# ---- random designs -----------------------------------------------------------------------------------------------------------------
def random_design(no, seed):
    rng = np.random.RandomState(seed)
    n = int(rng.randint(1, 6))
    pick = lambda *v: v[rng.randint(len(v))]
    layers = []
    for _ in range(n):
        u = rng.rand()
        if u < 0.3:
            ff = None
        elif u < 0.5:
            ff = no.dense(int(rng.randint(1, 40)))
        else:
            count, per = pick(1, 2, 3, 4), pick(1, 2, 3, 5)
            keep = int(rng.randint(1, count + 1))
            ff = no.moe(count * per, int(rng.randint(1, keep * per + 1)), pick(3, 8, 20), count, keep, float(rng.uniform(0.3, 3.0)), pick(None, 1, 7, 24))
        kind = pick("a", "a", "l", "m")
        if kind == "a":
            G, rep, D = pick(1, 2, 3), pick(1, 2, 4), pick(2, 4, 6, 10, 16)
            layers.append(no.att(heads=G * rep, kv_heads=G, dim=D, vdim=pick(2, 5, 8, 20), size=pick(None, 1, 3, 8, 20, 33, 70), scale=float(rng.uniform(0.1, 1.5)),
                                 softcap=pick(0, 3.0, 20.0), conv=pick(1, 2, 3, 4, 7), mlp=ff))
        elif kind == "l":
            layers.append(no.lat(heads=pick(1, 2, 5), dim=pick(1, 4, 9, 16), rot_dim=pick(2, 4, 10), vdim=pick(1, 4, 7, 16), kv_rank=pick(3, 8, 24), q_rank=pick(2, 8, 30),
                                 scale=float(rng.uniform(0.1, 0.6)), base=pick(5.0, 100.0, 10000.0, 500000.0),
                                 scaling=pick(None, (2.0, 16, 4.0, 1.0), (8.0, 100, 32.0, 0.5), (40.0, 4096, 32.0, 1.0)), mlp=ff))
        else:
            layers.append(no.mem(heads=pick(1, 2, 3, 5), dim=pick(1, 4, 6, 10, 33, 70), vdim=pick(1, 3, 8, 20), gate_cap=pick(1.0, 6.0, 15.0), mlp=ff))
    loop = None
    if rng.rand() < 0.6:
        a = int(rng.randint(0, n))
        loop = (a, int(rng.randint(a + 1, n + 1)), pick(1, 2, 3))
    return no.model_config(layers, width=pick(8, 20, 36, 50), vocab=int(rng.randint(5, 90)), eps=pick(1e-6, 1e-5, 1e-3), loop=loop)


@pytest.mark.parametrize("seed", range(16))
def test_random_designs(mk, no, seed):
    """Layer count and order, every size, windows, rotation, groups, loop and the constants drawn at random; whole prompt, prompt +
    decoded tail, uneven portions (steps on both attention paths)."""
    cfg = random_design(no, 100 + seed)
    m, W = mk(cfg, seed=seed, chunk=40)
    n = 90
    toks = tokens_for(cfg, n, seed)
    exp = no.run(cfg, W, toks)[0]
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [60]), exp) < F32_TOL
    assert rel(in_portions(m, toks, [3, 34, 2, 2, 17, 5, 27]), exp) < F32_TOL
