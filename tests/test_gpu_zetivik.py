"""The Zetivik design in the layer-list family (pre-norm blocks with norm weights stored around zero; grouped-query attention with
biases, weighted per-head query / key norm, half-split rotation, chunk mask and one output gate per head beside the gated delta
rule; lightning attention; clamped gated feed-forwards; a layer loop that adds the embedding again; a logit cap) against the plain
float64 statement in oracle/zetivik_oracle.py.  Every test mints its own small random checkpoint."""
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
    the same sequence (norms over a few entries can turn it into large errors in some rows, hence the quantiles)."""
    e = np.abs(np.asarray(a, np.float64) - b).max(-1) / max(np.abs(b).max(), 1e-30)
    q = lambda v, p: float(np.quantile(v, p))
    return q(e, 0.5) < 2.0 * q(noise, 0.5) + 2e-3 and q(e, 0.9) < 2.0 * q(noise, 0.9) + 5e-3 and q(e, 1.0) < 4.0 * q(noise, 1.0) + 1e-2


@pytest.fixture(scope="module")
def zo():
    import zetivik_oracle
    return zetivik_oracle


@pytest.fixture(scope="module")
def mk(tmp_path_factory, zo):
    """mk(cfg, seed, quant, chunk, context, edit) -> (dsk.Model, weights): mints the checkpoint, loads it through Model.from_dir."""
    import dsk
    root = tmp_path_factory.mktemp("zet")
    made, n = [], [0]

    def get(cfg, seed=0, quant="fp32", chunk=8, context=512, edit=None):
        W = zo.random_weights(cfg, seed)
        if edit:
            edit(W)
            W = {k: zo.bf16_to_f64(zo.to_bf16(v)).reshape(v.shape) for k, v in W.items()}
        n[0] += 1
        d = zo.write(str(root / f"m{n[0]}"), cfg, W)
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


def check_all_schedules(m, zo, cfg, W, toks, tol=F32_TOL):
    exp, exp_layers = zo.run(cfg, W, toks)
    n = len(toks)
    got, got_layers = m.forward_chunk(toks, 0, range(n), layers=True)
    assert got_layers.shape == exp_layers.shape
    assert rel(got_layers, exp_layers) < tol
    assert rel(got, exp) < tol
    assert rel(in_portions(m, toks, [n // 2]), exp) < tol
    return exp


# ---- each mechanism alone -------------------------------------------------------------------------------------------------
BARE = dict(heads=3, kv_heads=3, dim=8, vdim=8, size=None, dims=0)


def only_left(zo, ff=None, **a):
    return zo.par(zo.att(**dict(BARE, **a)), cl=1.0, cr=0.0, ff=ff)


def only_right(zo, ff=None, **b):
    return zo.par(zo.att(**BARE), zo.delta(**b), cl=0.0, cr=1.0, ff=ff)


@pytest.mark.parametrize("kind", ["attention", "rotation", "partial_rotation", "chunk_mask", "grouped", "one_key_head", "value_size", "delta", "delta_grouped",
                                  "delta_sizes", "delta_one_tap", "delta_long_conv", "delta_strong_decay", "both", "both_scales", "lightning", "lightning_sizes",
                                  "lightning_decays", "ff", "ff_limits", "loop", "loop_once", "loop_all", "no_cap"])
def test_mechanism_alone(mk, zo, kind):
    """One mechanism at a time (the oracle and the model read the same config.json keys, so a key left out switches the same thing
    off in both)."""
    kw, edit = {}, None
    if kind == "attention":
        layers = [only_left(zo)]
    elif kind == "rotation":
        layers = [only_left(zo, dims=8, base=100.0)]
    elif kind == "partial_rotation":
        layers = [only_left(zo, dim=10, dims=4, base=7.0)]
    elif kind == "chunk_mask":
        layers = [only_left(zo, size=5), only_left(zo, size=1), only_left(zo, size=16)]
    elif kind == "grouped":
        layers = [only_left(zo, heads=6, kv_heads=2)]
    elif kind == "one_key_head":
        layers = [only_left(zo, heads=4, kv_heads=1)]
    elif kind == "value_size":
        layers = [only_left(zo, vdim=5), only_left(zo, vdim=17)]
    elif kind == "delta":
        layers = [only_right(zo)]
    elif kind == "delta_grouped":
        layers = [only_right(zo, heads=6, kv_heads=2), only_right(zo, heads=9, kv_heads=1, dim=4)]
    elif kind == "delta_sizes":
        layers = [only_right(zo, heads=1, dim=3, vdim=9), only_right(zo, heads=5, dim=36, vdim=2), only_right(zo, heads=2, dim=17, vdim=41)]
    elif kind == "delta_one_tap":
        layers = [only_right(zo, conv=1)]
    elif kind == "delta_long_conv":
        layers = [only_right(zo, conv=9), only_right(zo, conv=2)]
    elif kind == "delta_strong_decay":     # decays of e^-100 next to decays near 1 inside one block of tokens
        layers = [only_right(zo, heads=4)]

        def edit(W):
            W["l0.mix.right.A_log"][:] = [3.0, 3.0, -6.0, 0.0]
            W["l0.mix.right.dt_bias"][:] = [5.0, -1.0, 0.0, 0.0]
            W["l0.mix.right.a"][:] *= 6.0
    elif kind == "both":
        layers = [zo.par(cl=1.0, cr=1.0)]
    elif kind == "both_scales":
        layers = [zo.par(cl=0.3, cr=1.7), zo.par(cl=-0.8, cr=0.4)]
    elif kind == "lightning":
        layers = [zo.light()]
    elif kind == "lightning_sizes":
        layers = [zo.light(heads=1, dim=3, vdim=9), zo.light(heads=5, dim=36, vdim=2), zo.light(heads=2, dim=17, vdim=41)]
    elif kind == "lightning_decays":
        layers = [zo.light(heads=4, decay=[0.0, 1.0, 1e-20, 0.999])]
    elif kind == "ff":
        layers = [zo.light(ff=24), only_left(zo, ff=9)]
    elif kind == "ff_limits":
        layers = [zo.light(ff=24, limit=0.2), zo.par(ff=17, limit=7.0)]
    elif kind == "loop":
        layers, kw = [zo.light(), zo.par(ff=12), zo.light(ff=8)], dict(loop=(1, 2, 4))
    elif kind == "loop_once":
        layers, kw = [zo.light(), zo.par(ff=12), zo.light()], dict(loop=(1, 3, 1))
    elif kind == "loop_all":
        layers, kw = [zo.par(), zo.light()], dict(loop=(0, 2, 3))
    else:
        layers, kw = [zo.light()], dict(cap=0)
    cfg = zo.model_config(layers, **kw)
    m, W = mk(cfg, seed=3, chunk=40, edit=edit)
    toks = tokens_for(cfg, 44, 1)
    exp = check_all_schedules(m, zo, cfg, W, toks)
    assert rel(in_portions(m, toks, [3, 5, 16, 4, 2]), exp) < F32_TOL


def test_mechanisms_matter(zo):
    """The parts are not no-ops in the oracle: the same weights with one of them changed give other logits."""
    full = zo.model_config([zo.par(zo.att(heads=4, kv_heads=2, dim=12, dims=8, base=30.0, size=5), zo.delta(conv=3), ff=12), zo.light(),
                            zo.par(zo.att(size=9), zo.delta(heads=4, kv_heads=2))], loop=(1, 3, 2))
    W = zo.random_weights(full, 2)
    toks = tokens_for(full, 20, 2)
    base = zo.run(full, W, toks)[0]

    def without(f):
        cfg = json.loads(json.dumps(full))
        f(cfg)
        return zo.run(cfg, W, toks)[0]
    mx = lambda c, i=0: c["layers"][i]["mixer"]
    for f in (lambda c: mx(c)["left"].pop("rot"), lambda c: mx(c)["left"].pop("mask"), lambda c: mx(c)["left"]["mask"].update(size=4),
              lambda c: mx(c)["left"]["rot"].update(dims=6), lambda c: mx(c)["left"].update(scale=0.2), lambda c: mx(c).update(left_scale=0.6),
              lambda c: mx(c).update(right_scale=1.0), lambda c: mx(c, 1)["decay"].reverse(), lambda c: c["layers"][0]["mlp"].update(limit=0.5),
              lambda c: c["loop"].update(times=1), lambda c: c.pop("loop"), lambda c: c.update(logit_softcap=10.0), lambda c: c.pop("logit_softcap")):
        assert rel(without(f), base) > 1e-3
    for name in ("l0.norm1", "l0.norm2", "final.norm", "loop.step", "l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.left.q.norm",
                 "l0.mix.left.k.norm", "l0.mix.left.g", "l0.mix.right.b", "l0.mix.right.a", "l0.mix.right.A_log", "l0.mix.right.dt_bias", "l0.mix.right.norm",
                 "l0.mix.right.g", "l0.mix.right.q.conv", "l0.mix.right.k.conv", "l0.mix.right.v.conv", "l1.mix.norm", "l1.mix.g"):
        W2 = dict(W, **{name: W[name] * 0.5})
        assert rel(zo.run(full, W2, toks)[0], base) > 1e-5, name


def test_delta_rule_as_the_only_mixer(mk, zo, tmp_path):
    """The delta rule without attention beside it (tensors mix.*): the same layer as a side-by-side one whose left scale is 0."""
    import dsk
    cfg = zo.model_config([only_right(zo, heads=4, kv_heads=2, dim=6, vdim=10, conv=3, ff=8), zo.light()])
    W = zo.random_weights(cfg, 4)
    toks = tokens_for(cfg, 40, 4)
    exp = zo.run(cfg, W, toks)[0]
    hc, specs = dsk.zetivik_from_config(cfg, quant="fp32", max_seq_len=64, chunk=32)
    specs[0].mixer, specs[0].mixer2 = dsk.MIX_GDN, 0
    m = dsk.Model(hc, layers=specs)
    for name, a in W.items():
        if ".mix.left." in name:
            continue
        m.upload(name.replace(".mix.right.", ".mix."), "F32", a.shape, a.astype(np.float32))
    m.finalize()
    assert rel(m.forward_chunk(toks, 0, range(40)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [7, 2, 19]), exp) < F32_TOL
    m.close()


# ---- schedules: whole prompt, token by token, portions ------------------------------------------------------------------------
@pytest.fixture(scope="module")
def full(mk, zo):
    cfg = zo.small_config()
    m, W = mk(cfg, seed=11, chunk=8)
    toks = tokens_for(cfg, 70, 4)
    exp, exp_layers = zo.run(cfg, W, toks)
    return cfg, m, W, toks, exp, exp_layers


def test_whole_prompt(full):
    cfg, m, W, toks, exp, exp_layers = full
    got, got_layers = m.forward_chunk(toks, 0, range(len(toks)), layers=True)   # 70 tokens = 9 internal steps of 8
    assert got_layers.shape[0] == 5 + 2 * 2                                     # two layers run three times
    assert rel(got_layers, exp_layers) < F32_TOL
    assert rel(got, exp) < F32_TOL


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


def test_first_tokens_and_single_token_sequence(full, zo):
    cfg, m, W, toks, exp, _ = full
    for n in (1, 2, 3, 4, 5):
        assert rel(m.forward_chunk(toks[:n], 0, range(n)), exp[:n]) < F32_TOL
    one = zo.run(cfg, W, [7])[0]
    assert rel(m.forward_chunk([7], 0, [0]), one) < F32_TOL
    assert rel(m.forward(7, 0)[0], one[0]) < F32_TOL


# ---- states: interleaved sequences, states given back and used again ---------------------------------------------------
def test_interleaved_sequences_and_state_reuse(full, zo):
    cfg, m, W, toks, exp, _ = full
    other = tokens_for(cfg, 41, 9)
    exp_o = zo.run(cfg, W, other)[0]
    sa, sb = m.new_state(), m.new_state()
    ra, rb, pa, pb = [], [], 0, 0
    for ca, cb in [(5, 2), (1, 9), (17, 3), (2, 11), (45, 16)]:
        ra.append(m.forward_chunk(toks[pa:pa + ca], pa, range(ca), state=sa)); pa += ca
        rb.append(m.forward_chunk(other[pb:pb + cb], pb, range(cb), state=sb)); pb += cb
    assert rel(np.concatenate(ra), exp) < F32_TOL
    assert rel(np.concatenate(rb), exp_o) < F32_TOL
    # give both back and run each request in the other's state: nothing of the previous owner may show (recurrent states,
    # convolution inputs, ring rows)
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


# ---- chunk mask: edges --------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("chunk", [8, 64])
@pytest.mark.parametrize("size", [1, 2, 5, 16, 24])
def test_chunk_edge_sensitivity(mk, zo, size, chunk):
    """One layer of attention alone: the logits at position i depend on the tokens of i's own chunk up to i and on nothing else.
    Changing the token ahead of the chunk changes nothing, bit for bit; changing the chunk's first token must.  In prompts and in
    decoding, for positions at, next to and far behind a chunk's start."""
    cfg = zo.model_config([only_left(zo, heads=4, kv_heads=2, dims=8, base=50.0, size=size)])
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
    start = (n - 1) // size * size
    for i in sorted({start, min(start + 1, n - 1), n - 1, start - 1}):
        first_in = i // size * size
        for decode in (False, True):
            ref = logits_at(base, i, decode)
            if first_in:
                outside = base.copy()
                outside[first_in - 1] = (outside[first_in - 1] + 1) % cfg["vocab"]
                assert np.array_equal(logits_at(outside, i, decode), ref)
            inside = base.copy()
            inside[first_in] = (inside[first_in] + 1) % cfg["vocab"]
            assert np.abs(logits_at(inside, i, decode) - ref).max() > 1e-5


@pytest.mark.parametrize("chunk", [8, 64])
def test_chunk_edges_and_far_keys_vs_oracle(mk, zo, chunk):
    """Sharp attention (unit-RMS queries and keys of 8 to 12 entries, scale 6: scores of up to +-70) over chunks of 23 and 150
    positions with recurrent parts beside and between, so dominant keys fall on every offset to step, ring and chunk borders.
    Prompt in uneven portions, then decoding while chunks end and begin in the decoded tokens."""
    cfg = zo.model_config([zo.par(zo.att(heads=3, dim=8, size=23, scale=6.0, dims=4, base=20.0), zo.delta(heads=2, dim=6, vdim=5), cr=0.3),
                           zo.light(heads=2, dim=6, vdim=5, ff=6),
                           zo.par(zo.att(heads=4, kv_heads=2, dim=12, vdim=6, size=150, scale=6.0, dims=12, base=1000.0), cr=0.2, ff=20)])
    m, W = mk(cfg, seed=23, chunk=chunk)
    n = 330
    toks = tokens_for(cfg, n, 6)
    exp = zo.run(cfg, W, toks)[0]
    assert rel(in_portions(m, toks, [7, 16, 2, 31, 9, 64, 23, 40]), exp) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL


FAR, ASKS = 39, 38      # the token whose key is to be found, and the token whose query looks for it


@pytest.mark.parametrize("size,at,n", [(300, 10, 299), (150, 151, 299), (120, 240, 301)])
def test_far_key_dominates(mk, zo, size, at, n):
    """A single key far back, among hundreds, takes nearly all of the softmax.  The query matrix is the key matrix behind a map
    that sends the embedding of token ASKS to that of token FAR (no rotation, plain norm weights, no biases, so a key is a function
    of its token alone): the query of ASKS equals the key of FAR (score 32 per head) and meets every other key at about 0 +- 6.
    FAR stands once in the sequence, at or near the start of the asking token's chunk."""
    cfg = zo.model_config([zo.par(zo.att(heads=2, kv_heads=2, dim=32, vdim=8, scale=1.0, dims=0, size=size), cl=2.0, cr=0.1)], vocab=40)

    def edit(W):
        ea, eb = W["embed"][FAR], W["embed"][ASKS]
        W["l0.mix.left.q"][:] = W["l0.mix.left.k"] @ (np.eye(len(ea)) + np.outer(ea - eb, eb) / (eb @ eb))
        W["l0.norm1"][:] = 0.0
        for t in "qk":
            W[f"l0.mix.left.{t}.b"][:] = 0.0
            W[f"l0.mix.left.{t}.norm"][:] = 1.0
    toks = np.random.RandomState(1).randint(0, 38, n).astype(np.int32)
    toks[at], toks[-1] = FAR, ASKS
    m, W = mk(cfg, seed=33, chunk=16, edit=edit)
    rows = zo.run(cfg, W, toks)[0]
    lost = toks.copy()
    lost[at] = 0
    assert rel(zo.run(cfg, W, lost)[0][n - 1:], rows[n - 1:]) > 0.05          # the far key carries the result in the oracle
    got = in_portions(m, toks, [250])
    assert rel(got[249:], rows[249:]) < F32_TOL                # decoded, the step size far below the chunk's size
    assert rel(m.forward_chunk(toks, 0, [n - 1]), rows[n - 1:]) < F32_TOL
    m2, _ = mk(cfg, seed=33, chunk=128, edit=edit)             # in a prompt, through the matrix-product path
    assert rel(m2.forward_chunk(toks, 0, [n - 1]), rows[n - 1:]) < F32_TOL


def test_recurrences_remember_far_tokens(mk, zo):
    """Decays close to 1 and small steps: the states still hold the first tokens after 300, so a state that was lost, reset or
    rounded along the way shows.  Whole prompt, portions, and decoding from a carried state; across loop passes, each with a state
    of its own."""
    cfg = zo.model_config([zo.light(heads=2, dim=6, vdim=10, decay=[0.999, 0.9995]), only_right(zo, heads=3, dim=9, vdim=4, ff=8)], loop=(0, 2, 2))

    def edit(W):
        W["l1.mix.right.A_log"][:] = -8.0
        W["l1.mix.right.b"][:] *= 0.1
    m, W = mk(cfg, seed=37, chunk=32, edit=edit)
    n = 320
    toks = tokens_for(cfg, n, 2)
    exp = zo.run(cfg, W, toks)[0]
    other = toks.copy()
    other[3] = (other[3] + 1) % cfg["vocab"]
    assert rel(zo.run(cfg, W, other)[0][-1:], exp[-1:]) > 1e-3            # token 3 still matters at the end, in the oracle
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [70, 2, 33, 100, 5]), exp) < F32_TOL


@pytest.mark.parametrize("decode", [False, True])
def test_convolution_reach(mk, zo, decode):
    """A delta rule whose decay is 0 (the state holds the current token's write only): the logits at position i depend on the
    convolution's taps alone, tokens i - taps + 1 .. i."""
    taps = 5
    cfg = zo.model_config([only_right(zo, conv=taps)])

    def edit(W):
        W["l0.mix.right.A_log"][:] = 8.0
        W["l0.mix.right.dt_bias"][:] = 20.0
        W["l0.mix.right.a"][:] = 0.0
    m, W = mk(cfg, seed=39, chunk=16, edit=edit)
    base = tokens_for(cfg, 41, 3)
    i = 40

    def at(toks):
        return in_portions(m, toks, [29, 5] if decode else [len(toks)])[i]
    ref = at(base)
    for off, matters in ((taps, False), (taps - 1, True), (1, True)):
        t = base.copy()
        t[i - off] = (t[i - off] + 1) % cfg["vocab"]
        assert np.array_equal(at(t), ref) != matters


def test_long_decoding_wraps_the_rings(mk, zo):
    """Steps of 2 tokens and chunks of 5 and 3: the key rings have 6 and 4 rows and the convolution rings 9 and 12, so 160 decoded
    tokens go round them many times, while the recurrent states are carried all the way."""
    cfg = zo.model_config([zo.par(zo.att(heads=2, size=5), zo.delta(conv=2), ff=12), zo.light(ff=5),
                           zo.par(zo.att(heads=4, kv_heads=1, dim=6, vdim=16, size=3, dims=2), zo.delta(heads=2, dim=5, vdim=3, conv=5))], loop=(0, 1, 2))
    m, W = mk(cfg, seed=29, chunk=2)
    toks = tokens_for(cfg, 160, 8)
    exp = zo.run(cfg, W, toks)[0]
    assert rel(in_portions(m, toks, []), exp) < F32_TOL
    assert rel(m.forward_chunk(toks, 0, range(160)), exp) < F32_TOL


def test_context_limit_and_refused_configurations(mk, zo):
    import dsk
    cfg = zo.model_config([zo.par(zo.att(size=None))])
    m, W = mk(cfg, seed=1, context=20, chunk=8)
    toks = tokens_for(cfg, 21, 1)
    assert rel(m.forward_chunk(toks[:20], 0, range(20)), zo.run(cfg, W, toks[:20])[0]) < F32_TOL
    with pytest.raises(dsk.DskError):
        m.forward_chunk(toks[20:], 20, [0])
    for edit in (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=3, heads=4),
                 lambda c: c["layers"][0]["mixer"]["right"].update(dim=300), lambda c: c["layers"][0]["mixer"]["right"].update(conv=0),
                 lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=10), lambda c: c["layers"][1]["mixer"]["decay"].__setitem__(0, 1.5),
                 lambda c: c.update(loop={"start": 1, "stop": 5, "times": 2})):
        cfg = zo.model_config([zo.par(zo.att(dim=8)), zo.light()])
        edit(cfg)
        hc, specs = dsk.zetivik_from_config(cfg, max_seq_len=32, chunk=8)
        with pytest.raises(dsk.DskError):
            dsk.Model(hc, layers=specs)


# ---- other sizes --------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("case", ["ones", "odd", "wide", "largest_heads", "lightning_first", "parallel_only", "lightning_only"])
def test_other_sizes(mk, zo, case):
    kw, tol = {}, F32_TOL
    if case == "ones":      # every count that can be 1 is 1 (norms over one value turn rounding into large relative errors)
        layers = [zo.par(zo.att(heads=1, dim=2, vdim=1, size=1), zo.delta(heads=1, dim=1, vdim=1, conv=1), ff=1), zo.light(heads=1, dim=1, vdim=1, ff=1)]
        kw, tol = dict(width=3, vocab=3, loop=(0, 1, 1)), 2e-3
    elif case == "odd":     # nothing is a multiple of 4; three query heads per key head; rotation of one pair only
        layers = [zo.par(zo.att(heads=9, kv_heads=3, dim=7, vdim=5, size=11, dims=2, base=3.0), zo.delta(heads=6, kv_heads=3, dim=7, vdim=11, conv=3), ff=5),
                  zo.light(heads=3, dim=7, vdim=11, ff=9), zo.par(zo.att(heads=5, kv_heads=5, dim=6, vdim=3, size=7), zo.delta(heads=5, kv_heads=1, dim=9, vdim=6, conv=7), ff=3)]
        kw = dict(width=42, vocab=97, loop=(1, 3, 2))
    elif case == "wide":    # larger sizes: 16 heads of 64 over 4 key heads, a chunk wider than the prompt, recurrent heads of 128 x 64
        layers = [zo.par(zo.att(heads=16, kv_heads=4, dim=64, vdim=32, size=128, scale=0.11, dims=48, base=50000.0), zo.delta(heads=8, kv_heads=4, dim=128, vdim=64), ff=320, limit=3.0),
                  zo.light(heads=4, dim=128, vdim=128), zo.light(heads=6, dim=64, vdim=96, ff=200),
                  zo.par(zo.att(heads=16, kv_heads=4, dim=64, vdim=32, size=16, scale=0.11, base=50000.0), zo.delta(heads=4, dim=32, vdim=256))]
        kw = dict(width=192, vocab=300)
    elif case == "largest_heads":   # states too large for one CTA's registers: the block kernels serve decoding too
        layers = [zo.par(zo.att(heads=2, dim=160, vdim=96, scale=0.08), zo.delta(heads=2, dim=200, vdim=200)), zo.light(heads=2, dim=256, vdim=132)]
        kw = dict(width=96, vocab=120)
    elif case == "lightning_first":
        layers = [zo.light(ff=12), zo.par(), zo.light(heads=2, dim=6, vdim=2), zo.par(zo.att(heads=6, kv_heads=3, vdim=8, size=9), ff=10)]
        kw = dict(loop=(2, 4, 2))
    elif case == "parallel_only":
        layers = [zo.par(ff=8), zo.par(zo.att(heads=2, kv_heads=1, vdim=12, size=4)), zo.par(zo.att(size=30), zo.delta(heads=8, kv_heads=4, dim=3, vdim=6, conv=6), ff=8)]
    else:
        layers = [zo.light(ff=8), zo.light(heads=4, dim=2, vdim=3, ff=4)]
        kw = dict(loop=(0, 2, 2))
    cfg = zo.model_config(layers, **kw)
    m, W = mk(cfg, seed=31, chunk=16)
    toks = tokens_for(cfg, 45, 3)
    exp = check_all_schedules(m, zo, cfg, W, toks, tol)
    if case == "ones":      # a norm over one to three values turns rounding into sign flips: no bfloat16 comparison here
        return
    mb, _ = mk(cfg, seed=31, chunk=64, quant="bf16")            # the bfloat16 kernels on the same sizes, matrix-product attention
    noise = zo.rounding_noise(cfg, W, toks)
    assert close_bf16(mb.forward_chunk(toks, 0, range(45)), exp, noise)
    assert close_bf16(in_portions(mb, toks, [20]), exp, noise)


def test_large_steps_and_many_wanted_rows(mk, zo):
    """A step above 256 tokens with every row wanted: two blocks of queries in the matrix-product attention, the second seeing
    keys of the first; the LM head runs over the wanted rows in several groups; the recurrences run over many blocks of tokens."""
    cfg = zo.model_config([zo.par(zo.att(heads=4, kv_heads=2, size=200), zo.delta(heads=4, kv_heads=2, dim=12, vdim=20), ff=24), zo.light(),
                           zo.par(zo.att(heads=4, kv_heads=2, size=50))])
    toks = tokens_for(cfg, 330, 7)
    for quant in ("fp32", "bf16"):
        m, W = mk(cfg, seed=41, chunk=512, quant=quant)
        exp = zo.run(cfg, W, toks)[0]
        noise = zo.rounding_noise(cfg, W, toks) if quant == "bf16" else None
        ok = (lambda a, b: rel(a, b) < F32_TOL) if quant == "fp32" else (lambda a, b: close_bf16(a, b, noise))
        assert ok(m.forward_chunk(toks, 0, range(330)), exp)
        assert ok(m.forward_chunk(toks[:300], 0, [0, 150, 299]), exp[[0, 150, 299]])
        assert ok(m.forward_chunk(toks[300:], 300, range(30)), exp[300:])      # a portion that continues a long step


def test_bf16_matrices(mk, zo):
    cfg = zo.small_config()
    m, W = mk(cfg, seed=11, quant="bf16", chunk=8)
    toks = tokens_for(cfg, 50, 4)
    exp = zo.run(cfg, W, toks)[0]
    noise = zo.rounding_noise(cfg, W, toks)
    assert close_bf16(m.forward_chunk(toks, 0, range(50)), exp, noise)
    assert close_bf16(in_portions(m, toks, [30]), exp, noise)


# ---- generation through the framework's own entry points -------------------------------------------------------------------------
def oracle_greedy(zo, cfg, W, prompt, steps):
    seq = zo.Sequence(cfg, W)
    for t in prompt:
        lg = seq.feed(int(t))
    out, margins = [], []
    for _ in range(steps):
        top = np.sort(lg)[-2:]
        margins.append(top[1] - top[0])
        out.append(int(np.argmax(lg)))
        lg = seq.feed(out[-1])
    return out, min(margins)


def test_greedy_generation(full, zo):
    cfg, m, W, toks, exp, _ = full
    prompt, steps = toks[:12], 24
    want, margin = oracle_greedy(zo, cfg, W, prompt, steps)
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


@pytest.mark.parametrize("vocab", [16384, 40001])
def test_arg_max_over_a_large_vocabulary(mk, zo, vocab):
    """The device's arg-max against numpy's on the same logits; of two equal largest logits the lower index wins."""
    cfg = zo.model_config([zo.light(heads=1, dim=4, vdim=4)], width=12, vocab=vocab, cap=0)
    m, W = mk(cfg, seed=2)
    for t in (3, 77, vocab - 1):
        lg = m.forward_chunk([5, t], 0, [1])[0]
        assert m.sample(temperature=0.0) == int(np.argmax(lg))
    best = int(np.argmax(m.forward_chunk([5, 77], 0, [1])[0]))
    twin = vocab - 2 if best < vocab // 2 else 9

    def edit(W):
        W["embed"][twin] = W["embed"][best]
    m2, _ = mk(cfg, seed=2, edit=edit)
    lg = m2.forward_chunk([5, 77], 0, [1])[0]
    assert lg[best] == lg[twin] and m2.sample(temperature=0.0) == min(best, twin)


def test_device_loop_continues_and_hands_over(full, zo):
    """The captured step carries positions, rings and states on the device: a second run of the loop and a host step continue it."""
    cfg, m, W, toks, exp, _ = full
    prompt = toks[:10]
    m.forward_chunk(prompt, 0, [9])
    a, _ = m.decode_greedy(10, 7)
    b, _ = m.decode_greedy(17, 6)
    got, _ = m.forward(int(m.sample(temperature=0.0)), 23)
    seq = np.concatenate([prompt, a, b])
    nxt = zo.run(cfg, W, seq)[0]
    last = int(np.argmax(nxt[-1]))
    assert rel(got, zo.run(cfg, W, np.append(seq, last))[0][-1]) < F32_TOL


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
def random_design(zo, seed):
    rng = np.random.RandomState(seed)
    n = int(rng.randint(1, 6))
    pick = lambda *v: v[rng.randint(len(v))]
    layers = []
    for _ in range(n):
        ff, limit = (None if rng.rand() < 0.4 else int(rng.randint(1, 40))), float(rng.uniform(0.3, 4.0))
        if rng.rand() < 0.6:
            G, rep, D = pick(1, 2, 3), pick(1, 2, 4), pick(2, 4, 6, 10, 16)
            a = zo.att(heads=G * rep, kv_heads=G, dim=D, vdim=pick(2, 5, 8, 20), size=pick(None, 1, 3, 8, 20, 33, 70), scale=float(rng.uniform(0.1, 2.0)),
                       dims=pick(*[d for d in (0, 2, 4, 6, 10, 16) if d <= D]), base=pick(5.0, 100.0, 10000.0, 500000.0))
            G = pick(1, 2, 3)
            b = zo.delta(heads=G * pick(1, 2, 3), kv_heads=G, dim=pick(1, 3, 4, 8, 18, 33, 40), vdim=pick(1, 3, 8, 20, 36), conv=pick(1, 2, 3, 4, 6, 12))
            layers.append(zo.par(a, b, cl=float(rng.uniform(0.2, 1.5)), cr=float(rng.uniform(0.2, 1.5)), ff=ff, limit=limit))
        else:
            H = pick(1, 2, 3, 5)
            layers.append(zo.light(heads=H, dim=pick(1, 4, 6, 10, 33, 70), vdim=pick(1, 3, 8, 20), decay=rng.uniform(0.3, 1.0, H), ff=ff, limit=limit))
    loop = None
    if rng.rand() < 0.6:
        a = int(rng.randint(0, n))
        loop = (a, int(rng.randint(a + 1, n + 1)), pick(1, 2, 3))
    return zo.model_config(layers, width=pick(8, 20, 36, 50), vocab=int(rng.randint(5, 90)), eps=pick(1e-6, 1e-5, 1e-3), cap=pick(0, 3.0, 30.0), loop=loop)


@pytest.mark.parametrize("seed", range(12))
def test_random_designs(mk, zo, seed):
    """Layer count and order, every size, chunks, rotation, loop and the constants drawn at random; whole prompt, prompt + decoded
    tail, uneven portions (steps on both attention paths)."""
    cfg = random_design(zo, 100 + seed)
    m, W = mk(cfg, seed=seed, chunk=40)
    n = 90
    toks = tokens_for(cfg, n, seed)
    exp = zo.run(cfg, W, toks)[0]
    assert rel(m.forward_chunk(toks, 0, range(n)), exp) < F32_TOL
    assert rel(in_portions(m, toks, [60]), exp) < F32_TOL
    assert rel(in_portions(m, toks, [3, 34, 2, 2, 17, 5, 27]), exp) < F32_TOL
