"""netusun_oracle.py — plain, slow float64 statement of the Netusun design (a layer-list model), for tests only.

One function per mechanism, written from the equations with numpy, token by token, and sharing no code with the CUDA path.
`Sequence.feed` carries what a sequence carries: per layer run the attention keys and values (or latents and rotated key parts),
the recurrent state, and the inputs of the short convolutions that are still in reach.

Notation: W x for a stored [out, in] matrix; rms(v) = v / sqrt(mean(v^2) + eps); sg = logistic function; silu(z) = z sg(z).

  embedding:  x = e = E[token]
  layer:      x <- x + ls1 . (rms(mixer(rms(x) w1)) w1b);  x <- x + ls2 . (rms(ff(rms(x) w2)) w2b)    (no feed-forward: no second line)
  loop:       layers start .. stop-1 run `times` times; ahead of pass t:  x <- L [x; e] + step[t].  Every pass keeps its own state
  attention:  q, k, v = conv(W h) per channel (causal, no activation);  q <- rms_head(q) w_qn, k <- rms_head(k) w_kn;  s_j = cap tanh(scale q . k_j / cap)
              over the last `size` positions;  p_j = e^s_j / (1 + sum e^s);  W_o concat_h(sum_j p_j v_j)
  latent:     q = W_uq (rms(W_dq h) w) per head [plain | turned];  [c | r] = W_dkv h, c <- rms(c) w;  keys W_uk c and the shared r, values W_uv c;
              q_turned and r rotate, entries (i, i + dims/2) together, angles pos f_i with f_i YaRN-scaled, cos and sin times 0.1 ln(factor) + 1;
              p_j = e^s_j / (e^sink_h + sum e^s) over all j <= i;  W_o (sg(W_g h) . concat_h(sum_j p_j v_j))
  mlstm:      q = W_q h / sqrt(D), k = W_k h, v = W_v h per head;  a = cap tanh((W_i h + b_i) / cap),  f = log sg(cap tanh((W_f h + b_f) / cap));
              m' = max(f + m, a);  S <- e^(f + m - m') S + e^(a - m') k v^T;  n likewise with k;  o = S^T q / (max(|n . q|, e^-m') + 1e-6);
              W_o (sg(W_g h) . w . concat_h rms(o))
  ff dense:   W_down (silu(W_gate h) (W_up h))
  ff routed:  s = softmax(R h); the experts fall into `count` groups of neighbours, those of the `keep` groups with the largest best score stay;
              the `top` largest of them, weights scale s;  + sg(g h) shared(h)
  output:     logits = E (rms(x) w)
"""
import math

import numpy as np

from hybrid_oracle import bf16_to_f64, to_bf16, write_checkpoint  # noqa: F401  (checkpoint minting helpers)

DEN_EPS = 1e-6


# ---- mechanisms -------------------------------------------------------------------------------------------------------
def rms(v, eps):
    v = np.asarray(v, dtype=np.float64)
    return v / math.sqrt(float(np.mean(v * v)) + eps)


def logistic(z):
    z = np.asarray(z, dtype=np.float64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * logistic(z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def short_conv(w, past, cur):
    """Per-channel convolution over the last taps - 1 inputs (older first, missing ones zero) and the current one."""
    taps = w.shape[1]
    rows = [np.zeros_like(cur)] * max(0, taps - 1 - len(past)) + list(past[-(taps - 1):] if taps > 1 else []) + [cur]
    return sum(w[:, j] * rows[j] for j in range(taps))


def window_first(size, pos):
    """First position that `pos` sees."""
    return 0 if size is None else max(0, pos - size + 1)


def softmax_with(scores, extra):
    """Softmax whose denominator also holds e^extra (a sink without a key)."""
    m = max(float(scores.max()), float(extra))
    e = np.exp(scores - m)
    return e / (math.exp(extra - m) + e.sum())


def attention_step(W, p, mx, h, pos, st, eps):
    """One token through windowed attention.  st: {"k": [...], "v": [...], "past": inputs of the convolutions}."""
    H, G, D, P = mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"], mx["vdim"]
    act = {}
    for n in "qkv":
        cur = W[p + n] @ h
        act[n] = short_conv(W[p + n + ".conv"], st["past"][n], cur)
        st["past"][n].append(cur)
    q, k = act["q"].reshape(H, D), act["k"].reshape(G, D)
    st["k"].append(np.array([rms(r, eps) * W[p + "k.norm"] for r in k]))
    st["v"].append(act["v"].reshape(G, P))
    lo = window_first((mx.get("mask") or {}).get("size"), pos)
    keys, vals = np.array(st["k"][lo:]), np.array(st["v"][lo:])
    out = np.zeros((H, P))
    for a in range(H):
        g = a // (H // G)
        s = soft_cap(mx["scale"] * (keys[:, g] @ (rms(q[a], eps) * W[p + "q.norm"])), mx.get("softcap"))
        out[a] = softmax_with(s, 0.0) @ vals[:, g]
    return W[p + "o"] @ out.reshape(-1)


def rotation_table(rot):
    """(frequencies, magnitude) of a rotation of rot["dims"] entries, with or without YaRN scaling."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    at = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_half(v, rot, pos):
    """Entries (i, i + dims/2) of the first rot["dims"] entries turn together; the rest pass.  Positions and angles are 32-bit
    numbers in this design, so the angle is a 32-bit product here too."""
    out = np.array(v, dtype=np.float64)
    if not rot or not rot.get("dims"):
        return out
    f, mag = rotation_table(rot)
    half = rot["dims"] // 2
    for i in range(half):
        a = float(np.float32(pos) * np.float32(f[i]))
        c, s = mag * math.cos(a), mag * math.sin(a)
        u, w = out[i], out[i + half]
        out[i], out[i + half] = u * c - w * s, w * c + u * s
    return out


def latent_step(W, p, mx, h, pos, st, eps):
    """One token through latent attention.  st: {"k": [latents], "v": [rotated key parts]}."""
    H, D, Rd, P, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    q = (W[p + "uq"] @ (rms(W[p + "dq"] @ h, eps) * W[p + "dq.norm"])).reshape(H, D + Rd)
    d = W[p + "dkv"] @ h
    st["k"].append(rms(d[:R], eps) * W[p + "dkv.norm"])
    st["v"].append(rotate_half(d[R:], mx.get("rot"), pos))
    lat, rot = np.array(st["k"]), np.array(st["v"])
    keys = (lat @ np.asarray(W[p + "uk"][:]).T).reshape(len(lat), H, D)
    vals = (lat @ np.asarray(W[p + "uv"][:]).T).reshape(len(lat), H, P)
    out = np.zeros((H, P))
    for a in range(H):
        s = mx["scale"] * (keys[:, a] @ q[a, :D] + rot @ rotate_half(q[a, D:], mx.get("rot"), pos))
        out[a] = softmax_with(s, float(W[p + "sink"][a])) @ vals[:, a]
    return W[p + "o"] @ (logistic(W[p + "g"] @ h) * out.reshape(-1))


def log_logistic(z):
    return -np.logaddexp(0.0, -z)


def mlstm_step(W, p, mx, h, st, eps):
    """One token through the matrix memory.  st: S [H, D, P], n [H, D], m [H], updated in place."""
    H, D, P, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    q, k, v = (W[p + "q"] @ h).reshape(H, D) / math.sqrt(D), (W[p + "k"] @ h).reshape(H, D), (W[p + "v"] @ h).reshape(H, P)
    li = soft_cap(W[p + "i"] @ h + W[p + "i.b"], cap)
    lf = log_logistic(soft_cap(W[p + "f"] @ h + W[p + "f.b"], cap))
    out = np.zeros((H, P))
    for a in range(H):
        m = max(lf[a] + st["m"][a], li[a])
        keep, write = math.exp(lf[a] + st["m"][a] - m), math.exp(li[a] - m)
        st["S"][a] = keep * st["S"][a] + write * np.outer(k[a], v[a])
        st["n"][a] = keep * st["n"][a] + write * k[a]
        st["m"][a] = m
        o = st["S"][a].T @ q[a] / (max(abs(float(st["n"][a] @ q[a])), math.exp(-m)) + DEN_EPS)
        out[a] = rms(o, eps)
    return W[p + "o"] @ (out.reshape(-1) * W[p + "norm"] * logistic(W[p + "g"] @ h))


def gated(W, p, x):
    return W[p + "down"] @ (silu(W[p + "gate"] @ x) * (W[p + "up"] @ x))


def route(z, r):
    """(chosen experts, weights) from the router's logits."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    gr = r.get("groups") or {"count": 1, "keep": 1}
    per = len(s) // gr["count"]
    best = [s[g * per:(g + 1) * per].max() for g in range(gr["count"])]
    kept = sorted(range(gr["count"]), key=lambda g: (-best[g], g))[:gr["keep"]]
    open_ = [e for g in kept for e in range(g * per, (g + 1) * per)]
    chosen = sorted(open_, key=lambda e: (-s[e], e))[:r["top"]]
    return chosen, [s[e] * r["scale"] for e in chosen]


def routed(W, p, ff, x):
    chosen, w = route(W[p + "router"] @ x, ff["router"])
    y = sum(we * gated(W, f"{p}e{e}.", x) for e, we in zip(chosen, w))
    if ff.get("shared"):
        y = y + float(logistic(W[p + "shared.sg"] @ x)[0]) * gated(W, p + "shared.", x)
    return y


def layer_runs(cfg):
    """(layer, pass opened by this run or None) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


# ---- a sequence -------------------------------------------------------------------------------------------------------
class Sequence:
    def __init__(self, cfg, W):
        self.cfg, self.W, self.eps = cfg, W, cfg["norm"]["eps"]
        self.runs = layer_runs(cfg)
        self.st = []
        for i, _ in self.runs:
            lc = cfg["layers"][i]
            mx, st = lc["mixer"], {"k": [], "v": [], "past": {n: [] for n in "qkv"}}
            if lc["type"] == "mlstm":
                st.update(S=np.zeros((mx["heads"], mx["dim"], mx["vdim"])), n=np.zeros((mx["heads"], mx["dim"])), m=np.zeros(mx["heads"]))
            self.st.append(st)
        self.pos = 0

    def feed(self, token, layers_out=None):
        cfg, W, eps = self.cfg, self.W, self.eps
        emb = W["embed"][token].astype(np.float64)
        x = emb.copy()
        for (i, opens), st in zip(self.runs, self.st):
            lc, p = cfg["layers"][i], f"l{i}."
            mx, m = lc["mixer"], p + "mix."
            if opens is not None:
                x = W["loop.in"] @ np.concatenate([x, emb]) + W["loop.step"][opens]
            h = rms(x, eps) * W[p + "norm1"]
            if lc["type"] == "attention":
                y = attention_step(W, m, mx, h, self.pos, st, eps)
            elif lc["type"] == "latent_attention":
                y = latent_step(W, m, mx, h, self.pos, st, eps)
            elif lc["type"] == "mlstm":
                y = mlstm_step(W, m, mx, h, st, eps)
            else:
                raise ValueError(lc["type"])
            x = x + W[p + "ls1"] * (rms(y, eps) * W[p + "norm1b"])
            if lc.get("mlp"):
                ff, h = lc["mlp"], rms(x, eps) * W[p + "norm2"]
                y = gated(W, p + "mlp.", h) if ff["kind"] == "dense" else routed(W, p + "mlp.", ff, h)
                x = x + W[p + "ls2"] * (rms(y, eps) * W[p + "norm2b"])
            if layers_out is not None:
                layers_out.append(x.copy())
        self.pos += 1
        return W["embed"] @ (rms(x, eps) * W["final.norm"])


def run(cfg, W, tokens):
    """Logits [n, vocab] and residual traces [layer runs, n, width] of a whole sequence."""
    seq = Sequence(cfg, W)
    logits, traces = [], []
    for t in tokens:
        lo = []
        logits.append(seq.feed(int(t), lo))
        traces.append(lo)
    return np.array(logits), np.array(traces).transpose(1, 0, 2)


class RoundedProduct:
    """A matrix whose products round the vector to bfloat16 first."""

    def __init__(self, w):
        self.w = w
        self.shape = w.shape

    def __matmul__(self, x):
        return self.w @ bf16_to_f64(to_bf16(np.asarray(x, dtype=np.float64))).reshape(np.shape(x))

    def __getitem__(self, i):
        return self.w[i]


def rounding_noise(cfg, W, tokens):
    """Per-token error of the logits (largest entry, in units of the largest logit) that rounding the activations of every matrix
    product but the router's to bfloat16 causes on its own."""
    R = {k: RoundedProduct(v) if v.ndim == 2 and not k.endswith((".conv", ".router", ".sg")) and k != "loop.step" else v for k, v in W.items()}
    exact = run(cfg, W, tokens)[0]
    return np.abs(run(cfg, R, tokens)[0] - exact).max(-1) / np.abs(exact).max()


# ---- synthetic checkpoints ------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    Wd, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, Wd), "final.norm": (Wd,)}
    if cfg.get("loop"):
        shapes["loop.in"], shapes["loop.step"] = (Wd, 2 * Wd), (cfg["loop"]["times"], Wd)
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        m = p + "mix."
        shapes.update({p + "norm1": (Wd,), p + "norm1b": (Wd,), p + "ls1": (Wd,)})
        H, D, P = mx["heads"], mx["dim"], mx["vdim"]
        if lc["type"] == "attention":
            G, taps = mx.get("kv_heads", H), mx["conv"]
            for n, c in (("q", H * D), ("k", G * D), ("v", G * P)):
                shapes.update({m + n: (c, Wd), m + n + ".conv": (c, taps)})
            shapes.update({m + "q.norm": (D,), m + "k.norm": (D,)})
        elif lc["type"] == "latent_attention":
            Q, R, Rd = mx["q_rank"], mx["kv_rank"], mx["rot_dim"]
            shapes.update({m + "dq": (Q, Wd), m + "dq.norm": (Q,), m + "uq": (H * (D + Rd), Q), m + "dkv": (R + Rd, Wd), m + "dkv.norm": (R,),
                           m + "uk": (H * D, R), m + "uv": (H * P, R), m + "sink": (H,), m + "g": (H * P, Wd)})
        else:
            shapes.update({m + "q": (H * D, Wd), m + "k": (H * D, Wd), m + "v": (H * P, Wd), m + "g": (H * P, Wd), m + "norm": (H * P,),
                           m + "i": (H, Wd), m + "i.b": (H,), m + "f": (H, Wd), m + "f.b": (H,)})
        shapes[m + "o"] = (Wd, H * P)
        ff = lc.get("mlp")
        if not ff:
            continue
        shapes.update({p + "norm2": (Wd,), p + "norm2b": (Wd,), p + "ls2": (Wd,)})
        glu = lambda q, f: {q + "gate": (f, Wd), q + "up": (f, Wd), q + "down": (Wd, f)}
        if ff["kind"] == "dense":
            shapes.update(glu(p + "mlp.", ff["ff"]))
        else:
            for e in range(ff["router"]["experts"]):
                shapes.update(glu(f"{p}mlp.e{e}.", ff["expert"]["ff"]))
            shapes[p + "mlp.router"] = (ff["router"]["experts"], Wd)
            if ff.get("shared"):
                shapes.update(glu(p + "mlp.shared.", ff["shared"]["ff"]))
                shapes[p + "mlp.shared.sg"] = (1, Wd)
    return shapes


def random_weights(cfg, seed=0):
    """bfloat16-representable random weights (as float64) of a size that keeps activations O(1)."""
    rng = np.random.RandomState(seed)
    W = {}
    for name, shp in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf.startswith("norm"):
            a = 1.0 + 0.2 * rng.randn(*shp)
        elif leaf in ("ls1", "ls2"):
            a = 0.7 + 0.2 * rng.randn(*shp)
        elif leaf == "conv":
            a = rng.randn(*shp)
        elif name.endswith(".i.b"):
            a = rng.uniform(-2.0, 2.0, shp)
        elif name.endswith(".f.b"):
            a = rng.uniform(0.0, 5.0, shp)
        elif leaf == "sink":
            a = rng.randn(*shp)
        elif leaf == "step":
            a = 0.5 * rng.randn(*shp)
        elif name == "embed":
            a = rng.randn(*shp)
        elif leaf == "router":
            a = 3.0 * rng.randn(*shp) / math.sqrt(shp[-1])
        else:
            a = 1.5 * rng.randn(*shp) / math.sqrt(shp[-1])
        W[name] = bf16_to_f64(to_bf16(np.asarray(a, dtype=np.float64))).reshape(shp)
    return W


def write(dirname, cfg, W):
    return write_checkpoint(dirname, cfg, W)


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=12, count=1, keep=1, scale=1.5, shared=10):
    """Routed feed-forward; shared: hidden size of the shared expert or None; count 0: no "groups" key."""
    m = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}
    if count:
        m["router"]["groups"] = {"count": count, "keep": keep}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def att(heads=4, kv_heads=None, dim=8, vdim=8, size=6, scale=0.4, softcap=5.0, conv=3, mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if size is not None:
        mx["mask"] = {"size": size}
    if softcap:
        mx["softcap"] = softcap
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def lat(heads=3, dim=8, rot_dim=4, vdim=6, kv_rank=12, q_rank=16, scale=0.35, base=100.0, scaling=None, mlp=None):
    """scaling: None or (factor, original, fast, slow)."""
    mx = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
          "rot": {"dims": rot_dim, "base": base}}
    if scaling:
        mx["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def mem(heads=3, dim=8, vdim=8, gate_cap=6.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def model_config(layers, width=40, vocab=53, eps=1e-5, loop=None):
    cfg = {"architecture": "Netusun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def small_config():
    """A small model with every mechanism; sizes deliberately unequal from layer to layer and mostly not powers of two."""
    layers = [att(heads=6, kv_heads=2, dim=10, vdim=6, size=7, scale=0.6, softcap=4.0, conv=3, mlp=moe(9, 3, 14, 3, 2, 1.7, 11)),
              mem(heads=3, dim=5, vdim=9, gate_cap=4.0, mlp=dense(28)),
              lat(heads=4, dim=9, rot_dim=6, vdim=7, kv_rank=13, q_rank=18, base=300.0, scaling=(3.0, 40, 6.0, 0.5), mlp=moe(5, 2, 8, 0, 0, 0.8, None)),
              att(heads=2, kv_heads=1, dim=12, vdim=14, size=11, scale=0.4, softcap=9.0, conv=5, mlp=moe(8, 1, 16, 4, 1, 2.5, 24)),
              mem(heads=2, dim=12, vdim=4, gate_cap=9.0, mlp=moe(4, 4, 10, 2, 2, 1.0, 6)),
              lat(heads=3, dim=6, rot_dim=8, vdim=8, kv_rank=10, q_rank=9, base=10000.0)]
    return model_config(layers, width=44, vocab=61, loop=(1, 4, 3))
