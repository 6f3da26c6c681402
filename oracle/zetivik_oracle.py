"""zetivik_oracle.py — plain, slow float64 statement of the Zetivik design (a layer-list model), for tests only.

One function per mechanism, written from the equations with numpy, token by token, and sharing no code with the CUDA path.
`Sequence.feed` carries what a sequence carries: per layer run the attention keys and values, the recurrent state and the
inputs of the short convolutions that are still in reach.

Notation: W x for a stored [out, in] matrix; rms(v) = v / sqrt(mean(v^2) + eps); sg = logistic function; silu(z) = z sg(z).

  embedding:  x = e = E[token]
  layer:      x <- x + mixer(rms(x) (1 + w1));  x <- x + ff(rms(x) (1 + w2))     (a layer without a feed-forward skips the second)
  loop:       layers start .. stop-1 run `times` times; ahead of pass t:  x <- x + [t > 0] e + step[t].  Every pass keeps its own state
  attention:  q = rms_head(W_q h + b_q) w_qn, k = rms_head(W_k h + b_k) w_kn, v = W_v h + b_v;  entries (i, i + dims/2) of the first
              rot.dims entries of every q and k head turn by pos base^(-2i/dims);  p = softmax_j(scale q_h . k_j[h // (H/G)]) over the
              positions j <= i of i's own chunk of `size` positions;  W_o concat_h(sg(g_h) sum_j p_j v_j[h // (H/G)]),  g = W_g h
  delta rule: q, k [G, D], v [H, P] = silu(conv(W h)) (causal, per channel);  q, k <- unit(q) / sqrt(D), unit(k) per head, unit(z) = z / sqrt(sum z^2 + 1e-6);
              b = sg(W_b h), log a = -exp(A) softplus(W_a h + dt);  per head S <- a S;  S <- S + k (b (v - S^T k))^T;  o = S^T q;
              W_o concat_h(rms(o_h) w_n silu(g_h)),  g = W_g h
  parallel:   c_l attention(h) + c_r delta(h)
  lightning:  q, k [H, D], v [H, P] = silu(W h);  S <- a_h S + k v^T;  o = S^T q;  W_o (rms(concat o) w_n sg(W_g h))
  ff:         g = min(W_gate x, L), u = clip(W_up x, -L, L);  W_down (g sg(1.702 g) (u + 1))
  output:     z = E (rms(x) (1 + w));  logits = cap tanh(z / cap)
"""
import math

import numpy as np

from hybrid_oracle import bf16_to_f64, to_bf16, write_checkpoint  # noqa: F401  (checkpoint minting helpers)

UNIT_EPS = 1e-6


# ---- mechanisms -------------------------------------------------------------------------------------------------------
def rms(v, eps):
    v = np.asarray(v, dtype=np.float64)
    return v / math.sqrt(float(np.mean(v * v)) + eps)


def unit(v):
    return v / math.sqrt(float(np.sum(v * v)) + UNIT_EPS)


def logistic(z):
    z = np.asarray(z, dtype=np.float64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * logistic(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_half(v, rot, pos):
    """Entries (i, i + dims/2) of the first rot["dims"] entries of v turn together; the rest pass.  Positions and angles are
    32-bit numbers in this design, so the angle is a 32-bit product here too."""
    out = np.array(v, dtype=np.float64)
    if not rot or not rot.get("dims"):
        return out
    half = rot["dims"] // 2
    for i in range(half):
        a = float(np.float32(pos) * np.float32(rot["base"] ** (-2.0 * i / rot["dims"])))
        c, s = math.cos(a), math.sin(a)
        u, w = out[i], out[i + half]
        out[i], out[i + half] = u * c - w * s, w * c + u * s
    return out


def chunk_first(size, pos):
    """First position that `pos` sees: the start of its chunk, counted from the start of the sequence."""
    return 0 if size is None else (pos // size) * size


def attention_step(W, p, mx, h, pos, cache, eps):
    """One token through the attention half.  cache: {"k": [...], "v": [...]} over all earlier positions."""
    H, G, D, P = mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"], mx["vdim"]
    q = (W[p + "q"] @ h + W[p + "q.b"]).reshape(H, D)
    k = (W[p + "k"] @ h + W[p + "k.b"]).reshape(G, D)
    v = (W[p + "v"] @ h + W[p + "v.b"]).reshape(G, P)
    cache["k"].append(np.array([rotate_half(rms(k[g], eps) * W[p + "k.norm"], mx.get("rot"), pos) for g in range(G)]))
    cache["v"].append(v)
    lo = chunk_first((mx.get("mask") or {}).get("size"), pos)
    keys, vals = np.array(cache["k"][lo:]), np.array(cache["v"][lo:])
    gate = logistic(W[p + "g"] @ h)
    out = np.zeros((H, P))
    for a in range(H):
        g = a // (H // G)
        s = mx["scale"] * (keys[:, g] @ rotate_half(rms(q[a], eps) * W[p + "q.norm"], mx.get("rot"), pos))
        e = np.exp(s - s.max())
        out[a] = gate[a] * ((e / e.sum()) @ vals[:, g])
    return W[p + "o"] @ out.reshape(-1)


def short_conv(w, past, cur):
    """Per-channel convolution over the last taps - 1 inputs (older first, missing ones zero) and the current one."""
    taps = w.shape[1]
    rows = [np.zeros_like(cur)] * max(0, taps - 1 - len(past)) + list(past[-(taps - 1):] if taps > 1 else []) + [cur]
    return sum(w[:, j] * rows[j] for j in range(taps))


def delta_step(W, p, mx, h, S, past, eps):
    """One token through the gated delta rule.  S [H, D, P] is updated in place; past: inputs of the convolutions so far."""
    H, G, D, P = mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"], mx["vdim"]
    act = {}
    for n in "qkv":
        cur = W[p + n] @ h
        act[n] = silu(short_conv(W[p + n + ".conv"], past[n], cur))
        past[n].append(cur)
    q, k, v = act["q"].reshape(G, D), act["k"].reshape(G, D), act["v"].reshape(H, P)
    q = np.array([unit(r) / math.sqrt(D) for r in q])
    k = np.array([unit(r) for r in k])
    beta = logistic(W[p + "b"] @ h)
    decay = np.exp(-np.exp(W[p + "A_log"]) * softplus(W[p + "a"] @ h + W[p + "dt_bias"]))
    gate = silu(W[p + "g"] @ h).reshape(H, P)
    out = np.zeros((H, P))
    for a in range(H):
        g = a // (H // G)
        S[a] *= decay[a]
        S[a] += np.outer(k[g], beta[a] * (v[a] - S[a].T @ k[g]))
        out[a] = rms(S[a].T @ q[g], eps) * W[p + "norm"] * gate[a]
    return W[p + "o"] @ out.reshape(-1)


def lightning_step(W, p, mx, h, S, eps):
    """One token through lightning attention.  S [H, D, P] is updated in place."""
    H, D, P = mx["heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(W[p + n] @ h).reshape(H, -1) for n in "qkv")
    out = np.zeros((H, P))
    for a in range(H):
        S[a] = mx["decay"][a] * S[a] + np.outer(k[a], v[a])
        out[a] = S[a].T @ q[a]
    return W[p + "o"] @ (rms(out.reshape(-1), eps) * W[p + "norm"] * logistic(W[p + "g"] @ h))


def clamped_glu(W, p, x, limit):
    g = np.minimum(W[p + "gate"] @ x, limit)
    u = np.clip(W[p + "up"] @ x, -limit, limit)
    return W[p + "down"] @ (g * logistic(1.702 * g) * (u + 1.0))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


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
            mx = lc["mixer"]
            r = mx["right"] if lc["type"] == "parallel" else mx
            self.st.append({"k": [], "v": [], "S": np.zeros((r["heads"], r["dim"], r["vdim"])), "past": {n: [] for n in "qkv"}})
        self.pos = 0

    def feed(self, token, layers_out=None):
        cfg, W, eps = self.cfg, self.W, self.eps
        emb = W["embed"][token].astype(np.float64)
        x = emb.copy()
        for (i, opens), st in zip(self.runs, self.st):
            lc, p = cfg["layers"][i], f"l{i}."
            mx = lc["mixer"]
            if opens is not None:
                if opens > 0:
                    x = x + emb
                x = x + W["loop.step"][opens]
            h = rms(x, eps) * (1.0 + W[p + "norm1"])
            if lc["type"] == "parallel":
                x = x + mx["left_scale"] * attention_step(W, p + "mix.left.", mx["left"], h, self.pos, st, eps) \
                      + mx["right_scale"] * delta_step(W, p + "mix.right.", mx["right"], h, st["S"], st["past"], eps)
            elif lc["type"] == "lightning":
                x = x + lightning_step(W, p + "mix.", mx, h, st["S"], eps)
            else:
                raise ValueError(lc["type"])
            if lc.get("mlp"):
                x = x + clamped_glu(W, p + "mlp.", rms(x, eps) * (1.0 + W[p + "norm2"]), lc["mlp"]["limit"])
            if layers_out is not None:
                layers_out.append(x.copy())
        self.pos += 1
        return soft_cap(W["embed"] @ (rms(x, eps) * (1.0 + W["final.norm"])), cfg.get("logit_softcap"))


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

    def __matmul__(self, x):
        return self.w @ bf16_to_f64(to_bf16(np.asarray(x, dtype=np.float64))).reshape(np.shape(x))

    def __getitem__(self, i):
        return self.w[i]


def rounding_noise(cfg, W, tokens):
    """Per-token error of the logits (largest entry, in units of the largest logit) that rounding the activations of every matrix
    product to bfloat16 causes on its own."""
    R = {k: RoundedProduct(v) if v.ndim == 2 and not k.endswith(".conv") and k != "loop.step" else v for k, v in W.items()}
    exact = run(cfg, W, tokens)[0]
    return np.abs(run(cfg, R, tokens)[0] - exact).max(-1) / np.abs(exact).max()


# ---- synthetic checkpoints ------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    Wd, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, Wd), "final.norm": (Wd,)}
    if cfg.get("loop"):
        shapes["loop.step"] = (cfg["loop"]["times"], Wd)
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        shapes[p + "norm1"] = (Wd,)
        if lc["type"] == "parallel":
            a, b = mx["left"], mx["right"]
            H, G, D, P = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a["vdim"]
            l = p + "mix.left."
            shapes.update({l + "q": (H * D, Wd), l + "q.b": (H * D,), l + "k": (G * D, Wd), l + "k.b": (G * D,), l + "v": (G * P, Wd), l + "v.b": (G * P,),
                           l + "q.norm": (D,), l + "k.norm": (D,), l + "g": (H, Wd), l + "o": (Wd, H * P)})
            H, G, D, P, taps = b["heads"], b.get("kv_heads", b["heads"]), b["dim"], b["vdim"], b["conv"]
            r = p + "mix.right."
            for n, c in (("q", G * D), ("k", G * D), ("v", H * P)):
                shapes.update({r + n: (c, Wd), r + n + ".conv": (c, taps)})
            shapes.update({r + "b": (H, Wd), r + "A_log": (H,), r + "norm": (P,), r + "a": (H, Wd), r + "dt_bias": (H,), r + "g": (H * P, Wd), r + "o": (Wd, H * P)})
        else:
            H, D, P = mx["heads"], mx["dim"], mx["vdim"]
            m = p + "mix."
            shapes.update({m + "q": (H * D, Wd), m + "k": (H * D, Wd), m + "v": (H * P, Wd), m + "g": (H * P, Wd), m + "o": (Wd, H * P), m + "norm": (H * P,)})
        if lc.get("mlp"):
            ff = lc["mlp"]["ff"]
            shapes.update({p + "norm2": (Wd,), p + "mlp.gate": (ff, Wd), p + "mlp.up": (ff, Wd), p + "mlp.down": (Wd, ff)})
    return shapes


def random_weights(cfg, seed=0):
    """bfloat16-representable random weights (as float64) of a size that keeps activations O(1)."""
    rng = np.random.RandomState(seed)
    W = {}
    for name, shp in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            a = 0.3 * rng.randn(*shp)
        elif leaf == "norm":
            a = 1.0 + 0.2 * rng.randn(*shp)
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            a = 0.3 * rng.randn(*shp)
        elif leaf == "conv":
            a = rng.randn(*shp)
        elif leaf == "A_log":
            a = rng.uniform(-2.0, 1.0, shp)
        elif leaf == "dt_bias":
            a = rng.uniform(-3.0, 1.0, shp)
        elif leaf == "step":
            a = 0.5 * rng.randn(*shp)
        elif name == "embed":
            a = rng.randn(*shp)
        else:
            a = 1.5 * rng.randn(*shp) / math.sqrt(shp[-1])
        W[name] = bf16_to_f64(to_bf16(np.asarray(a, dtype=np.float64))).reshape(shp)
    return W


def write(dirname, cfg, W):
    return write_checkpoint(dirname, cfg, W)


def att(heads=4, kv_heads=None, dim=8, vdim=8, size=6, scale=0.3, dims=None, base=100.0):
    """Attention half of a parallel mixer.  size None: plain causal attention; dims 0: no rotation."""
    a = {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        a["mask"] = {"size": size}
    dims = dim if dims is None else dims
    if dims:
        a["rot"] = {"dims": dims, "base": base}
    return a


def delta(heads=2, kv_heads=None, dim=8, vdim=8, conv=4):
    """Delta-rule half of a parallel mixer."""
    return {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim, "conv": conv}


def par(left=None, right=None, cl=0.7, cr=1.1, ff=None, limit=1.5):
    """One parallel layer; ff: hidden size of the feed-forward or None."""
    return {"type": "parallel", "mixer": {"left": left or att(), "right": right or delta(), "left_scale": cl, "right_scale": cr},
            "mlp": ff_config(ff, limit)}


def light(heads=3, dim=8, vdim=8, decay=None, ff=None, limit=1.5):
    """One lightning layer; decay: one number per head."""
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": [float(d) for d in (np.linspace(0.5, 0.99, heads) if decay is None else decay)]},
            "mlp": ff_config(ff, limit)}


def ff_config(ff, limit):
    return None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}


def model_config(layers, width=40, vocab=53, eps=1e-5, cap=20.0, loop=None):
    cfg = {"architecture": "Zetivik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if cap:
        cfg["logit_softcap"] = cap
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def small_config():
    """A small model with every mechanism; sizes deliberately unequal from layer to layer and mostly not powers of two."""
    layers = [par(att(heads=6, kv_heads=2, dim=10, vdim=6, size=7, scale=0.6, dims=6, base=50.0), delta(heads=4, kv_heads=2, dim=5, vdim=7, conv=3), ff=28, limit=0.8),
              light(heads=3, dim=5, vdim=9, decay=[0.4, 0.9, 0.995]),
              par(att(heads=2, kv_heads=1, dim=12, vdim=14, size=11, scale=0.4, base=10000.0), delta(heads=3, kv_heads=1, dim=12, vdim=4, conv=5), cl=1.2, cr=0.5),
              light(heads=2, dim=12, vdim=4, decay=[0.7, 0.98], ff=20, limit=2.0),
              par(att(heads=3, kv_heads=3, dim=6, vdim=8, size=4, scale=0.9, dims=2), delta(heads=2, kv_heads=2, dim=9, vdim=8, conv=2), ff=16, limit=1.0)]
    return model_config(layers, width=44, vocab=61, cap=8.0, loop=(1, 3, 3))
