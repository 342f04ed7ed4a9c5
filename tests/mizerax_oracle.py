"""Plain float64 restatement of the Mizerax design, one function per mechanism, query by query where the order matters.

Nothing here is shared with the product: the tests hold the CUDA path against these functions.  A model is a dict `cfg` (the parsed
config.json) and a dict `w` of numpy arrays by tensor name.  Notation: `h` is what a sublayer reads (T, width), `p0` the position of
its first row, `state` a dict that carries whatever the sequence keeps between calls (so a prompt can be fed in portions).
"""
from __future__ import annotations

import math

import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def layer_norm(x, w, b, eps):
    """Mean taken off, then over the root of the mean squared deviation, then weight and bias."""
    c = x - x.mean(-1, keepdims=True)
    return c / np.sqrt((c ** 2).mean(-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(-1, keepdims=True) + eps) * w


def embed_rows(w, tokens, p0):
    """Token row plus the row of the token's position."""
    return w["embed"][np.asarray(tokens)] + w["pos"][p0:p0 + len(tokens)]


def query_temperature(p, q_temp):
    """What multiplies a query at position p: one more logarithm of the blocks of `every` positions that are complete."""
    if not q_temp:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log(math.floor((p + 1) / q_temp["every"]) + 1.0)


def head_slopes(H):
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def biased_attention(q, k, v, pos0, scale, slopes):
    """q (T, H, d) at positions pos0 .., k / v (pos0 + T, G, ...): score scale q.k - slope (i - j) for j <= i; the softmax's denominator holds one
    more term exp(0) that has no value.  Returns (T, H, dv)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        i = pos0 + t
        j = np.arange(i + 1)
        for h in range(H):
            g = h // (H // G)
            s = k[:i + 1, g] @ q[t, h] * scale - slopes[h] * (i - j)
            m = max(s.max(), 0.0)
            e = np.exp(s - m)
            out[t, h] = (e @ v[:i + 1, g]) / (e.sum() + math.exp(-m))
    return out


def attention_mixer(h, mx, w, pre, p0, state, eps):
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = rms_norm((h @ w[pre + "q"].T).reshape(T, H, d), w[pre + "q.norm"], eps)
    k = rms_norm((h @ w[pre + "k"].T).reshape(T, G, d), w[pre + "k.norm"], eps)
    v = (h @ w[pre + "v"].T).reshape(T, G, dv)
    q = q * np.array([query_temperature(p0 + t, mx.get("q_temp")) for t in range(T)])[:, None, None]
    if "k" in state:
        k, v = np.concatenate([state["k"], k]), np.concatenate([state["v"], v])
    state["k"], state["v"] = k, v
    o = biased_attention(q, k, v, p0, mx["scale"], head_slopes(H))
    o = o / (1.0 + np.exp(-(h @ w[pre + "g"].T)))[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + "o"].T


def gated_ff(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(logits, correction, top):
    """Softmax over every output (identity experts included); the choice looks at score + correction, the weights are the scores themselves.
    Returns (experts (T, top), weights (T, top)), best choice first, ties to the lower index."""
    s = np.exp(logits - logits.max(-1, keepdims=True))
    s = s / s.sum(-1, keepdims=True)
    idx = np.array([sorted(range(s.shape[1]), key=lambda e: (-(s[t, e] + correction[e]), e))[:top] for t in range(s.shape[0])])
    return idx, np.take_along_axis(s, idx, 1)


def expert_ff(h, mlp, w, pre):
    r = mlp["router"]
    E = r["experts"]
    idx, wgt = route(h @ w[pre + "router"].T, w[pre + "correction"], r["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(idx[t], wgt[t]):
            out[t] += p * (gated_ff(h[t], w, f"{pre}e{e}.") if e < E else h[t])
    if mlp.get("shared"):
        out = out + gated_ff(h, w, pre + "shared.")
    return out


def layer_runs(cfg):
    """(layer index, True where a pass over the loop begins) in the order the layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(lp["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, state, keep=None):
    """Runs `tokens` from where `state` (a dict, {} at a sequence's start) stands; returns logits (T, vocab).  keep: a list that receives the
    residual stream after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    p0 = state.get("pos", 0)
    state["pos"] = p0 + len(tokens)
    x0 = embed_rows(w, tokens, p0)
    x = x0
    for run, (li, begins) in enumerate(layer_runs(cfg)):
        lc, pre = cfg["layers"][li], f"l{li}."
        if begins:
            x = np.concatenate([x, x0], -1) @ w["loop.in"].T
        h = layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
        y = w[pre + "ls1"] * attention_mixer(h, lc["mixer"], w, pre + "mix.", p0, state.setdefault(("run", run), {}), eps)
        if lc.get("mlp"):
            y = y + w[pre + "ls2"] * expert_ff(h, lc["mlp"], w, pre + "mlp.")
        x = x + m * y
        if keep is not None:
            keep.append(x.copy())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this configuration holds, in file order."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "pos": (cfg["max_positions"], W)}
    if cfg.get("loop"):
        out["loop.in"] = (W, 2 * W)
    for li, lc in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{li}.", lc["mixer"], lc.get("mlp")
        H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        out[p + "norm1"] = out[p + "norm1.b"] = (W,)
        out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.v"] = (H * d, W), (G * d, W), (G * dv, W)
        out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (d,)
        out[p + "mix.g"], out[p + "mix.o"] = (H, W), (W, H * dv)
        if mlp:
            r = mlp["router"]
            total = r["experts"] + r.get("identity", 0)
            ffs = [(f"{p}mlp.e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
            if mlp.get("shared"):
                ffs.append((p + "mlp.shared.", mlp["shared"]["ff"]))
            for pe, ff in ffs:
                out[pe + "gate"], out[pe + "up"], out[pe + "down"] = (ff, W), (ff, W), (W, ff)
            out[p + "mlp.router"], out[p + "mlp.correction"] = (total, W), (total,)
        out[p + "ls1"] = (W,)
        if mlp:
            out[p + "ls2"] = (W,)
    out["final.norm"] = out["final.norm.b"] = (W,)
    return out


# ---- test models -------------------------------------------------------------------------------------------------------------------------
def bf16_round(a):
    """Round to the nearest bfloat16 (ties to even), as float64."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def attention_layer(heads, kv_heads, dim, vdim, scale, q_temp=None, mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if q_temp:
        mx["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def moe(ff, experts, top, identity=0, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def make_config(vocab, width, layers, max_positions=256, eps=1e-5, mult=0.5, loop=None):
    cfg = {"architecture": "Mizerax", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps}, "residual_mult": mult,
           "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed):
    """name -> float64 array, every value exactly representable in bfloat16 (so that both storage modes hold the same numbers)."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name in ("embed", "pos"):
            a = rng.standard_normal(shape)
        elif len(shape) == 2:
            a = rng.standard_normal(shape) / math.sqrt(shape[1]) * (2.0 if leaf in ("g", "router") else 1.0)
        elif leaf == "norm" or leaf == "norm1":
            a = 1.0 + 0.2 * rng.standard_normal(shape)
            if name.endswith(("q.norm", "k.norm")):
                a *= 1.5                                 # sharper attention
        elif leaf in ("ls1", "ls2"):
            a = 1.0 + 0.4 * rng.standard_normal(shape)
        elif leaf == "correction":
            a = 0.3 * rng.standard_normal(shape)         # large enough to change choices
        else:
            a = 0.3 * rng.standard_normal(shape)         # biases of the norms
        w[name] = bf16_round(a)
    return w
