"""Plain float64 restatement of the Pavitar design, one function per mechanism, query by query where the order matters.

Nothing here is shared with the product: the tests hold the CUDA path against these functions.  A model is a dict `cfg` (the parsed
config.json) and a dict `w` of numpy arrays by tensor name.  Notation: `h` is what a sublayer reads (T, width), `p0` the position of
its first row, `state` a dict that carries whatever the sequence keeps between calls (so a prompt can be fed in portions).
"""
from __future__ import annotations

import math

import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(-1, keepdims=True) + eps) * w


def sees_window(i, j, size):
    """Position i and the size - 1 before it."""
    return 0 <= i - j < size


def sees_chunk(i, j, size):
    """Positions are cut into runs of `size` from the sequence's start; only the query's own run is visible, up to the query."""
    return j <= i and j // size == i // size


def attend(q, k, v, p0, scale, sees):
    """q (T, H, d) at positions p0 .., k / v (p0 + T, G, ...): softmax over the keys that sees(i, j) lets through.  Returns (T, H, dv)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        js = [j for j in range(p0 + t + 1) if sees(p0 + t, j)]
        for h in range(H):
            g = h // (H // G)
            s = k[js, g] @ q[t, h] * scale
            e = np.exp(s - s.max())
            out[t, h] = (e / e.sum()) @ v[js, g]
    return out


def carry(state, **rows):
    """Appends the rows to what the sequence already holds under their names."""
    for n, r in rows.items():
        state[n] = np.concatenate([state[n], r]) if n in state else r
    return [state[n] for n in rows]


def latent_mixer(h, mx, w, pre, p0, state, eps):
    """Keys and values of every head come out of one normed latent row per position; no rotation; one gate value per head."""
    H, d, dv, R = mx["heads"], mx["dim"], mx["vdim"], mx["kv_rank"]
    T = h.shape[0]
    q = (rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).reshape(T, H, d)
    (c,) = carry(state, c=rms_norm(h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], eps))
    assert c.shape[1] == R
    k, v = (c @ w[pre + "uk"].T).reshape(-1, H, d), (c @ w[pre + "uv"].T).reshape(-1, H, dv)
    o = attend(q, k, v, p0, mx["scale"], lambda i, j: sees_window(i, j, mx["mask"]["size"]))
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + "o"].T


def turn_pairs(x, p0, base, dims):
    """x (T, heads, d): entries 2i and 2i + 1 of the first `dims` are the two coordinates of a point turned by position * base^(-2i / dims)."""
    x = x.copy()
    pos = p0 + np.arange(x.shape[0])
    for i in range(dims // 2):
        a = (pos * base ** (-2.0 * i / dims))[:, None]
        u, v = x[:, :, 2 * i].copy(), x[:, :, 2 * i + 1].copy()
        x[:, :, 2 * i], x[:, :, 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return x


def attention_mixer(h, mx, w, pre, p0, state, eps):
    """Queries and keys are normed as whole rows (all heads together), then split and turned."""
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = rms_norm(h @ w[pre + "q"].T, w[pre + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ w[pre + "k"].T, w[pre + "k.norm"], eps).reshape(T, G, d)
    v = (h @ w[pre + "v"].T).reshape(T, G, dv)
    rot = mx["rot"]
    q, k = turn_pairs(q, p0, rot["base"], rot["dims"]), turn_pairs(k, p0, rot["base"], rot["dims"])
    k, v = carry(state, k=k, v=v)
    o = attend(q, k, v, p0, mx["scale"], lambda i, j: sees_chunk(i, j, mx["mask"]["size"]))
    return o.reshape(T, H * dv) @ w[pre + "o"].T


MIXERS = {"latent_attention": latent_mixer, "attention": attention_mixer}


def gated_ff(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, top):
    """The `top` largest logits (ties to the lower index), weighted by the softmax over those alone.  Returns (experts, weights), best first."""
    idx = np.array([sorted(range(z.shape[1]), key=lambda e: (-z[t, e], e))[:top] for t in range(z.shape[0])])
    s = np.take_along_axis(z, idx, 1)
    s = np.exp(s - s.max(-1, keepdims=True))
    return idx, s / s.sum(-1, keepdims=True)


def expert_ff(h, mlp, w, pre):
    idx, wgt = route(h @ w[pre + "router"].T + w[pre + "router.b"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(idx[t], wgt[t]):
            out[t] += p * gated_ff(h[t], w, f"{pre}e{e}.")
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[pre + "shared.sg"].T) * gated_ff(h, w, pre + "shared.")
    return out


def layer_runs(cfg):
    """(layer index, number of the pass over the loop that begins here or 0) in the order the layers run; the passes count from 1."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, 0) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    return [(i, 0) for i in range(a)] + [(i, r + 1 if i == a else 0) for r in range(lp["times"]) for i in range(a, b)] + [(i, 0) for i in range(b, n)]


def forward(cfg, w, tokens, state, keep=None):
    """Runs `tokens` from where `state` (a dict, {} at a sequence's start) stands; returns logits (T, vocab).  keep: a list that receives the
    residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    p0 = state.get("pos", 0)
    state["pos"] = p0 + len(tokens)
    x0 = w["embed"][np.asarray(tokens)]
    x = x0
    for run, (li, begins) in enumerate(layer_runs(cfg)):
        lc, pre = cfg["layers"][li], f"l{li}."
        if begins > 1:
            x = x + x0
        x = x + MIXERS[lc["type"]](rms_norm(x, 1.0 + w[pre + "norm1"], eps), lc["mixer"], w, pre + "mix.", p0, state.setdefault(("run", run), {}), eps)
        if lc.get("mlp"):
            x = x + expert_ff(rms_norm(x, 1.0 + w[pre + "norm2"], eps), lc["mlp"], w, pre + "mlp.")
        if keep is not None:
            keep.append(x.copy())
    logits = rms_norm(x, 1.0 + w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this configuration holds, in file order."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W)}
    for li, lc in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{li}.", lc["mixer"], lc.get("mlp")
        m = p + "mix."
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        out[p + "norm1"] = (W,)
        if mlp:
            out[p + "norm2"] = (W,)
        if lc["type"] == "latent_attention":
            R, Rq = mx["kv_rank"], mx["q_rank"]
            out[m + "dq"], out[m + "dq.norm"], out[m + "uq"] = (Rq, W), (Rq,), (H * d, Rq)
            out[m + "dkv"], out[m + "dkv.norm"], out[m + "uk"], out[m + "uv"] = (R, W), (R,), (H * d, R), (H * dv, R)
            out[m + "g"] = (H, W)
        else:
            G = mx["kv_heads"]
            out[m + "q"], out[m + "k"], out[m + "v"] = (H * d, W), (G * d, W), (G * dv, W)
            out[m + "q.norm"], out[m + "k.norm"] = (H * d,), (G * d,)
        out[m + "o"] = (W, H * dv)
        if mlp:
            E = mlp["router"]["experts"]
            ffs = [(f"{p}mlp.e{e}.", mlp["expert"]["ff"]) for e in range(E)]
            if mlp.get("shared"):
                ffs.append((p + "mlp.shared.", mlp["shared"]["ff"]))
            for pe, ff in ffs:
                out[pe + "gate"], out[pe + "up"], out[pe + "down"] = (ff, W), (ff, W), (W, ff)
            out[p + "mlp.router"], out[p + "mlp.router.b"] = (E, W), (E,)
            if mlp.get("shared"):
                out[p + "mlp.shared.sg"] = (1, W)
    out["final.norm"] = (W,)
    return out


# ---- test models -------------------------------------------------------------------------------------------------------------------------
def bf16_round(a):
    """Round to the nearest bfloat16 (ties to even), as float64."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def latent_layer(heads, dim, vdim, q_rank, kv_rank, window, scale, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window}, "scale": scale}}


def attention_layer(heads, kv_heads, dim, vdim, chunk, scale, rot, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": scale,
                      "rot": {"base": rot[0], "dims": rot[1]}}}


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def make_config(vocab, width, layers, eps=1e-5, cap=12.0, loop=None):
    cfg = {"architecture": "Pavitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap:
        cfg["logit_softcap"] = cap
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed):
    """name -> float64 array, every value exactly representable in bfloat16 (so that both storage modes hold the same numbers)."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            a = rng.standard_normal(shape)
        elif len(shape) == 2:
            a = rng.standard_normal(shape) / math.sqrt(shape[1]) * (2.0 if leaf in ("g", "router", "sg") else 1.0)
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            a = 0.2 * rng.standard_normal(shape)             # stored around zero
        elif leaf == "norm":
            a = (1.0 + 0.3 * rng.standard_normal(shape)) * (1.7 if name.endswith(("q.norm", "k.norm")) else 1.0)   # sharper attention
        else:
            a = 0.8 * rng.standard_normal(shape)             # the router's bias: large enough to change choices
        w[name] = bf16_round(a)
    return w
