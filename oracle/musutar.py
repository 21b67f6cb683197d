"""NumPy restatement of the Musutar design (test infrastructure, CPU): a decoder-only model of sliding-window attention and
lightning attention layers over several residual streams.

Per sublayer (mixer, feed-forward): the streams are read as one weighted sum u; the sublayer sees h = layer_norm(u); its
result is gated by sigmoid(W h + b) and written back while the streams are mixed with one another.  A mixer reads h plus a
short causal convolution of h.

One function per mechanism, for a WHOLE sequence of one request from position 0, token after token where the mechanism is a
recurrence.  Everything is computed in `F` (float64), so that a difference from the device is the device's rounding;
`rounded()` (oracle/fuzudra.py) rounds what the device stores in 16 bits.  No code is shared with `versenext_b200/`.
"""

from __future__ import annotations

import numpy as np

from . import fuzudra as base
from .fuzudra import F, bf16, causal_conv, linear, rms, rounded, sigmoid, silu  # noqa: F401


def store(a):
    return base._store[0](a)


# ---- small pieces ---------------------------------------------------------------------------------------------
def layer_norm(x, w, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def rope_frequencies(rot):
    """(frequencies of the dims / 2 pairs, factor of cos and sin); YaRN when rot has 'scaling'."""
    dims, base_ = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=F)
    f = base_ ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def dim_of(turns):
        return dims * np.log(s["original"] / (2 * np.pi * turns)) / (2 * np.log(base_))
    lo, hi = max(np.floor(dim_of(s["fast"])), 0.0), min(np.ceil(dim_of(s["slow"])), dims - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(s["factor"]) + 1.0


def rotate(x, rot, start=0):
    """x [T, heads, dim]: dimension i of the first rot.dims is paired with i + dims / 2."""
    f, m = rope_frequencies(rot)
    n = len(f)
    a = np.arange(start, start + x.shape[0], dtype=F)[:, None, None] * f
    c, s = np.cos(a) * m, np.sin(a) * m
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], axis=-1)


def windowed_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, vd] -> [T, H, vd]."""
    T, H = q.shape[:2]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = (j <= i) if not window else ((j <= i) & (i - j < window))
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        g = h // (H // k.shape[1])
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e @ v[:, g]) / e.sum(axis=1, keepdims=True)
    return out


def decayed_state(q, k, v, decay, state=None):
    """One head: S <- decay S + k v^T, o = S^T q.  q, k [T, d]; v [T, vd] -> (o [T, vd], state [d, vd])."""
    S = np.zeros((k.shape[1], v.shape[1]), F) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = q[t] @ S
    return o, S


def read_streams(xs, w_in):
    return np.einsum("s,std->td", w_in, xs)


def write_streams(xs, mix, out, y):
    """mix is indexed [from, to]."""
    return np.einsum("st,snd->tnd", mix, xs) + out[:, None, None] * y[None]


# ---- mixers: h [T, width] -> [T, width]; `kept`: keys and values of the layers so far -----------------------------
def attention(h, W, cfg, eps, i, kept):
    H, G, d, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]

    def conv(name):
        return causal_conv(store(linear(h, W[name])), W[name + ".conv"])
    q = store(rotate(conv("q").reshape(T, H, d), cfg["rot"]))
    if cfg.get("kv_from") is None:
        kept[i] = (store(rotate(conv("k").reshape(T, G, d), cfg["rot"])), store(conv("v").reshape(T, G, vd)))
        k, v = kept[i]
    else:
        k, v = kept[i] = kept[cfg["kv_from"]]
    o = windowed_attention(q, k, v, cfg["scale"], (cfg.get("mask") or {}).get("size"))
    return linear(o.reshape(T, H * vd) * sigmoid(linear(h, W["g"])), W["o"])


def lightning(h, W, cfg, eps, i, kept):
    H, d, vd = cfg["heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q = store(silu(linear(h, W["q"]))).reshape(T, H, d)
    k = store(silu(linear(h, W["k"]))).reshape(T, H, d)
    v = store(silu(linear(h, W["v"]))).reshape(T, H, vd)
    o = np.stack([decayed_state(q[:, a], k[:, a], v[:, a], cfg["decay"][a])[0] for a in range(H)], axis=1)
    return linear(rms(o.reshape(T, H * vd), eps) * W["norm"] * sigmoid(linear(h, W["g"])), W["o"])


MIXERS = {"attention": attention, "lightning": lightning}


def feed_forward(h, W):
    return linear(squared_relu(linear(h, W["up"])), W["down"])


# ---- the model ------------------------------------------------------------------------------------------------
def _part(sd, prefix):
    return {n[len(prefix):]: np.asarray(a, F) for n, a in sd.items() if n.startswith(prefix)}


def sublayer(xs, q, W, eps, run):
    """One sublayer of a layer (q: 1 mixer, 2 feed-forward) on the streams xs [s, T, width]; W: the layer's tensors."""
    h = store(layer_norm(read_streams(xs, W[f"hc{q}.in"]), W[f"norm{q}"], eps))
    y = run(h) * sigmoid(linear(h, W[f"rg{q}"]) + W[f"rg{q}.b"])
    return write_streams(xs, W[f"hc{q}.mix"], W[f"hc{q}.out"], y)


def layer(xs, sd, cfg, i, kept):
    L, eps, W = cfg["layers"][i], cfg["norm"]["eps"], _part(sd, f"l{i}.")
    mix = {n[4:]: a for n, a in W.items() if n.startswith("mix.")}
    mlp = {n[4:]: a for n, a in W.items() if n.startswith("mlp.")}
    xs = sublayer(xs, 1, W, eps, lambda h: MIXERS[L["type"]](store(h + causal_conv(h, W["canon1"])), mix, L["mixer"], eps, i, kept))
    if L.get("mlp"):
        xs = sublayer(xs, 2, W, eps, lambda h: feed_forward(h, mlp))
    return xs


def forward(sd, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; `collect` (a list) receives the sum of the streams after every layer."""
    x = np.asarray(sd["embed"], F)[np.asarray(tokens)]
    xs = np.stack([x] * cfg["streams"])
    kept = {}
    for i in range(len(cfg["layers"])):
        xs = layer(xs, sd, cfg, i, kept)
        if collect is not None:
            collect.append(xs.sum(axis=0))
    return linear(layer_norm(xs.sum(axis=0), np.asarray(sd["final.norm"], F), cfg["norm"]["eps"]), np.asarray(sd["head"], F))
