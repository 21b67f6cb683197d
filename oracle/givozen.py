"""NumPy restatement of the Givozen design (test infrastructure, CPU): a decoder-only model of grouped-query attention layers
with a temperature and a gate per query head, each with an optional PolyNorm feed-forward or a mixture of clamped experts,
norms before and behind every sublayer, tied embeddings, and optionally a block of layers that runs several times.

One function per mechanism, for a WHOLE sequence of one request from position 0.  Everything is computed in `F` (float64), so
that a difference from the device is the device's rounding; `rounded()` (oracle/fuzudra.py) rounds what the device stores in
16 bits.  No code is shared with `versenext_b200/`.
"""

from __future__ import annotations

import numpy as np

from . import fuzudra as base
from .fuzudra import F, bf16, layer_runs, linear, norm, rms, rounded, sigmoid  # noqa: F401


def store(a):
    return base._store[0](a)


# ---- small pieces ---------------------------------------------------------------------------------------------
def rope_frequencies(rot):
    """Frequencies of the dims / 2 pairs.  rot['scaling'] divides those of long wavelengths (more than original / low) by
    `factor`, keeps short ones (less than original / high) and blends in between, linearly in turns over `original`."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2, dtype=F) / rot["dims"])
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for x in f:
        wave = 2 * np.pi / x
        if wave < s["original"] / s["high"]:
            out.append(x)
        elif wave > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            share = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - share) * x / s["factor"] + share * x)
    return np.array(out, F)


def rotate(x, rot, start=0):
    """x [T, heads, dim]: dimension i of the first rot.dims is paired with i + dims / 2."""
    f = rope_frequencies(rot)
    n = len(f)
    a = np.arange(start, start + x.shape[0], dtype=F)[:, None, None] * f
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * n:]], axis=-1)


def softmax_attention(q, k, v, scale, temp):
    """q [T, H, d], k [T, G, d], v [T, G, vd], temp [H] -> [T, H, vd]: causal; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    seen = np.arange(T)[None, :] <= np.arange(T)[:, None]
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        g = h // (H // k.shape[1])
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale * temp[h], -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e @ v[:, g]) / e.sum(axis=1, keepdims=True)
    return out


def attention(h, W, cfg):
    """h [T, width] -> [T, width]."""
    H, G, d, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]

    def heads(name, n, w):
        return (linear(h, W[name]) + W[name + ".b"]).reshape(T, n, w)
    q, k, v = heads("q", H, d), heads("k", G, d), heads("v", G, vd)
    if cfg.get("rot"):
        q, k = rotate(q, cfg["rot"]), rotate(k, cfg["rot"])
    o = softmax_attention(store(q), store(k), store(v), cfg["scale"], W["temp"])
    o = o * sigmoid(linear(h, W["g"]))[:, :, None]
    return linear(o.reshape(T, H * vd), W["o"])


# ---- feed-forwards --------------------------------------------------------------------------------------------
def poly_norm(z, act, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e, N: a row over its root mean square."""
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def clamped_gate(g, u, limit):
    """g sigmoid(1.702 g) (u + 1) with g capped from above and u from both sides."""
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def expert(h, W, name, limit):
    return linear(clamped_gate(linear(h, W[name + ".gate"]), linear(h, W[name + ".up"]), limit), W[name + ".down"])


def route(z, top):
    """Router logits z [T, E] -> (chosen [T, top], their sigmoids)."""
    s = sigmoid(z)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def mixture(h, W, cfg):
    r = cfg["router"]
    chosen, weight = route(linear(h, W["router"]), r["top"])
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        t, j = np.nonzero(chosen == e)
        if len(t):
            out[t] += expert(weight[t, j][:, None] * h[t], W, f"e{e}", cfg["expert"]["limit"])
    if cfg.get("shared"):
        out += sigmoid(linear(h, W["shared.sg"])) * expert(h, W, "shared", cfg["shared"]["limit"])
    return out


def feed_forward(h, W, cfg, eps):
    if cfg["kind"] == "moe":
        return mixture(h, W, cfg)
    return linear(poly_norm(store(linear(h, W["up"])), W["act"], eps), W["down"])


# ---- the model ------------------------------------------------------------------------------------------------
def _part(sd, prefix):
    return {n[len(prefix):]: np.asarray(a, F) for n, a in sd.items() if n.startswith(prefix)}


def layer(x, sd, cfg, i):
    L, eps, W = cfg["layers"][i], cfg["norm"]["eps"], _part(sd, f"l{i}.")
    mix = {n[4:]: a for n, a in W.items() if n.startswith("mix.")}
    mlp = {n[4:]: a for n, a in W.items() if n.startswith("mlp.")}
    x = x + norm(attention(norm(x, W["norm1"], eps), mix, L["mixer"]), W["norm1b"], eps)
    if L.get("mlp"):
        x = x + norm(feed_forward(norm(x, W["norm2"], eps), mlp, L["mlp"], eps), W["norm2b"], eps)
    return x


def forward(sd, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; `collect` (a list) receives the residual stream after every layer run."""
    tokens = np.asarray(tokens)
    table = np.asarray(sd["embed"], F)
    x = x0 = table[tokens]
    for i, t in layer_runs(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            x = (x + x0 if t else x) + np.asarray(sd["loop.step"], F)[t]
        x = layer(x, sd, cfg, i)
        if collect is not None:
            collect.append(x)
    return linear(norm(x, np.asarray(sd["final.norm"], F), cfg["norm"]["eps"]), table)
