"""NumPy restatement of the Bozasun design (test infrastructure, CPU): a decoder-only model of chunked grouped-query
attention, latent attention with a rotated part, and Mamba-2 layers, each with an optional gated feed-forward or a
mixture of experts, and with an input of its own for every token behind every layer.

One function per mechanism, for a WHOLE sequence of one request from position 0, token after token where the mechanism is a
recurrence.  Everything is computed in `F` (float64), so that a difference from the device is the device's rounding;
`rounded()` (oracle/fuzudra.py) rounds what the device stores in 16 bits.  No code is shared with `versenext_b200/`.
"""

from __future__ import annotations

import numpy as np

from . import fuzudra as base
from .fuzudra import F, bf16, causal_conv, gelu_tanh, linear, rms, rounded, sigmoid, silu, softplus  # noqa: F401


def store(a):
    return base._store[0](a)


# ---- small pieces ---------------------------------------------------------------------------------------------
def norm(x, w, eps):
    """RMS norm with a plain weight."""
    return rms(x, eps) * w


def rope_frequencies(rot):
    """Frequencies of the dims / 2 pairs; rot['scaling'] (linear) divides them all."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2, dtype=F) / rot["dims"])
    return f / float((rot.get("scaling") or {}).get("factor") or 1.0)


def rotate(x, rot, start=0):
    """x [T, heads, dim]: dimensions 2 i and 2 i + 1 of the first rot.dims form a pair."""
    f = rope_frequencies(rot)
    a = np.arange(start, start + x.shape[0], dtype=F)[:, None, None] * f
    y, n = x.copy(), 2 * len(f)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1:n:2] = v * np.cos(a) + u * np.sin(a)
    return y


def causal(T):
    return np.arange(T)[None, :] <= np.arange(T)[:, None]


def same_chunk(T, size):
    """Keys of the query's own chunk; chunks are counted from position 0."""
    c = np.arange(T) // size
    return causal(T) & (c[:, None] == c[None, :])


def softmax_attention(q, k, v, scale, seen, softcap=None):
    """q [T, H, d], k [T, G, d], v [T, G, vd] -> [T, H, vd]; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        g = h // (H // k.shape[1])
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * np.tanh(s / softcap)
        s = np.where(seen, s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e @ v[:, g]) / e.sum(axis=1, keepdims=True)
    return out


def ssm(x, B, C, dt, A, D, state=None):
    """One head of the state-space recurrence: x [T, P], B and C [T, N], dt [T], A < 0 and D numbers.
    S <- exp(A dt) S + dt B x^T, y = S^T C + D x -> (y [T, P], S [N, P])."""
    S = np.zeros((B.shape[1], x.shape[1]), F) if state is None else state.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(A * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        y[t] = C[t] @ S + D * x[t]
    return y, S


def grouped_rms(x, groups, eps):
    T = x.shape[0]
    return rms(x.reshape(T, groups, -1), eps).reshape(T, -1)


# ---- mixers: h [T, width] -> [T, width] ---------------------------------------------------------------------
def attention(h, W, cfg, eps):
    H, G, d, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]

    def head(name, n, w):
        return (linear(h, W[name]) + W[name + ".b"]).reshape(T, n, w)
    q = store(rotate(norm(head("q", H, d), W["q.norm"], eps), cfg["rot"]))
    k = store(rotate(norm(head("k", G, d), W["k.norm"], eps), cfg["rot"]))
    v = store(head("v", G, vd))
    size = (cfg.get("mask") or {}).get("size")
    o = softmax_attention(q, k, v, cfg["scale"], same_chunk(T, size) if size else causal(T), cfg.get("softcap"))
    return linear(o.reshape(T, H * vd), W["o"]) + W["o.b"]


def latent_attention(h, W, cfg, eps):
    H, d, r, vd, R = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    T = h.shape[0]
    q = linear(h, W["q"]).reshape(T, H, d + r)
    down = linear(h, W["dkv"])
    c = store(norm(down[:, :R], W["dkv.norm"], eps))
    shared = rotate(down[:, None, R:], cfg["rot"])
    k = np.concatenate([linear(c, W["uk"]).reshape(T, H, d), np.repeat(shared, H, axis=1)], axis=2)
    q = np.concatenate([q[..., :d], rotate(q[..., d:], cfg["rot"])], axis=2)
    o = softmax_attention(store(q), store(k), linear(c, W["uv"]).reshape(T, H, vd), cfg["scale"], causal(T))
    return linear(o.reshape(T, H * vd) * sigmoid(linear(h, W["g"])), W["o"])


def mamba2(h, W, cfg, eps):
    H, P, N, G = cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    T, n = h.shape[0], H * P
    z, xbc, dt = np.split(linear(h, W["in"]), [n, 2 * n + 2 * G * N], axis=1)
    x, B, C = np.split(store(silu(causal_conv(store(xbc), W["conv"], W["conv.b"]))), [n, n + G * N], axis=1)
    dt = softplus(dt + W["dt_bias"])
    y = []
    for a in range(H):
        g = slice(a // (H // G) * N, (a // (H // G) + 1) * N)
        y.append(ssm(x[:, a * P:(a + 1) * P], B[:, g], C[:, g], dt[:, a], -np.exp(W["A_log"][a]), W["D"][a])[0])
    u = np.concatenate(y, axis=1) * silu(z)
    return linear(grouped_rms(u, cfg["norm_groups"], eps) * W["norm"], W["o"])


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mamba2": mamba2}


# ---- feed-forwards --------------------------------------------------------------------------------------------
def gated(h, gate, up, down):
    return linear(silu(linear(h, gate)) * linear(h, up), down)


def route(z, correction, top, groups, keep):
    """Router logits z [T, E] -> (chosen [T, top], their weights): soft-max over all; the choice, made among the `keep` groups
    of neighbours with the largest member, sees the correction, the weights do not."""
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    choice = s + correction
    T, E = z.shape
    best = choice.reshape(T, groups, E // groups).max(axis=2)
    kept = np.zeros((T, groups), bool)
    np.put_along_axis(kept, np.argsort(-best, axis=1, kind="stable")[:, :keep], True, axis=1)
    choice = np.where(np.repeat(kept, E // groups, axis=1), choice, -np.inf)
    chosen = np.argsort(-choice, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def experts(h, W, cfg):
    r = cfg["router"]
    n, groups = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    chosen, weight = route(linear(h, W["router"]), W["correction"], r["top"], groups["count"], groups["keep"])
    out = np.zeros_like(h)
    for e in range(n + r.get("identity", 0)):
        t, j = np.nonzero(chosen == e)
        if len(t):
            y = gated(h[t], *(W[f"e{e}.{p}"] for p in ("gate", "up", "down"))) if e < n else store(h[t])
            out[t] += weight[t, j][:, None] * y
    return out


def feed_forward(h, W, cfg):
    return experts(h, W, cfg) if cfg["kind"] == "moe" else gated(h, W["gate"], W["up"], W["down"])


def side_input(x, e, W, eps):
    """What a layer adds for the token itself: e [T, dim] is the layer's part of the tokens' side embeddings."""
    y = linear(gelu_tanh(linear(x, W["side.gate"])) * e, W["side.proj"])
    return rms(y, eps) * W["side.norm"]


# ---- the model ------------------------------------------------------------------------------------------------
def _part(sd, prefix):
    return {n[len(prefix):]: np.asarray(a, F) for n, a in sd.items() if n.startswith(prefix)}


def layer(x, tokens, sd, cfg, i):
    L, eps, W = cfg["layers"][i], cfg["norm"]["eps"], _part(sd, f"l{i}.")
    mix = {n[4:]: a for n, a in W.items() if n.startswith("mix.")}
    mlp = {n[4:]: a for n, a in W.items() if n.startswith("mlp.")}
    x = x + MIXERS[L["type"]](norm(x, W["norm1"], eps), mix, L["mixer"], eps)
    if L.get("mlp"):
        x = x + feed_forward(norm(x, W["norm2"], eps), mlp, L["mlp"])
    n = cfg["token_side"]["dim"]
    return x + side_input(x, np.asarray(sd["side.embed"], F)[tokens, i * n:(i + 1) * n], W, eps)


def forward(sd, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; `collect` (a list) receives the residual after every layer."""
    tokens = np.asarray(tokens)
    x = np.asarray(sd["embed"], F)[tokens]
    for i in range(len(cfg["layers"])):
        x = layer(x, tokens, sd, cfg, i)
        if collect is not None:
            collect.append(x)
    return linear(norm(x, np.asarray(sd["final.norm"], F), cfg["norm"]["eps"]), np.asarray(sd["head"], F))
