"""NumPy restatement of the Fuzudra design (test infrastructure, CPU): a decoder-only model whose layers are latent
attention, a selective scan or a gated delta rule with one decay per key channel, with an optional block of layers that
is run several times with the same weights.

One function per mechanism, written for a WHOLE sequence of one request from position 0, token after token where the
mechanism is a recurrence.  Everything is computed in `F` (float64 by default), so that a difference from the device is
the device's rounding.  No code is shared with `versenext_b200/`.

Weights: dict name -> array, names as in a checkpoint ("embed", "l<i>.norm1", "l<i>.mix.<x>", "l<i>.mlp.<x>",
"final.norm", "head", "loop.in", "loop.step").
"""

from __future__ import annotations

import numpy as np

F = np.float64


def bf16(a):
    """Round to bfloat16 (nearest even), returned as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return (((u + (((u >> 16) & 1) + 0x7FFF)) >> 16) << 16).astype(np.uint32).view(np.float32)


# Applied to the operand of every matrix product and to every value that is kept for later tokens.  `rounded()` makes it
# a rounding to bfloat16, which shows what storing those in 16 bits costs at every position.
_store = [lambda a: a]


class rounded:
    def __enter__(self):
        self.old, _store[0] = _store[0], lambda a: bf16(a).astype(F)

    def __exit__(self, *exc):
        _store[0] = self.old
        return False


def linear(x, w):
    return _store[0](x) @ w.T


# ---- small pieces -----------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """The layers' norm: a weight stored around zero."""
    return rms(x, eps) * (1.0 + w)


def positions(n, width, start=0):
    """Sinusoidal position vectors [n, width]."""
    p = np.arange(start, start + n, dtype=F)[:, None]
    i = np.arange((width + 1) // 2, dtype=F)
    ang = p * 10000.0 ** (-2.0 * i / width)
    out = np.zeros((n, width), F)
    out[:, 0::2] = np.sin(ang)[:, :out[:, 0::2].shape[1]]
    out[:, 1::2] = np.cos(ang)[:, :out[:, 1::2].shape[1]]
    return out


def causal_conv(x, w, b=None):
    """Per-channel convolution over time: x [T, C], w [C, taps], the last tap meets the current token."""
    T, taps = x.shape[0], w.shape[1]
    xp = np.concatenate([np.zeros((taps - 1, x.shape[1]), F), x], axis=0)
    y = sum(xp[j:j + T] * w[:, j] for j in range(taps))
    return y if b is None else y + b


# ---- mixers: h [T, width] -> [T, width] ---------------------------------------------------------------------
def latent_attention(h, W, cfg, eps):
    H, d, vd, R = cfg["heads"], cfg["dim"], cfg["vdim"], cfg["kv_rank"]
    size = (cfg.get("mask") or {}).get("size")
    T = h.shape[0]
    q = linear(h, W["q"]).reshape(T, H, d)
    c = _store[0](rms(linear(h, W["dkv"]), eps) * W["dkv.norm"])
    k = linear(c, W["uk"]).reshape(T, H, d)
    v = linear(c, W["uv"]).reshape(T, H, vd)
    gate = sigmoid(linear(h, W["g"]))
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = (j <= i) if size is None else ((j <= i) & (i - j < size))
    out = np.zeros((T, H, vd), F)
    for a in range(H):
        s = np.where(seen, (q[:, a] @ k[:, a].T) * cfg["scale"], -np.inf)
        top = np.maximum(s.max(axis=1), W["sink"][a])
        e = np.exp(s - top[:, None])
        out[:, a] = (e @ v[:, a]) / (e.sum(axis=1) + np.exp(W["sink"][a] - top))[:, None] * gate[:, a:a + 1]
    return linear(out.reshape(T, H * vd), W["o"])


def selective_scan(x, dt, Bm, Cm, A, D, state=None):
    """x, dt [T, C]; Bm, Cm [T, N]; A [C, N]; D [C] -> (y [T, C], state [C, N])."""
    S = np.zeros(A.shape, F) if state is None else state.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * Bm[t][None, :]
        y[t] = S @ Cm[t] + D * x[t]
    return y, S


def mamba1(h, W, cfg, eps):
    n, r, N = cfg["inner"], cfg["dt_rank"], cfg["state"]
    xz = linear(h, W["in"])
    x = _store[0](silu(causal_conv(_store[0](xz[:, :n]), W["conv"], W["conv.b"])))
    p = linear(x, W["x"])
    dt = softplus(linear(p[:, :r], W["dt"]) + W["dt.b"])
    y, _ = selective_scan(x, dt, p[:, r:r + N], p[:, r + N:], -np.exp(W["A_log"]), W["D"])
    return linear(y * silu(_store[0](xz[:, n:])), W["o"])


def delta_rule(q, k, v, g, beta, state=None):
    """One head: q, k, g [T, d]; v [T, vd]; beta [T] -> (o [T, vd], state [d, vd])."""
    S = np.zeros((k.shape[1], v.shape[1]), F) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - k[t] @ S)
        S = S + np.outer(k[t], u)
        o[t] = q[t] @ S
    return o, S


def channel_delta(h, W, cfg, eps):
    H, KH, d, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q = silu(causal_conv(_store[0](linear(h, W["q"])), W["q.conv"])).reshape(T, KH, d)
    k = silu(causal_conv(_store[0](linear(h, W["k"])), W["k.conv"])).reshape(T, KH, d)
    v = silu(causal_conv(_store[0](linear(h, W["v"])), W["v.conv"])).reshape(T, H, vd)
    q = q / np.sqrt((q * q).sum(-1, keepdims=True) + 1e-6) * d ** -0.5
    k = k / np.sqrt((k * k).sum(-1, keepdims=True) + 1e-6)
    beta = sigmoid(linear(h, W["b"]))
    a = (linear(linear(h, W["a1"]), W["a2"]) + W["dt_bias"]).reshape(T, H, d)
    g = np.exp(-np.exp(W["A_log"])[None, :, None] * softplus(a))
    gate = sigmoid(linear(linear(h, W["g1"]), W["g2"])).reshape(T, H, vd)
    out = np.zeros((T, H, vd), F)
    for i in range(H):
        kh = i // (H // KH)
        o, _ = delta_rule(q[:, kh], k[:, kh], v[:, i], g[:, i], beta[:, i])
        out[:, i] = rms(o, eps) * W["norm"] * gate[:, i]
    return linear(out.reshape(T, H * vd), W["o"])


MIXERS = {"latent_attention": latent_attention, "mamba1": mamba1, "channel_delta": channel_delta}


def feed_forward(h, W):
    return linear(gelu_tanh(linear(h, W["gate"])) * linear(h, W["up"]), W["down"])


# ---- the model ----------------------------------------------------------------------------------------------
def _part(sd, prefix):
    return {n[len(prefix):]: np.asarray(a, F) for n, a in sd.items() if n.startswith(prefix)}


def layer(x, sd, cfg, i):
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    x = x + MIXERS[L["type"]](norm(x, np.asarray(sd[p + "norm1"], F), eps), _part(sd, p + "mix."), L["mixer"], eps)
    if L.get("mlp"):
        x = x + feed_forward(norm(x, np.asarray(sd[p + "norm2"], F), eps), _part(sd, p + "mlp."))
    return x


def layer_runs(cfg):
    """(layer, pass or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(sd, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; `collect` (a list) receives the residual stream after every layer run."""
    tokens = np.asarray(tokens)
    x0 = np.asarray(sd["embed"], F)[tokens]
    x0 = x0 + positions(len(tokens), x0.shape[1])
    x = x0
    for i, t in layer_runs(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            x = linear(np.concatenate([x, x0], axis=1), np.asarray(sd["loop.in"], F)) + np.asarray(sd["loop.step"], F)[t]
        x = layer(x, sd, cfg, i)
        if collect is not None:
            collect.append(x)
    return linear(norm(x, np.asarray(sd["final.norm"], F), cfg["norm"]["eps"]), np.asarray(sd["head"], F))
