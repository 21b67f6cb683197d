"""Small random models of the Bozasun design for the tests: configurations, weights, prompts."""

import numpy as np

from oracle import bozasun as OB
from oracle.fuzudra import bf16
import fuzudra_cases as FC
from fuzudra_cases import err  # noqa: F401

CODE = 8          # of the width: dimensions that only the embedding writes and that routers read


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=3, top=3, groups=5, keep=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top,
                                                             "groups": {"count": groups, "keep": keep}}}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, chunk=37, scale=0.3, rot=16, base=1000.0, factor=2.5, softcap=6.0, mlp=dense()):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "mask": {"size": chunk} if chunk else None,
        "rot": {"base": base, "dims": rot, "scaling": {"factor": factor} if factor else None}}}


def latent(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, scale=0.3, base=500.0, mlp=dense()):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                              "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def mamba(heads=6, vdim=20, state=12, groups=3, norm_groups=2, conv=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def config(layers, width=72, vocab=101, eps=1e-4, side=10):
    return {"architecture": "Bozasun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "token_side": {"dim": side}}


def weights(cfg, seed=0):
    """Random weights rounded to bfloat16, scaled so that every mechanism has a visible share of the result.  The last CODE
    dimensions of the residual belong to the embedding alone, and routers read mostly those, so that a choice of experts
    does not rest on the rounding of what the layers before it add."""
    rng = np.random.default_rng(seed)
    D, V, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    sd = {}

    def put(name, shape, std, mean=0.0):
        sd[name] = bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    def lin(name, o, i, gain=1.0):
        put(name, (o, i), gain / np.sqrt(i))

    def out(name, i, gain=1.0):
        lin(name, D, i, gain)
        sd[name][-CODE:] = 0

    put("embed", (V, D), 1.0)
    put("side.embed", (V, n * len(cfg["layers"])), 1.0)
    put("final.norm", (D,), 0.2, 1.0)
    lin("head", V, D)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        put(p + "norm1", (D,), 0.3, 1.0)
        if L["type"] == "attention":
            H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for t, w in (("q", H * d), ("k", G * d), ("v", G * vd)):
                lin(p + "mix." + t, w, D, 1.5)
                put(p + f"mix.{t}.b", (w,), 0.5)
            put(p + "mix.q.norm", (d,), 0.3, 1.2)
            put(p + "mix.k.norm", (d,), 0.3, 1.2)
            out(p + "mix.o", H * vd, 1.5)
            put(p + "mix.o.b", (D,), 0.3)
            sd[p + "mix.o.b"][-CODE:] = 0
        elif L["type"] == "latent_attention":
            H, d, r, vd, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            lin(p + "mix.q", H * (d + r), D, 1.5)
            lin(p + "mix.dkv", R + r, D, 1.5)
            put(p + "mix.dkv.norm", (R,), 0.2, 1.0)
            lin(p + "mix.uk", H * d, R)
            lin(p + "mix.uv", H * vd, R, 2.0)
            lin(p + "mix.g", H * vd, D, 2.0)
            out(p + "mix.o", H * vd, 2.0)
        else:
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            C = H * P + 2 * G * N
            lin(p + "mix.in", H * P + C + H, D, 1.5)
            put(p + "mix.conv", (C, m["conv"]), 0.6)
            put(p + "mix.conv.b", (C,), 0.3)
            put(p + "mix.dt_bias", (H,), 1.0, -1.5)
            put(p + "mix.A_log", (H,), 1.0, -1.0)
            put(p + "mix.D", (H,), 0.5, 0.7)
            put(p + "mix.norm", (H * P,), 0.2, 1.0)
            out(p + "mix.o", H * P)
        mlp = L["mlp"]
        if mlp:
            put(p + "norm2", (D,), 0.3, 1.0)
        if mlp and mlp["kind"] == "moe":
            r, E = mlp["router"], mlp["router"]["experts"] + mlp["router"]["identity"]
            put(p + "mlp.router", (E, D), 0.02)
            sd[p + "mlp.router"][:, -CODE:] = bf16((rng.standard_normal((E, CODE)) * 0.7).astype(np.float32))
            put(p + "mlp.correction", (E,), 0.06, -0.1)
            for e in range(r["experts"]):
                lin(p + f"mlp.e{e}.gate", mlp["expert"]["ff"], D, 2.0)
                lin(p + f"mlp.e{e}.up", mlp["expert"]["ff"], D, 2.0)
                out(p + f"mlp.e{e}.down", mlp["expert"]["ff"], 3.0)
        elif mlp:
            lin(p + "mlp.gate", mlp["ff"], D, 1.5)
            lin(p + "mlp.up", mlp["ff"], D, 1.5)
            out(p + "mlp.down", mlp["ff"], 1.5)
        lin(p + "side.gate", n, D, 1.5)
        out(p + "side.proj", n)
        put(p + "side.norm", (D,), 0.2, 0.6)
        sd[p + "side.norm"][-CODE:] = 0
    return sd


# sizes that are odd, unequal, or just past a kernel's tile; layers in several orders
MODELS = {
    "plain": config([attention(), mamba(mlp=moe()), latent(mlp=moe(experts=5, identity=1, top=2, groups=2, keep=1)), attention(chunk=64, mlp=None)]),
    "other_order": config([mamba(heads=4, groups=1, norm_groups=4, mlp=dense(40)), latent(heads=2, rot_dim=16, mlp=None), mamba(heads=2, vdim=33, groups=2, norm_groups=1, conv=2),
                           attention(heads=6, kv_heads=1, dim=40, vdim=64, rot=40, chunk=70, scale=0.15, softcap=None, factor=None, mlp=moe(identity=0, groups=1, keep=1, experts=6))],
                          width=96, vocab=130, side=16),
    "unaligned": config([latent(heads=5, dim=10, rot_dim=6, vdim=7, kv_rank=19, mlp=moe(experts=3, identity=3, top=4, groups=3, keep=3, ff=14)),
                         attention(heads=3, kv_heads=3, dim=10, vdim=6, rot=6, chunk=9, mlp=dense(22)), mamba(heads=3, vdim=5, state=7, groups=3, norm_groups=5, conv=5, mlp=dense(30))],
                        width=50, vocab=77, eps=1e-2, side=7),
    "ones": config([attention(heads=1, kv_heads=1, dim=16, vdim=16, rot=16, chunk=1, mlp=moe(experts=1, identity=1, top=1, groups=1, keep=1)),
                    mamba(heads=1, vdim=16, state=1, groups=1, norm_groups=1, conv=1, mlp=moe(experts=4, identity=0, top=1, groups=4, keep=1, ff=8)),
                    latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, mlp=None)], width=40, side=1),
}


def build(cfg, sd, dtype):
    import versenext_b200 as vn
    return vn.BozasunLM.from_state_dict(cfg, sd, dtype=dtype)


def close_calls(sd, cfg, toks):
    """Positions at which some router's choice is close, and the logits."""
    plain, found = OB.route, np.zeros(len(toks), bool)

    def watch(z, correction, top, groups, keep):
        chosen, weight = plain(z, correction, top, groups, keep)
        s = np.exp(z - z.max(axis=1, keepdims=True))
        s /= s.sum(axis=1, keepdims=True)
        c, E = s + correction, z.shape[1]
        best = c.reshape(len(z), groups, E // groups)
        at = best.argmax(axis=2)
        size = np.take_along_axis(s.reshape(best.shape), at[..., None], axis=2)[..., 0]      # what rounding moves: the scores
        best = best.max(axis=2)
        order = np.argsort(-best, axis=1, kind="stable")
        allowed = np.zeros((len(z), groups), bool)
        np.put_along_axis(allowed, order[:, :keep], True, axis=1)

        def near(values, sizes, k):
            if k >= values.shape[1]:
                return np.zeros(len(values), bool)
            o = np.argsort(-values, axis=1, kind="stable")
            v, w = np.take_along_axis(values, o, 1), np.take_along_axis(sizes, o, 1)
            return v[:, k - 1] - v[:, k] < 0.025 * (w[:, k - 1] + w[:, k]) + 5e-5
        c = np.where(np.repeat(allowed, E // groups, axis=1), c, -1e9)
        found[:] |= near(best, size, keep) | near(c, s, top)
        return chosen, weight
    OB.route = watch
    try:
        OB.forward(sd, cfg, toks)
    finally:
        OB.route = plain
    return found


def prompt(cfg, n, seed=1, sd=None):
    """Random tokens; with the weights, none whose experts depend on rounding."""
    rng = np.random.default_rng(seed)
    toks = rng.integers(0, cfg["vocab"], n)
    if sd is not None and any((L["mlp"] or {}).get("kind") == "moe" for L in cfg["layers"]):
        for _ in range(40):
            close = close_calls(sd, cfg, toks)
            if not close.any():
                return toks
            new = rng.integers(0, cfg["vocab"], n)
            if n > 9:                                        # half of them from those that are clear in this prompt
                new = np.where(rng.random(n) < 0.5, rng.choice(toks[~close], n), new)
            toks = np.where(close, new, toks)
        raise AssertionError("no prompt without close calls")
    return toks


class Expected(FC.Expected):
    oracle = OB


def greedy(sd, cfg, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(np.argmax(OB.forward(sd, cfg, toks)[-1])))
    return toks[-n:]
