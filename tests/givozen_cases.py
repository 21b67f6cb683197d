"""Small random models of the Givozen design for the tests: configurations, weights, prompts."""

import numpy as np

from oracle import givozen as OG
from oracle.fuzudra import bf16
import fuzudra_cases as FC
from fuzudra_cases import err  # noqa: F401

CODE = 8          # of the width: dimensions that only embeddings write and that routers read


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, top=3, ff=24, limit=1.2, shared_ff=40, shared_limit=2.1):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def rot(dims=16, base=1000.0, factor=3.0, low=1.0, high=4.0, original=200):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "low": low, "high": high, "original": original} if factor else None}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.3, rot=rot(), mlp=dense()):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}}


def config(layers, width=72, vocab=101, eps=1e-4, loop=None):
    loop = loop and dict(zip(("start", "stop", "times"), loop))
    return {"architecture": "Givozen", "layers": layers, "loop": loop, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg, seed=0):
    """Random weights rounded to bfloat16, scaled so that every mechanism has a visible share of the result.  The last CODE
    dimensions of the residual belong to embeddings alone, and routers read mostly those, so that a choice of experts does not
    rest on the rounding of what the layers before it add."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    sd = {}

    def put(name, shape, std, mean=0.0):
        sd[name] = bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    def lin(name, o, i, gain=1.0):
        put(name, (o, i), gain / np.sqrt(i))

    def behind(name, gain):
        put(name, (D,), 0.2 * gain, gain - 1.0)
        sd[name][-CODE:] = -1                             # the factor is 1 + weight

    put("embed", (V, D), 1.0)
    put("final.norm", (D,), 0.2)
    if cfg.get("loop"):
        put("loop.step", (cfg["loop"]["times"], D), 0.5)
        sd["loop.step"][:, -CODE:] = 0
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L["mlp"]
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(p + "norm1", (D,), 0.3)
        behind(p + "norm1b", 0.8)
        put(p + "norm2", (D,), 0.3)
        behind(p + "norm2b", 0.8)
        for t, w in (("q", H * d), ("k", G * d), ("v", G * vd)):
            lin(p + "mix." + t, w, D, 1.5)
            put(p + f"mix.{t}.b", (w,), 0.5)
        put(p + "mix.temp", (H,), 0.4, 1.0)
        lin(p + "mix.g", H, D, 2.0)
        lin(p + "mix.o", D, H * vd)
        if mlp and mlp["kind"] == "moe":
            E = mlp["router"]["experts"]
            put(p + "mlp.router", (E, D), 0.02)
            sd[p + "mlp.router"][:, -CODE:] = bf16((rng.standard_normal((E, CODE)) * 0.5).astype(np.float32))
            parts = [(f"mlp.e{e}.", mlp["expert"]["ff"]) for e in range(E)]
            if mlp.get("shared"):
                parts.append(("mlp.shared.", mlp["shared"]["ff"]))
                lin(p + "mlp.shared.sg", 1, D, 2.0)
            for part, f in parts:                         # gates and ups that often reach their limits
                lin(p + part + "gate", f, D, 2.5)
                lin(p + part + "up", f, D, 2.5)
                lin(p + part + "down", D, f, 2.0)
        elif mlp:
            lin(p + "mlp.up", mlp["ff"], D, 1.5)
            lin(p + "mlp.down", D, mlp["ff"])
            put(p + "mlp.act", (4,), 0.2, 0.6)
    return sd


A, E = attention, moe
# sizes that are odd, unequal, or just past a kernel's tile; blocks that run several times at every place
MODELS = {
    "plain": config([A(), A(mlp=E()), A(heads=2, kv_heads=1, mlp=E(experts=5, top=2, shared_ff=24, shared_limit=1.2)), A(mlp=None)], loop=(1, 3, 2)),
    "other_order": config([A(heads=6, kv_heads=1, dim=40, vdim=64, scale=0.15, rot=rot(40, 50.0, None), mlp=E(experts=6, top=1, ff=40)),
                           A(heads=3, kv_heads=3, dim=32, vdim=40, rot=rot(8, 300.0, 8.0, 0.5, 3.0, 60), mlp=None), A(mlp=dense(40))],
                          width=96, vocab=130, loop=(0, 2, 3)),
    "unaligned": config([A(heads=3, kv_heads=3, dim=10, vdim=6, rot=rot(6), mlp=E(experts=3, top=3, ff=14, shared_ff=11)),
                         A(heads=5, kv_heads=5, dim=10, vdim=7, rot=rot(2), mlp=dense(22)), A(heads=6, kv_heads=2, dim=9, vdim=5, rot=rot(4), mlp=dense(13))],
                        width=50, vocab=77, eps=1e-2, loop=(1, 2, 2)),
    "ones": config([A(heads=1, kv_heads=1, dim=16, vdim=16, rot=rot(16), mlp=E(experts=1, top=1, ff=8, shared_ff=8)),
                    A(heads=1, kv_heads=1, dim=2, vdim=1, rot=None, mlp=E(experts=4, top=4, ff=1, shared_ff=None)), A(mlp=dense(1))], width=40, loop=(0, 3, 1)),
    "no_loop": config([A(rot=rot(24, 2e5, 6.0, 1.5, 5.0, 700), mlp=E(top=2)), A(mlp=dense())]),
}


def build(cfg, sd, dtype):
    import versenext_b200 as vn
    return vn.GivozenLM.from_state_dict(cfg, sd, dtype=dtype)


def close_calls(sd, cfg, toks):
    """Positions at which some router's choice is close."""
    plain, found = OG.route, np.zeros(len(toks), bool)

    def watch(z, top):
        if top < z.shape[1]:
            v = -np.sort(-OG.sigmoid(z), axis=1)
            found[:] |= v[:, top - 1] - v[:, top] < 0.02 * v[:, top - 1] * (1 - v[:, top]) + 1e-3
        return plain(z, top)
    OG.route = watch
    try:
        OG.forward(sd, cfg, toks)
    finally:
        OG.route = plain
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
    oracle = OG


def greedy(sd, cfg, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(np.argmax(OG.forward(sd, cfg, toks)[-1])))
    return toks[-n:]
