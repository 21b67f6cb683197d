"""Small random models of the Musutar design for the tests: configurations, weights, prompts."""

import numpy as np

from oracle import musutar as OM
from oracle.fuzudra import bf16
import fuzudra_cases as FC
from fuzudra_cases import err, prompt  # noqa: F401


def yarn(factor=3.0, original=60, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, window=37, scale=0.25, conv=3, rot=16, base=1000.0, scaling=yarn(), ff=48, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "mask": {"size": window},
         "rot": {"base": base, "dims": rot, "scaling": scaling}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def lightning(heads=3, dim=20, vdim=28, ff=40, decay=None):
    decay = decay if decay is not None else [float(1 - 0.6 ** (1.3 * i + 0.5)) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=101, eps=1e-4, streams=3, taps=3):
    return {"architecture": "Musutar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams,
            "canon": {"taps": taps}}


def weights(cfg, seed=0):
    """Random weights rounded to bfloat16, scaled so that every mechanism has a visible share of the result."""
    rng = np.random.default_rng(seed)
    D, V, ns = cfg["width"], cfg["vocab"], cfg["streams"]
    sd = {}

    def put(name, shape, std, mean=0.0):
        sd[name] = bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    def lin(name, o, i, gain=1.0):
        put(name, (o, i), gain / np.sqrt(i))

    put("embed", (V, D), 1.0)
    put("final.norm", (D,), 0.2, 1.0)
    lin("head", V, D)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for q in (1, 2) if L["mlp"] else (1,):
            put(p + f"norm{q}", (D,), 0.3, 1.0)
            put(p + f"hc{q}.in", (ns,), 0.4, 0.5)
            put(p + f"hc{q}.out", (ns,), 0.3, 0.5)
            sd[p + f"hc{q}.mix"] = bf16((np.eye(ns) * 0.9 + 0.1 * rng.standard_normal((ns, ns))).astype(np.float32))
            lin(p + f"rg{q}", D, D, 1.5)
            put(p + f"rg{q}.b", (D,), 0.5, 0.5)
        put(p + "canon1", (D, cfg["canon"]["taps"]), 0.4)
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            parts = [("q", H * d, 1.5)] + ([("k", m["kv_heads"] * d, 1.5), ("v", m["kv_heads"] * vd, 2.0)] if m.get("kv_from") is None else [])
            for t, w, gain in parts:
                lin(p + "mix." + t, w, D, gain)
                put(p + f"mix.{t}.conv", (w, m["conv"]), 0.6)
        else:
            for t, w in (("q", H * d), ("k", H * d), ("v", H * vd)):
                lin(p + "mix." + t, w, D, 2.0)
            put(p + "mix.norm", (H * vd,), 0.2, 1.0)
        lin(p + "mix.g", H * vd, D, 2.0)
        lin(p + "mix.o", D, H * vd, 2.0)
        if L["mlp"]:
            lin(p + "mlp.up", L["mlp"]["ff"], D, 1.5)
            lin(p + "mlp.down", D, L["mlp"]["ff"], 1.5)
    return sd


# sizes that are odd, unequal, or just past a kernel's tile; layers in several orders; one to five streams
MODELS = {
    "plain": config([lightning(), attention(), attention(kv_from=1, window=9, ff=0, scale=0.4, heads=4), lightning(heads=2, dim=32, vdim=16, ff=0)]),
    "shared": config([attention(window=5, ff=0), attention(window=70, kv_from=0), lightning(), attention(kv_from=0, window=64)], width=64,
                     streams=2, taps=4),
    "one_stream": config([attention(heads=6, kv_heads=1, dim=40, vdim=64, rot=40, conv=2, window=33, scaling=yarn(1.5, 500, 2.0, 0.5)),
                          lightning(heads=1, dim=100, vdim=72)], width=96, vocab=130, streams=1, taps=2),
    "unaligned": config([lightning(heads=3, dim=14, vdim=10, ff=30), attention(heads=3, kv_heads=3, dim=10, vdim=6, rot=6, conv=4, window=9, ff=22),
                         attention(heads=3, kv_heads=3, dim=10, vdim=6, rot=6, conv=5, window=2, ff=0, kv_from=1)], width=50, vocab=77, eps=1e-2, taps=6),
    "one_tap": config([attention(heads=2, kv_heads=2, dim=16, vdim=16, rot=8, conv=1, window=1), lightning(heads=2, dim=8, vdim=8, decay=[0.999, 0.3])],
                      width=40, streams=5, taps=1),
}


def build(cfg, sd, dtype):
    import versenext_b200 as vn
    return vn.MusutarLM.from_state_dict(cfg, sd, dtype=dtype)


class Expected(FC.Expected):
    oracle = OM


def greedy(sd, cfg, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(np.argmax(OM.forward(sd, cfg, toks)[-1])))
    return toks[-n:]
