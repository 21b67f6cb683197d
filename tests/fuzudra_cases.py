"""Small random models of the Fuzudra design for the tests: configurations, weights, prompts."""

import numpy as np

from oracle import fuzudra as OF


def latent(heads=3, dim=24, vdim=16, kv_rank=40, window=37, scale=0.3, ff=48):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "mask": {"size": window}}}


def mamba(inner=80, state=10, dt_rank=5, conv=4, ff=0):
    return {"type": "mamba1", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def delta(heads=4, kv_heads=2, dim=32, vdim=20, conv=3, ff=0):
    return {"type": "channel_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, width=72, vocab=101, eps=1e-4, loop=None):
    return {"architecture": "Fuzudra", "layers": layers, "loop": loop, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg, seed=0, rank_a=9, rank_g=17):
    """Random weights rounded to bfloat16, scaled so that every mechanism has a visible share of the result."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    sd = {}

    def put(name, shape, std, mean=0.0):
        sd[name] = OF.bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    def lin(name, o, i, gain=1.0):
        put(name, (o, i), gain / np.sqrt(i))

    put("embed", (V, D), 1.0)
    put("final.norm", (D,), 0.2)
    lin("head", V, D)
    if cfg.get("loop"):
        lin("loop.in", D, 2 * D)
        put("loop.step", (cfg["loop"]["times"], D), 0.5)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        put(p + "norm1", (D,), 0.3)
        if L["type"] == "latent_attention":
            H, d, vd, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            lin(p + "mix.q", H * d, D, 1.5)
            lin(p + "mix.dkv", R, D)
            put(p + "mix.dkv.norm", (R,), 0.2, 1.0)
            lin(p + "mix.uk", H * d, R)
            lin(p + "mix.uv", H * vd, R, 2.0)
            put(p + "mix.sink", (H,), 1.0, 1.5)
            lin(p + "mix.g", H, D, 2.0)
            lin(p + "mix.o", D, H * vd, 1.5)
        elif L["type"] == "mamba1":
            n, r, N = m["inner"], m["dt_rank"], m["state"]
            lin(p + "mix.in", 2 * n, D)
            put(p + "mix.conv", (n, m["conv"]), 0.5)
            put(p + "mix.conv.b", (n,), 0.3)
            lin(p + "mix.x", r + 2 * N, n)
            lin(p + "mix.dt", n, r)
            put(p + "mix.dt.b", (n,), 1.0, -2.5)
            put(p + "mix.A_log", (n, N), 1.2, -1.0)
            put(p + "mix.D", (n,), 0.5, 1.0)
            lin(p + "mix.o", D, n)
        else:
            H, K, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for t, w in (("q", K * d), ("k", K * d), ("v", H * vd)):
                lin(p + "mix." + t, w, D, 2.0)
                put(p + f"mix.{t}.conv", (w, m["conv"]), 0.6)
            lin(p + "mix.b", H, D)
            put(p + "mix.A_log", (H,), 0.8, -1.5)
            put(p + "mix.norm", (vd,), 0.2, 1.0)
            lin(p + "mix.a1", rank_a, D)
            lin(p + "mix.a2", H * d, rank_a)
            put(p + "mix.dt_bias", (H * d,), 1.0, -1.5)
            lin(p + "mix.g1", rank_g, D)
            lin(p + "mix.g2", H * vd, rank_g, 2.0)
            lin(p + "mix.o", D, H * vd)
        if L["mlp"]:
            put(p + "norm2", (D,), 0.3)
            lin(p + "mlp.gate", L["mlp"]["ff"], D, 2.0)
            lin(p + "mlp.up", L["mlp"]["ff"], D)
            lin(p + "mlp.down", D, L["mlp"]["ff"])
    return sd


# sizes that are odd, unequal, or just past a kernel's tile; layers in several orders; loops inside, at the ends, absent
MODELS = {
    "plain": config([mamba(), latent(), delta()]),
    "loop_inside": config([delta(ff=40), latent(window=5), mamba(state=16), latent(heads=2, kv_rank=33, window=64)], width=64,
                          loop={"start": 1, "stop": 3, "times": 3}),
    "loop_all": config([latent(window=70, ff=0), delta(heads=2, kv_heads=2, dim=48, vdim=48, conv=2)], width=96, vocab=130,
                       loop={"start": 0, "stop": 2, "times": 2}),
    "loop_once": config([delta(heads=6, kv_heads=1, dim=20, vdim=64, conv=5), mamba(inner=72, state=3, dt_rank=1, conv=2, ff=24),
                         latent(heads=1, dim=8, vdim=40, kv_rank=16, window=1)], width=40, eps=1e-2,
                        loop={"start": 2, "stop": 3, "times": 1}),
    "unaligned": config([latent(heads=5, dim=10, vdim=6, kv_rank=18, window=9, ff=30), mamba(inner=36, state=7, dt_rank=3, conv=3),
                         delta(heads=3, kv_heads=3, dim=14, vdim=10, conv=4)], width=50, vocab=77),
}


def build(cfg, sd, dtype):
    import versenext_b200 as vn
    return vn.FuzudraLM.from_state_dict(cfg, sd, dtype=dtype)


def err(got, want):
    """Root mean square of the difference over that of the expected values' spread, the worst row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.max(np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.std(want)))


class Expected:
    """Logits of one sequence and what rounding costs there: fp32 a fixed fraction of their spread; bf16 a multiple of the
    error of the restatement itself when it stores what the device stores in 16 bits."""

    oracle = OF

    def __init__(self, sd, cfg, toks):
        self.runs = []
        self.logits = self.oracle.forward(sd, cfg, toks, self.runs)
        rough = []
        with OF.rounded():
            r = self.oracle.forward(sd, cfg, toks, rough)
        self.tol = {"f32": 3e-5, "bf16": 4 * max(err(r, self.logits), 2e-3)}
        self.run_tol = [{"f32": 3e-5, "bf16": 4 * max(err(a, b), 2e-3)} for a, b in zip(rough, self.runs)]
        self.spread = np.std(self.logits)

    def check(self, got, dtype, rows=slice(None), what=""):
        got, want = np.asarray(got, np.float64), self.logits[rows]
        assert got.shape == want.shape, what
        worst = float(np.max(np.sqrt(np.mean((got - want) ** 2, axis=-1)))) / self.spread
        assert worst < self.tol[dtype], (what, worst, self.tol[dtype])


TOL = {"f32": 3e-5}


def prompt(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)
