"""Seeded synthetic weights for benchmarks and smoke runs.

Random N(0, init_std) weights of the VerseNexLM architecture with the reference's residual scaling
(verse_nex/cometspark.py:455-481: attn.proj and SwiGLU w_down times 1/sqrt(2 n_layer)), unit norm gains
and zero gate logits.  Tensors are produced one at a time so that a 1.1 B-parameter model never sits on
the host in full.
"""

from __future__ import annotations

from typing import Iterator, Tuple

import numpy as np


def mate_kwargs(**over) -> dict:
    """CometSparkV05 factory defaults (spark/src/base_model.py:760-786)."""
    kw = dict(vocab_size=248320, dim=1024, n_layer=20, n_head=16, n_kv_head=8,
              layer_pattern=["mod" if i % 4 == 0 else "trisparse" for i in range(20)],
              window_size=1024, num_global_tokens=128, use_alibi=False, use_rope=True, max_seq_len=4096,
              num_dense_parts=4, num_experts_per_part=4, top_k=2, tie_weights=True, embedding_scale=True)
    kw.update(over)
    return kw


def draft_kwargs(**over) -> dict:
    """The small draft of the full speculative-decode workload: 2 layers, dim 256, 4 heads, all TriSparse."""
    kw = dict(vocab_size=248320, dim=256, n_layer=2, n_head=4, max_seq_len=2048)
    kw.update(over)
    return kw


def _shapes(kw: dict) -> Iterator[Tuple[str, tuple]]:
    D, H = kw["dim"], kw["n_head"]
    n_kv = kw.get("n_kv_head") or H
    hd = D // H
    pattern = kw.get("layer_pattern") or ["trisparse"] * kw["n_layer"]
    mult = kw.get("mlp_hidden_multiple", 4)
    hidden = int((mult * D * 2 / 3 + 63) // 64) * 64
    eh = kw.get("expert_hidden") or max(int(D * 8 / 3 / 64) * 64, 64)
    P, E = kw.get("num_dense_parts", 5), kw.get("num_experts_per_part", 8)
    yield "tok_emb.weight", (kw["vocab_size"], D)
    yield "norm.weight", (D,)
    if not kw.get("tie_weights", True):
        yield "head.weight", (kw["vocab_size"], D)
    for i, kind in enumerate(pattern):
        p = f"blocks.{i}."
        yield p + "norm1.weight", (D,)
        yield p + "norm2.weight", (D,)
        n_g = kw.get("num_global_tokens", 64)
        if kind in ("vda", "dsa", "kda", "gmla"):
            # the modules of verse_nex/delta_attention.py: a vda layer holds one of each under its own prefix
            lat = kw.get("latent_dim") or n_kv * hd
            for sub in (("dsa", "kda", "gmla") if kind == "vda" else (kind,)):
                q = p + "attn." + (sub + "." if kind == "vda" else "")
                yield q + "wq.weight", (H * hd, D)
                if sub == "gmla":
                    yield q + "w_kv_down.weight", (lat, D)
                    yield q + "w_k_up.weight", (n_kv * hd, lat)
                    yield q + "w_v_up.weight", (n_kv * hd, lat)
                else:
                    yield q + "wk.weight", (n_kv * hd, D)
                    yield q + "wv.weight", (n_kv * hd, D)
                if sub == "dsa":
                    yield q + "global_tokens.weight", (n_g, D)
                if sub != "kda":
                    yield q + "head_gate_logits", (H,)
            if kind == "vda":
                yield p + "attn.gate_logits", (3,)
            yield p + "attn.proj.weight", (D, H * hd)
        else:
            yield p + "attn.gate_logits", (3,)
            yield p + "attn.wq.weight", (H * hd, D)
            yield p + "attn.wk.weight", (n_kv * hd, D)
            yield p + "attn.wv.weight", (n_kv * hd, D)
            yield p + "attn.proj.weight", (D, H * hd)
            yield p + "attn.global_tokens.weight", (n_g, D)
        if kind == "mod":
            yield p + "ffn.part_router.gate.weight", (P, D)
            for q in range(P):
                yield p + f"ffn.parts.{q}.router.gate.weight", (E, D)
                for e in range(E):
                    pe = p + f"ffn.parts.{q}.experts.{e}."
                    yield pe + "w_gate.weight", (eh, D)
                    yield pe + "w_up.weight", (eh, D)
                    yield pe + "w_down.weight", (D, eh)
        else:
            yield p + "ffn.w_gate.weight", (hidden, D)
            yield p + "ffn.w_up.weight", (hidden, D)
            yield p + "ffn.w_down.weight", (D, hidden)


def random_tensors(kw: dict, seed: int, init_std: float = 0.02) -> Iterator[Tuple[str, np.ndarray]]:
    rs = np.float32(1.0 / ((2 * kw["n_layer"]) ** 0.5))
    for j, (name, shape) in enumerate(_shapes(kw)):
        if name.endswith(("norm1.weight", "norm2.weight")) or name == "norm.weight":
            yield name, np.ones(shape, dtype=np.float32)
        elif name.endswith("gate_logits"):
            yield name, np.zeros(shape, dtype=np.float32)
        else:
            rng = np.random.default_rng([seed, j])
            w = rng.standard_normal(shape, dtype=np.float32) * np.float32(init_std)
            if name.endswith("attn.proj.weight") or name.endswith("ffn.w_down.weight"):
                w *= rs
            yield name, w


def load_random(model, kw: dict, seed: int, init_std: float = 0.02):
    """Fill a device model tensor by tensor and finalise it."""
    for name, w in random_tensors(kw, seed, init_std):
        model.load_tensor(name, w)
    model.finalize()
    return model


def param_count(kw: dict) -> int:
    return int(sum(int(np.prod(s)) for _, s in _shapes(kw)))


# ---- composed models (fuzudra.py): layers of the sizes a real model of that width would have ---------------------------
def fuzudra_config(width: int, vocab: int = 32000, n_layer: int = 4, loop_times: int = 0) -> dict:
    """config.json contents: latent attention, selective scan and two delta rule layers in turn, a feed-forward behind
    each (as wide as VerseNexLM's), heads of 128 (64 below width 2048), a window of 1024."""
    hd = 128 if width >= 2048 else 64
    heads, ff = width // hd, int((4 * width * 2 / 3 + 63) // 64) * 64
    mlp = {"kind": "dense", "ff": ff}
    kinds = [{"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": hd, "vdim": hd, "kv_rank": width // 4,
              "scale": hd ** -0.5, "mask": {"size": 1024}}},
             {"type": "mamba1", "mlp": mlp, "mixer": {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}},
             {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": heads, "dim": hd, "vdim": hd, "conv": 4}}]
    layers = [kinds[(0, 1, 2, 2)[i % 4]] for i in range(n_layer)]
    return {"architecture": "Fuzudra", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers,
            "loop": {"start": 0, "stop": n_layer, "times": loop_times} if loop_times else None}


def fuzudra_shapes(cfg: dict) -> dict:
    """Tensor name -> shape; the ranks of the two low-rank factors are a head's width."""
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    if cfg.get("loop"):
        s["loop.in"], s["loop.step"] = (D, 2 * D), (cfg["loop"]["times"], D)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        t = {"norm1": (D,)}
        if L["type"] == "latent_attention":
            H, d, v, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            t.update({"mix.q": (H * d, D), "mix.dkv": (R, D), "mix.dkv.norm": (R,), "mix.uk": (H * d, R), "mix.uv": (H * v, R),
                      "mix.sink": (H,), "mix.g": (H, D), "mix.o": (D, H * v)})
        elif L["type"] == "mamba1":
            n, r, N = m["inner"], m["dt_rank"], m["state"]
            t.update({"mix.in": (2 * n, D), "mix.conv": (n, m["conv"]), "mix.conv.b": (n,), "mix.x": (r + 2 * N, n),
                      "mix.dt": (n, r), "mix.dt.b": (n,), "mix.A_log": (n, N), "mix.D": (n,), "mix.o": (D, n)})
        else:
            H, K, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t.update({"mix.q": (K * d, D), "mix.q.conv": (K * d, m["conv"]), "mix.k": (K * d, D), "mix.k.conv": (K * d, m["conv"]),
                      "mix.v": (H * v, D), "mix.v.conv": (H * v, m["conv"]), "mix.b": (H, D), "mix.A_log": (H,),
                      "mix.norm": (v,), "mix.a1": (d, D), "mix.a2": (H * d, d), "mix.dt_bias": (H * d,), "mix.g1": (v, D),
                      "mix.g2": (H * v, v), "mix.o": (D, H * v)})
        if L["mlp"]:
            t.update({"norm2": (D,), "mlp.gate": (L["mlp"]["ff"], D), "mlp.up": (L["mlp"]["ff"], D), "mlp.down": (D, L["mlp"]["ff"])})
        s.update({p + n: x for n, x in t.items()})
    return s


def musutar_config(width: int, vocab: int = 32000, n_layer: int = 4) -> dict:
    """config.json contents: lightning attention and sliding-window attention in turn, every second attention layer with
    the keys and values of the one before it; four residual streams; heads of 128 (64 below width 2048), four query heads
    per key head, a window of 1024; feed-forwards with as many weights as VerseNexLM's gated ones."""
    hd = 128 if width >= 2048 else 64
    heads = width // hd
    mlp = {"kind": "dense", "ff": 4 * width}
    decay = [float(1 - 2.0 ** (-1 - 7.0 * i / max(heads - 1, 1))) for i in range(heads)]
    layers = []
    for i in range(n_layer):
        if i % 2 == 0:
            layers.append({"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": hd, "vdim": hd, "decay": decay}})
            continue
        m = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": hd, "vdim": hd, "conv": 4, "scale": hd ** -0.5, "mask": {"size": 1024},
             "rot": {"base": 10000.0, "dims": hd, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        if i % 4 == 3:
            m["kv_from"] = i - 2
        layers.append({"type": "attention", "mlp": mlp, "mixer": m})
    return {"architecture": "Musutar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "streams": 4, "canon": {"taps": 4}, "layers": layers}


def musutar_shapes(cfg: dict) -> dict:
    """Tensor name -> shape."""
    D, V, n = cfg["width"], cfg["vocab"], cfg["streams"]
    s = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    for i, L in enumerate(cfg["layers"]):
        m = L["mixer"]
        H, d, v = m["heads"], m["dim"], m["vdim"]
        t = {"canon1": (D, cfg["canon"]["taps"]), "mix.q": (H * d, D), "mix.g": (H * v, D), "mix.o": (D, H * v)}
        if L["type"] == "attention":
            G = m["kv_heads"]
            t["mix.q.conv"] = (H * d, m["conv"])
            if m.get("kv_from") is None:
                t.update({"mix.k": (G * d, D), "mix.v": (G * v, D), "mix.k.conv": (G * d, m["conv"]), "mix.v.conv": (G * v, m["conv"])})
        else:
            t.update({"mix.k": (H * d, D), "mix.v": (H * v, D), "mix.norm": (H * v,)})
        for q in (1, 2) if L["mlp"] else (1,):
            t.update({f"norm{q}": (D,), f"hc{q}.in": (n,), f"hc{q}.out": (n,), f"hc{q}.mix": (n, n), f"rg{q}": (D, D), f"rg{q}.b": (D,)})
        if L["mlp"]:
            t.update({"mlp.up": (L["mlp"]["ff"], D), "mlp.down": (D, L["mlp"]["ff"])})
        s.update({f"l{i}.{k}": x for k, x in t.items()})
    return s


def bozasun_config(width: int, vocab: int = 32000, n_layer: int = 4) -> dict:
    """config.json contents: chunked attention with a dense feed-forward, Mamba-2 and latent attention with mixtures, Mamba-2
    with a dense feed-forward in turn; heads of 128 (64 below width 2048), four query heads per key head, chunks of 2048, a
    state of 128 per channel, feed-forwards as wide as VerseNexLM's, mixtures of experts a quarter as wide of which a token
    uses about as many."""
    hd = 128 if width >= 2048 else 64
    heads, ff = width // hd, int((4 * width * 2 / 3 + 63) // 64) * 64
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": (ff // 4 + 63) // 64 * 64},
           "router": {"experts": 24, "identity": 8, "top": 6, "groups": {"count": 4, "keep": 3}}}
    rot = {"base": 10000.0, "dims": hd, "scaling": {"factor": 2.0}}
    attention = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": hd, "vdim": hd, "scale": hd ** -0.5, "softcap": 30.0, "mask": {"size": 2048}, "rot": rot}
    latent = {"heads": heads, "dim": hd, "rot_dim": hd // 2, "vdim": hd, "kv_rank": width // 4, "scale": (1.5 * hd) ** -0.5,
              "rot": {"base": 10000.0, "dims": hd // 2}}
    mamba = {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4}
    kinds = [{"type": "attention", "mixer": attention, "mlp": dense}, {"type": "mamba2", "mixer": mamba, "mlp": moe},
             {"type": "latent_attention", "mixer": latent, "mlp": moe}, {"type": "mamba2", "mixer": mamba, "mlp": dense}]
    return {"architecture": "Bozasun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "token_side": {"dim": width // 16},
            "layers": [kinds[i % 4] for i in range(n_layer)]}


def bozasun_shapes(cfg: dict) -> dict:
    """Tensor name -> shape."""
    D, V, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    s = {"embed": (V, D), "side.embed": (V, n * len(cfg["layers"])), "head": (V, D), "final.norm": (D,)}
    for i, L in enumerate(cfg["layers"]):
        m, mlp = L["mixer"], L.get("mlp")
        t = {"norm1": (D,), "side.gate": (n, D), "side.proj": (D, n), "side.norm": (D,)}
        H, v = m["heads"], m["vdim"]
        if L["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            for part, w in (("q", H * d), ("k", G * d), ("v", G * v)):
                t.update({f"mix.{part}": (w, D), f"mix.{part}.b": (w,)})
            t.update({"mix.q.norm": (d,), "mix.k.norm": (d,), "mix.o": (D, H * v), "mix.o.b": (D,)})
        elif L["type"] == "latent_attention":
            d, r, R = m["dim"], m["rot_dim"], m["kv_rank"]
            t.update({"mix.q": (H * (d + r), D), "mix.dkv": (R + r, D), "mix.dkv.norm": (R,), "mix.uk": (H * d, R), "mix.uv": (H * v, R),
                      "mix.g": (H * v, D), "mix.o": (D, H * v)})
        else:
            C = H * v + 2 * m["groups"] * m["state"]
            t.update({"mix.in": (H * v + C + H, D), "mix.conv": (C, m["conv"]), "mix.conv.b": (C,), "mix.dt_bias": (H,), "mix.A_log": (H,),
                      "mix.D": (H,), "mix.norm": (H * v,), "mix.o": (D, H * v)})
        parts = [("mlp.", mlp["ff"])] if mlp and mlp["kind"] == "dense" else []
        if mlp:
            t["norm2"] = (D,)
            if mlp["kind"] == "moe":
                r = mlp["router"]
                t.update({"mlp.router": (r["experts"] + r["identity"], D), "mlp.correction": (r["experts"] + r["identity"],)})
                parts = [(f"mlp.e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
        for p, f in parts:
            t.update({p + "gate": (f, D), p + "up": (f, D), p + "down": (D, f)})
        s.update({f"l{i}.{k}": x for k, x in t.items()})
    return s


def givozen_config(width: int, vocab: int = 32000, n_run: int = 4) -> dict:
    """config.json contents: `n_run` layer runs out of n_run - 1 layers, PolyNorm feed-forwards and mixtures, the mixture in the
    middle run twice; heads of 128 (64 below width 2048), four query heads per key head; feed-forwards with as many weights as
    VerseNexLM's gated ones, experts and the one that serves every token a quarter as wide, of which a token uses three."""
    hd = 128 if width >= 2048 else 64
    heads, ff = width // hd, int((4 * width * 2 / 3 + 63) // 64) * 64
    part = {"ff": (ff // 4 + 63) // 64 * 64, "limit": 7.0}
    dense, moe = {"kind": "dense", "ff": 4 * width}, {"kind": "moe", "expert": part, "shared": part, "router": {"experts": 24, "top": 3}}
    rot = {"base": 500000.0, "dims": hd, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": hd, "vdim": hd, "scale": hd ** -0.5, "rot": rot}
    return {"architecture": "Givozen", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "loop": {"start": 1, "stop": 2, "times": 2},
            "layers": [{"type": "attention", "mixer": mixer, "mlp": moe if i % 2 else dense} for i in range(n_run - 1)]}


def givozen_shapes(cfg: dict) -> dict:
    """Tensor name -> shape."""
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "final.norm": (D,)}
    if cfg.get("loop"):
        s["loop.step"] = (cfg["loop"]["times"], D)
    for i, L in enumerate(cfg["layers"]):
        m, mlp = L["mixer"], L.get("mlp")
        H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        t = {"norm1": (D,), "norm1b": (D,), "mix.temp": (H,), "mix.g": (H, D), "mix.o": (D, H * v)}
        for part, w in (("q", H * d), ("k", G * d), ("v", G * v)):
            t.update({f"mix.{part}": (w, D), f"mix.{part}.b": (w,)})
        if mlp:
            t.update({"norm2": (D,), "norm2b": (D,)})
        if mlp and mlp["kind"] == "dense":
            t.update({"mlp.up": (mlp["ff"], D), "mlp.down": (D, mlp["ff"]), "mlp.act": (4,)})
        elif mlp:
            parts = [(f"mlp.e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            t["mlp.router"] = (mlp["router"]["experts"], D)
            if mlp.get("shared"):
                parts.append(("mlp.shared.", mlp["shared"]["ff"]))
                t["mlp.shared.sg"] = (1, D)
            for p, f in parts:
                t.update({p + "gate": (f, D), p + "up": (f, D), p + "down": (D, f)})
        s.update({f"l{i}.{k}": x for k, x in t.items()})
    return s


def random_givozen(cfg: dict, seed: int = 0, **kw):
    """A GivozenLM with seeded random weights, tensor by tensor."""
    from .givozen import GivozenLM
    return _random_design(GivozenLM, cfg, givozen_shapes(cfg), seed, **kw)


def random_bozasun(cfg: dict, seed: int = 0, **kw):
    """A BozasunLM with seeded random weights, tensor by tensor."""
    from .bozasun import BozasunLM
    return _random_design(BozasunLM, cfg, bozasun_shapes(cfg), seed, **kw)


def random_fuzudra(cfg: dict, seed: int = 0, **kw):
    """A FuzudraLM with seeded random weights, tensor by tensor."""
    from .fuzudra import FuzudraLM
    return _random_design(FuzudraLM, cfg, fuzudra_shapes(cfg), seed, **kw)


def random_musutar(cfg: dict, seed: int = 0, **kw):
    """A MusutarLM with seeded random weights, tensor by tensor."""
    from .musutar import MusutarLM
    return _random_design(MusutarLM, cfg, musutar_shapes(cfg), seed, **kw)


# (name's end, standard deviation, mean) of the tensors that are not plain linear weights or norms around zero
_SPECIAL = (("mix.A_log", 1.0, -1.0), ("mix.dt_bias", 1.0, -2.0), ("mix.dt.b", 1.0, -3.0), ("mix.D", 0.1, 1.0), ("mix.sink", 1.0, 0.0),
            (".conv", 0.4, 0.0), ("canon1", 0.3, 0.0), ("mix.norm", 0.1, 1.0), ("dkv.norm", 0.1, 1.0), ("hc1.in", 0.1, 0.25), ("hc2.in", 0.1, 0.25),
            ("hc1.out", 0.1, 1.0), ("hc2.out", 0.1, 1.0), ("mlp.correction", 0.005, 0.0), ("mix.temp", 0.1, 1.0), ("mlp.act", 0.1, 0.5))


def _random_design(cls, cfg: dict, shapes: dict, seed: int, **kw):
    model = cls(cfg, shapes, **kw)
    rng = np.random.default_rng(seed)
    for name, shape in shapes.items():
        std, mean = (0.02, 0.0) if len(shape) == 2 else (0.1, 0.0)
        for end, s, m in _SPECIAL:
            if name.endswith(end):
                std, mean = s, m
        if cfg["architecture"] in ("Bozasun", "Musutar") and name.split(".")[-1] in ("norm", "norm1", "norm2"):
            mean = 1.0                                     # plain weights
        w = mean + std * rng.standard_normal(shape, dtype=np.float32)
        model.load_tensor(name, w + np.eye(shape[0], dtype=np.float32) if name.endswith(".mix") else w)
    model.finalize()
    return model
