"""The Bozasun design: config.json and checkpoint of such a model -> a `ComposedLM`.

Layers of grouped-query attention (chunked, biases, a norm of every query and key head, interleaved rotary positions with
linear scaling, capped scores), latent attention with a rotated part and a gate on every output element, or Mamba-2, each with
an optional gated feed-forward or a mixture of experts (grouped choice with a correction, identity experts), and behind every
layer an input of its own for every token; RMS norms with plain weights.  Weights are bfloat16 in `model.safetensors`, named
as the library takes them.
"""

from __future__ import annotations

from typing import Dict, Tuple

from .composed import DesignLM


def _rope(rot):
    if not rot:
        return None
    factor = (rot.get("scaling") or {}).get("factor")
    return {"dims": int(rot["dims"]), "base": float(rot["base"]), "interleaved": True,
            "scaling": {"kind": "linear", "factor": float(factor)} if factor else None}


def _attention(m: dict) -> dict:
    return {"mixer": "attention", **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}, "bias": True, "qk_norm": True,
            "rope": _rope(m.get("rot")), "chunk": int((m.get("mask") or {}).get("size") or 0), "softcap": float(m.get("softcap") or 0)}


def _latent_attention(m: dict) -> dict:
    return {"mixer": "latent_attention", **{k: m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale")}, "sink": False,
            "output_gate": "element", "rope": _rope(m.get("rot"))}


def _mamba2(m: dict) -> dict:
    return {"mixer": "mamba2", **{k: int(m[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")}}


_MIXERS = {"attention": _attention, "latent_attention": _latent_attention, "mamba2": _mamba2}


def _mlp(mlp: dict, i: int) -> dict:
    if mlp.get("kind") == "dense":
        return {"mlp_hidden": int(mlp["ff"]), "mlp_act": "silu"}
    if mlp.get("kind") != "moe":
        raise ValueError(f"layer {i}: feed-forward {mlp.get('kind')!r} is not part of this design")
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return {"mlp_hidden": int(mlp["expert"]["ff"]), "mlp_act": "silu",
            "experts": {"count": int(r["experts"]), "identity": int(r.get("identity") or 0), "top": int(r["top"]),
                        "groups": int(groups["count"]), "keep": int(groups["keep"]), "correction": True}}


def composed_config(config: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
    """The library's configuration of a Bozasun config.json."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        kind = entry["type"]
        if kind not in _MIXERS:
            raise ValueError(f"layer {i}: mixer {kind!r} is not part of this design {tuple(_MIXERS)}")
        out = _MIXERS[kind](entry["mixer"])
        if entry.get("mlp") is not None:
            out.update(_mlp(entry["mlp"], i))
        layers.append(out)
    return {"vocab_size": int(config["vocab"]), "dim": int(config["width"]), "norm_eps": float(config["norm"]["eps"]),
            "norm_weight": "plain", "token_side": int((config.get("token_side") or {}).get("dim") or 0), "layers": layers}


class BozasunLM(DesignLM):
    ARCHITECTURE = "Bozasun"
    composed_config = staticmethod(composed_config)
