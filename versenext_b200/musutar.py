"""The Musutar design: config.json and checkpoint of such a model -> a `ComposedLM`.

Layers of grouped-query attention (sliding window, rotary positions with YaRN scaling, short convolutions on q, k and v, an
output gate, optionally another layer's keys and values) or lightning attention, each with an optional squared-relu
feed-forward; layer norms, several residual streams, a gate on every sublayer's result, a short convolution on every mixer's
input.  Weights are bfloat16 in `model.safetensors`, named as the library takes them.
"""

from __future__ import annotations

from typing import Dict, Tuple

from .composed import DesignLM


def _attention(m: dict) -> dict:
    out = {"mixer": "attention", **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}, "output_gate": True}
    out["window"] = int((m.get("mask") or {}).get("size") or 0)
    for src, dst in (("conv", "conv"), ("rot", "rope"), ("kv_from", "kv_from")):
        if m.get(src) is not None:
            out[dst] = m[src]
    return out


def _lightning(m: dict) -> dict:
    return {"mixer": "lightning", **{k: m[k] for k in ("heads", "dim", "vdim", "decay")}}


_MIXERS = {"attention": _attention, "lightning": _lightning}


def composed_config(config: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
    """The library's configuration of a Musutar config.json."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        kind, mlp = entry["type"], entry.get("mlp")
        if kind not in _MIXERS:
            raise ValueError(f"layer {i}: mixer {kind!r} is not part of this design {tuple(_MIXERS)}")
        out = _MIXERS[kind](entry["mixer"])
        if mlp is not None:
            if mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: feed-forward {mlp.get('kind')!r} is not part of this design")
            out["mlp_hidden"], out["mlp_act"] = int(mlp["ff"]), "relu2"
        layers.append(out)
    return {"vocab_size": int(config["vocab"]), "dim": int(config["width"]), "norm": "layer",
            "norm_eps": float(config["norm"]["eps"]), "streams": int(config["streams"]),
            "input_conv": int(config["canon"]["taps"]), "residual_gate": True, "layers": layers}


class MusutarLM(DesignLM):
    ARCHITECTURE = "Musutar"
    composed_config = staticmethod(composed_config)
