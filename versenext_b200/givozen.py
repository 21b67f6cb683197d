"""The Givozen design: config.json and checkpoint of such a model -> a `ComposedLM`.

Layers of grouped-query attention (biases on q, k and v, half-split rotary positions with scaling by wavelength, a temperature
and a gate for every query head), each with an optional PolyNorm feed-forward or a mixture of clamped experts (sigmoid scores
that weigh an expert's input, an expert that serves every token); norms before and behind every sublayer, tied embeddings, and
an optional block of layers that runs several times and begins each pass by adding.  Weights are bfloat16 in
`model.safetensors`, named as the library takes them.
"""

from __future__ import annotations

from typing import Dict, Tuple

from .composed import DesignLM


def _attention(m: dict) -> dict:
    out = {"mixer": "attention", **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}, "bias": True, "out_bias": False,
           "temperature": True, "output_gate": "head"}
    rot = m.get("rot")
    if rot:
        s = rot.get("scaling")
        out["rope"] = {"dims": int(rot["dims"]), "base": float(rot["base"]),
                       "scaling": {"kind": "wavelength", **{k: float(s[k]) for k in ("factor", "low", "high", "original")}} if s else None}
    return out


def _mlp(mlp: dict, i: int) -> dict:
    if mlp.get("kind") == "dense":
        return {"mlp_hidden": int(mlp["ff"]), "mlp_act": "poly_norm"}
    if mlp.get("kind") != "moe":
        raise ValueError(f"layer {i}: feed-forward {mlp.get('kind')!r} is not part of this design")
    r, shared = mlp["router"], mlp.get("shared")
    experts = {"count": int(r["experts"]), "top": int(r["top"]), "score": "sigmoid", "weight": "input"}
    if shared:
        experts["shared"] = {"hidden": int(shared["ff"]), "limit": float(shared["limit"])}
    return {"mlp_hidden": int(mlp["expert"]["ff"]), "mlp_act": "clamped", "mlp_limit": float(mlp["expert"]["limit"]), "experts": experts}


def composed_config(config: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
    """The library's configuration of a Givozen config.json."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        if entry["type"] != "attention":
            raise ValueError(f"layer {i}: mixer {entry['type']!r} is not part of this design ('attention',)")
        out = _attention(entry["mixer"])
        if entry.get("mlp") is not None:
            out.update(_mlp(entry["mlp"], i))
        layers.append(out)
    out = {"vocab_size": int(config["vocab"]), "dim": int(config["width"]), "norm_eps": float(config["norm"]["eps"]), "post_norm": True,
           "tie_weights": True, "layers": layers}
    loop = config.get("loop")
    if loop:
        out["loop"] = {**{k: int(loop[k]) for k in ("start", "stop", "times")}, "entry": "add"}
    return out


class GivozenLM(DesignLM):
    ARCHITECTURE = "Givozen"
    composed_config = staticmethod(composed_config)
