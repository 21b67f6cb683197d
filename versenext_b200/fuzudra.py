"""The Fuzudra design: config.json and checkpoint of such a model -> a `ComposedLM`.

config.json names every layer (`type`, the sizes of its `mixer`, its `mlp`), the looped block (`loop`), the norm's eps,
the vocabulary and the width.  The ranks of the delta rule's two low-rank factors are read off the tensors' shapes.
Weights are bfloat16 in `model.safetensors`, named as the library takes them.
"""

from __future__ import annotations

from typing import Dict, Tuple

from .composed import DesignLM

_MIXER_KEYS = {
    "latent_attention": ("heads", "dim", "vdim", "kv_rank", "scale"),
    "mamba1": ("inner", "state", "dt_rank", "conv"),
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}


def composed_config(config: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
    """The library's configuration of a Fuzudra config.json; `shapes`: tensor name -> shape."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        kind, mixer, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind not in _MIXER_KEYS:
            raise ValueError(f"layer {i}: mixer {kind!r} is not part of this design {tuple(_MIXER_KEYS)}")
        out = {"mixer": kind, **{k: mixer[k] for k in _MIXER_KEYS[kind]}}
        if kind == "latent_attention":
            out["window"] = int((mixer.get("mask") or {}).get("size") or 0)
        elif kind == "channel_delta":
            out["decay_rank"] = int(shapes[f"l{i}.mix.a1"][0])
            out["gate_rank"] = int(shapes[f"l{i}.mix.g1"][0])
        if mlp is not None:
            if mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: feed-forward {mlp.get('kind')!r} is not part of this design")
            out["mlp_hidden"], out["mlp_act"] = int(mlp["ff"]), "gelu_tanh"
        layers.append(out)
    out = {"vocab_size": int(config["vocab"]), "dim": int(config["width"]), "norm_eps": float(config["norm"]["eps"]),
           "positions": "sinusoidal", "layers": layers}
    loop = config.get("loop")
    if loop:
        out["loop"] = {k: int(loop[k]) for k in ("start", "stop", "times")}
    return out


class FuzudraLM(DesignLM):
    ARCHITECTURE = "Fuzudra"
    composed_config = staticmethod(composed_config)
