"""Model designs by the name their configuration gives ("architecture"), and loading from a directory or file."""

from __future__ import annotations

import json
import os

from .bozasun import BozasunLM
from .fuzudra import FuzudraLM
from .givozen import GivozenLM
from .model import DeviceLM, VerseNexLM
from .musutar import MusutarLM

_DESIGNS: dict = {}


def register(architecture: str, cls) -> None:
    """`cls` needs `from_pretrained(path, dtype=, device=)`."""
    _DESIGNS[architecture] = cls


def architectures():
    return sorted(_DESIGNS)


def model_class(architecture: str):
    try:
        return _DESIGNS[architecture]
    except KeyError:
        raise ValueError(f"architecture {architecture!r} is not known {tuple(architectures())}") from None


def load_model(path: str, dtype: str = "bf16", device: str = "cuda", **kw) -> DeviceLM:
    """A model from a directory with config.json (the class by its "architecture") or from a `.vn` file / a directory
    with one (VerseNexLM)."""
    cfg = os.path.join(path, "config.json")
    if os.path.isdir(path) and os.path.exists(cfg):
        with open(cfg) as f:
            arch = json.load(f).get("architecture")
        return model_class(arch).from_pretrained(path, dtype=dtype, device=device, **kw)
    return VerseNexLM.from_pretrained(path, dtype=dtype, device=device, **kw)


register(BozasunLM.ARCHITECTURE, BozasunLM)
register(FuzudraLM.ARCHITECTURE, FuzudraLM)
register(GivozenLM.ARCHITECTURE, GivozenLM)
register(MusutarLM.ARCHITECTURE, MusutarLM)
register("VerseNexLM", VerseNexLM)
register("CometSparkNexLM", VerseNexLM)
