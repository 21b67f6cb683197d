"""Models composed of layers of different kinds: the device's `"family": "composed"` configurations.

`ComposedLM` takes the neutral configuration the library reads (a list of layers, each a mixer with its sizes and an
optional feed-forward; an optional looped block; the norm and its eps; the kind of positions; the arrangement of the
residual) and offers what every model of the package offers: weight loading, caches, uniform and ragged steps, generation,
speculative decoding as target or draft.  A named design is a subclass of `DesignLM` that translates its own config.json
(see bozasun.py, fuzudra.py, givozen.py, musutar.py).

Mixers: "latent_attention" (heads, dim, vdim, kv_rank, scale, window, rot_dim with rope, sink, output_gate "head", "element" or
"none"), "attention" (heads, kv_heads, dim, vdim, scale, window, chunk, softcap, conv, rope, bias, out_bias, qk_norm,
temperature, output_gate "head", "element" or "none", kv_from),
"mamba1" (inner, state, dt_rank, conv), "mamba2" (heads, vdim, state, groups, norm_groups, conv), "channel_delta" (heads,
kv_heads, dim, vdim, conv, decay_rank, gate_rank), "lightning" (heads, dim, vdim, decay).  rope: {dims, base, interleaved,
scaling: YaRN {factor, original, fast, slow}, {kind: "linear", factor} or {kind: "wavelength", factor, low, high, original}}.

Feed-forwards: mlp_hidden with mlp_act "silu", "gelu_tanh" or "clamped" (gated; the last one with mlp_limit) or "relu2" or
"poly_norm" (plain); with experts {count, identity, top, groups, keep, correction, score "softmax" or "sigmoid", weight of the
"result" or the "input", shared {hidden, limit}} a mixture of gated ones.

Model-wide: norm "rms" (weights stored around zero, or plain: norm_weight "plain") or "layer" (plain weights); streams (residual
streams, hyper-connections); input_conv (taps of the convolution that a mixer's input gets); residual_gate (sigmoid gate on every
sublayer's result); post_norm (an RMS norm of every sublayer's result); token_side (width of the input that every layer has for
each token); tie_weights; loop {start, stop, times, entry "project" or "add"}.
"""

from __future__ import annotations

import ctypes as C
import json
import os
from typing import Dict, Optional, Tuple

import numpy as np

from .device import as_device
from .model import DeviceLM, KVCache, _ptr
from .safetensors_file import SafetensorsFile


class ComposedLM(DeviceLM):
    def __init__(self, config: dict, dtype: str = "bf16", device: str = "cuda"):
        if dtype not in ("f32", "bf16"):
            raise ValueError("dtype must be 'f32' or 'bf16'")
        self._config = dict(config, family="composed", dtype=dtype)
        self.dtype = dtype
        self.vocab_size, self.dim = int(config["vocab_size"]), int(config["dim"])
        self.n_layer = len(config["layers"])
        self.max_seq_len = int(config.get("max_seq_len", 4096))
        loop = config.get("loop")
        self.n_runs = self.n_layer + (loop["stop"] - loop["start"]) * (loop["times"] - 1) if loop else self.n_layer
        self._create(self._config, device)

    def get_config(self) -> dict:
        return dict(self._config)

    def load_state_dict(self, sd: dict):
        for name, value in sd.items():
            self.load_tensor(name, getattr(value, "data", value) if not isinstance(value, np.ndarray) else value)
        self.finalize()

    # speculative engines switch the one-token route of VerseNexLM; there is only one route here
    def _set_recurrent(self, on: bool):
        pass

    def new_cache(self, max_batch: int, max_seq: Optional[int] = None, max_pending: int = 1, pool_tokens: int = 0) -> KVCache:
        """`pool_tokens` > 0: latent pages for that many tokens in all, shared by the sequences (else every sequence owns
        the pages of `max_seq` positions)."""
        return KVCache(self, max_batch, max_seq if max_seq is not None else self.max_seq_len, pool_tokens=pool_tokens,
                       max_pending=max_pending)

    def forward_ragged(self, cache: KVCache, slots, counts, tokens, out_rows):
        """One step over a ragged batch (see DeviceLM.forward_ragged): the entries run together."""
        if not self._finalized:
            self.finalize()
        slots = np.ascontiguousarray(slots, dtype=np.int32)
        counts = np.ascontiguousarray(counts, dtype=np.int32)
        rows = np.ascontiguousarray(out_rows, dtype=np.int32)
        tok = as_device(self.ctx, tokens, np.int64)
        if slots.shape != counts.shape or int(counts.sum()) != tok.size:
            raise ValueError("one count per slot, and as many tokens as the counts sum up to")
        out = self.ctx.empty((len(rows), self.vocab_size), np.float32) if len(rows) else None
        vp = C.c_void_p
        self.ctx._check(self.ctx.lib.vn_model_forward_ragged(
            self.handle, cache.handle, _ptr(tok), len(slots), slots.ctypes.data_as(vp), counts.ctypes.data_as(vp),
            len(rows), rows.ctypes.data_as(vp), None, _ptr(out)))
        return out

    def residuals(self, tokens) -> np.ndarray:
        """Diagnostic: the residual stream after every layer run for one sequence, (runs, T, dim)."""
        tokens = np.ascontiguousarray(tokens, dtype=np.int64).reshape(1, -1)
        T = tokens.shape[1]
        buf = self.ctx.empty((self.n_runs, T, self.dim), np.float32)
        cache = self.new_cache(1, T)
        self.ctx._check(self.ctx.lib.vn_model_set_probe(self.handle, _ptr(buf)))
        try:
            self.forward_cached(tokens, cache, last_only=True)
            return buf.numpy()
        finally:
            self.ctx._check(self.ctx.lib.vn_model_set_probe(self.handle, None))

    def generate(self, idx, max_new_tokens: int = 128, temperature: float = 0.0, top_k: Optional[int] = None,
                 eos_id: Optional[int] = None, seed: int = 0, draft: Optional[DeviceLM] = None, k: int = 4):
        """Generation for a batch of prompts: (B, T) or a list of prompts of any lengths.  Returns a list of 1-D arrays of
        the new tokens.  temperature <= 0 is greedy.  With `draft`, rounds of the speculative engine."""
        prompts = [np.asarray(p, dtype=np.int64).reshape(-1) for p in
                   (idx if isinstance(idx, (list, tuple)) else np.atleast_2d(np.asarray(idx)))]
        if draft is not None:
            from .engine import SpecEngine
            eng = SpecEngine(self, draft, max_batch=len(prompts), max_seq=max(map(len, prompts)) + max_new_tokens + 4 * (k + 2),
                             k=k, temperature=temperature, top_k=top_k or 0, seed=seed, max_new_tokens=max_new_tokens)
            return eng.serve(prompts, max_new_tokens, eos_id=eos_id)
        from .serving import BatchEngine
        eng = BatchEngine(self, max_batch=len(prompts), max_seq=max(map(len, prompts)) + max_new_tokens)
        return eng.run(prompts, max_new_tokens, temperature=temperature, top_k=top_k or 0, eos_id=eos_id, seed=seed)


class DesignLM(ComposedLM):
    """A named design: `ARCHITECTURE` and `composed_config(config, shapes)` make it a `ComposedLM`.  `config`: config.json's
    contents; `shapes`: tensor name -> shape."""

    ARCHITECTURE = ""

    @staticmethod
    def composed_config(config: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
        raise NotImplementedError

    def __init__(self, config: dict, shapes: Dict[str, Tuple[int, ...]], dtype: str = "bf16", device: str = "cuda",
                 max_seq_len: int = 4096):
        self.source_config = config
        super().__init__(dict(self.composed_config(config, shapes), max_seq_len=max_seq_len), dtype=dtype, device=device)

    @classmethod
    def from_state_dict(cls, config: dict, sd: dict, **kw):
        model = cls(config, {n: tuple(a.shape) for n, a in sd.items()}, **kw)
        model.load_state_dict(sd)
        return model

    @classmethod
    def from_pretrained(cls, path: str, dtype: str = "bf16", device: str = "cuda", **kw):
        """A directory with config.json and model.safetensors; tensors stream to the device one at a time."""
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        with SafetensorsFile(os.path.join(path, "model.safetensors")) as st:
            model = cls(config, st.shapes(), dtype=dtype, device=device, **kw)
            for name, arr in st:
                model.load_tensor(name, arr)
        model.finalize()
        return model
