"""Model folders: config.json names the architecture, which decides the decoder class, its weight file and the kernel
parts it needs.

  "llama", "deepseek", "gpt"   {"architecture", "vocab_size", "max_seq_len", "d_model", "n_heads", "n_layers", "d_ff",
                               "q_rank", "kv_rank"} with a DeepJ checkpoint model.bin (persistence/ModelSerializer.java),
                               quantized to Q8 on load; dtype "q8"
  "Punilix", "Somipel"         layers listed one by one (hybrid.py) with model.safetensors; dtype "bf16" or "f32"
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, Optional

from . import _lib, build

HYBRID = ("Punilix", "Somipel")
Q8_KINDS = ("llama", "deepseek", "gpt")
DTYPES = {"bfloat16": "bf16", "float32": "f32", "bf16": "bf16", "f32": "f32", "q8": "q8"}


class UnsupportedDtype(ValueError):
    """The architecture has no kernels for the requested number format."""


def read_config(folder: str) -> Dict[str, Any]:
    with open(os.path.join(folder, "config.json")) as f:
        rec = json.load(f)
    if rec.get("architecture") not in HYBRID + Q8_KINDS:
        raise ValueError(f"unknown architecture {rec.get('architecture')!r}")
    return rec


def dtypes_of(architecture: str) -> tuple:
    return ("bf16", "f32") if architecture in HYBRID else ("q8",)


def load_model(folder: str, dtype: Optional[str] = None, max_seq_len: Optional[int] = None, batch: int = 1, device: int = 0):
    """The decoder of a model folder, weights loaded.  `dtype` defaults to the format the family is served in;
    `max_seq_len` bounds the positions a sequence may hold (Q8 families: at most the model's own)."""
    rec = read_config(folder)
    arch = rec["architecture"]
    if dtype is not None and DTYPES.get(dtype) not in dtypes_of(arch):
        raise UnsupportedDtype(f"{arch} runs in {', '.join(dtypes_of(arch))}, not in {dtype}")
    dtype = DTYPES[dtype] if dtype else dtypes_of(arch)[0]
    _lib.load(build.ensure(("bf16",) if arch in HYBRID else ("*",)))
    from . import checkpoint
    if arch in HYBRID:
        from .hybrid import HybridConfig, HybridDecoder
        st = checkpoint.SafetensorsFile(os.path.join(folder, "model.safetensors"))
        cfg = HybridConfig.parse(rec, max_seq_len or 4096, lambda name: st.shape(name)[0] if name in st.header else None)
        dec = HybridDecoder(cfg, batch=batch, device=device, dtype=dtype)
        dec.load_weights(st.get)
        return dec
    from .decoder import DecoderConfig, Q8Decoder
    own = int(rec["max_seq_len"])
    if arch == "gpt" and max_seq_len is not None:
        max_seq_len = own            # the learned position table has a fixed length
    cfg = DecoderConfig(arch, rec["vocab_size"], min(own, max_seq_len or own), rec["d_model"], rec["n_heads"], rec["n_layers"], rec["d_ff"],
                        rec.get("q_rank", 0), rec.get("kv_rank", 0))
    dec = Q8Decoder(cfg, batch=batch, device=device)
    dec.load_weights(checkpoint.weight_getter(cfg, os.path.join(folder, "model.bin")))
    return dec
