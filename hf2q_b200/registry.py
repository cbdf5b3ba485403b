"""Model registry: which decoder class serves a model, by the architecture its files name."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from . import _lib, ops


def _fomatar(ctx, path, dtype, max_seq, n_slots, prefill_chunk):
    from .fomatar import FomatarDecoder
    return FomatarDecoder.from_directory(ctx, path, dtype=dtype, max_seq=max_seq, n_slots=n_slots, prefill_chunk=prefill_chunk)


def _runopel(ctx, path, dtype, max_seq, n_slots, prefill_chunk):
    from .runopel import RunopelDecoder
    return RunopelDecoder.from_directory(ctx, path, dtype=dtype, max_seq=max_seq, n_slots=n_slots, prefill_chunk=prefill_chunk)


def _llama(ctx, path, dtype, max_seq, n_slots, prefill_chunk):
    from .decoder import LlamaDecoder
    if dtype != torch.bfloat16:
        raise ops.Hf2qError(_lib.ERR_INVALID_ARGUMENT, "the quantized decoder has no 32-bit mode")
    return LlamaDecoder.from_gguf(ctx, path, max_seq=max_seq, prefill_chunk=prefill_chunk)


# config.json "architecture" of a model folder, or "general.architecture" of a GGUF file
ARCHITECTURES = {"Fomatar": _fomatar, "Runopel": _runopel, "llama": _llama}


def architecture_of(path) -> str:
    path = Path(path)
    if path.is_dir():
        return json.loads((path / "config.json").read_text())["architecture"]
    from .gguf import GgufFile
    with GgufFile(path) as g:
        return str(g.metadata["general.architecture"])


def load_model(ctx: ops.GpuContext, path, dtype=torch.bfloat16, max_seq: int = 32768, n_slots: int = 1, prefill_chunk: int = 2048):
    """The decoder that serves the model at ``path``: a folder with config.json and model.safetensors, or a .gguf file."""
    arch = architecture_of(path)
    if arch not in ARCHITECTURES:
        raise ops.Hf2qError(_lib.ERR_INVALID_ARGUMENT, f"architecture '{arch}' is not registered (have: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[arch](ctx, path, dtype, max_seq, n_slots, prefill_chunk)
