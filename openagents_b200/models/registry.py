"""Which engine serves which model, and where a model's weights come from.

A model path is a GGUF file or a checkpoint folder (``config.json`` + ``model.safetensors``); its configuration names the
architecture, and the architecture picks the engine class.
"""
from __future__ import annotations

import os

from .config import ModelConfig

COMPUTE_DTYPES = ("bfloat16", "float32")


def is_checkpoint_dir(path: str) -> bool:
    return os.path.isdir(path) and os.path.exists(os.path.join(path, "config.json"))


def open_source(path: str, device):
    """``WeightSource`` over the model at ``path``; its ``cfg`` is the model's configuration."""
    if is_checkpoint_dir(path):
        from .checkpoint_dir import CheckpointDirSource
        return CheckpointDirSource(path, device)
    from .qweight import GGUFSource
    return GGUFSource(path, device)


def peek_architecture(path: str) -> str:
    """The architecture of a model, without loading tensors."""
    if is_checkpoint_dir(path):
        import json
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            return str(json.load(f).get("architecture")).lower()
    from ..gguf import GGUFFile
    with GGUFFile(path) as f:
        return f.metadata.get("general.architecture")


def tokenizer_metadata(path: str) -> dict:
    """``tokenizer.*`` metadata of a GGUF file (a checkpoint folder carries none: raw bytes are its tokens)."""
    if is_checkpoint_dir(path):
        return {}
    from ..gguf import GGUFFile
    with GGUFFile(path) as f:
        return {k: v for k, v in f.metadata.items() if k.startswith("tokenizer.")}


def weights_file(path: str) -> str:
    """The file whose digest identifies the model's weights."""
    return os.path.join(path, "model.safetensors") if is_checkpoint_dir(path) else path


def engine_class(cfg: ModelConfig):
    if cfg.layers:
        from .hybrid_engine import HybridEngine
        return HybridEngine
    if cfg.n_experts:
        from .moe_engine import MoEEngine
        return MoEEngine
    from .engine import LlamaEngine
    return LlamaEngine


def build_engine(src, device, max_batch: int, max_ctx: int, max_tokens: int = 4096, n_pages: int | None = None, dtype: str = "bfloat16",
                 tp_rank: int = 0, tp_world: int = 1, ep_rank: int = 0, ep_world: int = 1, comm=None, state_slots: int | None = None, **options):
    """The engine for ``src.cfg``.  ``dtype``: "float32" computes everything in true 32-bit, for the families that have it;
    ``state_slots``: sequences that may be open at a time, for the families with a recurrent state; ``options`` are the family's own."""
    cfg, cls = src.cfg, engine_class(src.cfg)
    if dtype not in COMPUTE_DTYPES:
        raise ValueError(f"dtype is one of {COMPUTE_DTYPES}")
    common = dict(device=device, max_batch=max_batch, max_ctx=max_ctx, max_tokens=max_tokens, n_pages=n_pages, **options)
    if cfg.layers:
        if max(tp_world, ep_world) > 1:
            raise ValueError(f"{cfg.arch} models are served on one GPU")
        return cls(cfg, src, dtype=dtype, state_slots=state_slots, **common)
    if dtype != "bfloat16":
        raise ValueError(f"{cfg.arch} models have no 32-bit mode")
    if cfg.n_experts:
        return cls(cfg, src, ep_rank=ep_rank, ep_world=ep_world, comm=comm, **common)
    return cls(cfg, src, tp_rank=tp_rank, tp_world=tp_world, comm=comm, **common)
