"""Builds the GPU decode backend of a model: decoder class, weights, paged pool and step runner."""
from __future__ import annotations

import torch

from ..contracts.errors import LoadError
from ..models.config import ModelConfig
from ..models.registry import gpu_model
from .backend import GpuBackend
from .kv_pool import PagedKvPool
from .runner import ModelRunner

BLOCK = 16


def gpu_backend(cfg: ModelConfig, weights: dict[str, torch.Tensor], comm=None, *, dtype: torch.dtype = torch.bfloat16,
                max_batch: int = 16, max_context: int | None = None, kv_tokens: int | None = None) -> GpuBackend:
    """kv_tokens: the pool holds exactly that many tokens (rounded up to pages) and, for recurrent layers, the states of
    max_batch sequences; None sizes it for max_batch full contexts, at most 60 % of the free memory, and twice max_batch
    states (cached prefixes and checkpoints of speculative steps hold some)."""
    if not torch.cuda.is_available():
        raise LoadError("the b200 backend needs a CUDA device (use the cpu runtime bundle on hosts without one)")
    dev = comm.device if comm is not None else torch.device("cuda", torch.cuda.current_device())
    model = gpu_model(cfg, comm=comm, device=dev, dtype=dtype).load_state_dict(weights)
    ctx = max_context or min(cfg.max_position_embeddings or 8192, 32768)
    own_pool = hasattr(model, "make_pool")
    if kv_tokens is not None:
        nblocks = (kv_tokens + BLOCK - 1) // BLOCK
    else:
        free, _total = torch.cuda.mem_get_info(dev)
        per_block = model.kv_block_bytes(BLOCK) if own_pool else cfg.num_layers * 2 * model.hkv * BLOCK * cfg.head_dim * 2
        want = max_batch * ((ctx + BLOCK - 1) // BLOCK) + 64
        nblocks = max(64, min(want, int(free * 0.6) // max(1, per_block)))
    extra = {"state_slots": max_batch * (2 if kv_tokens is None else 1)} if getattr(model, "recurrent", False) else {}
    pool = model.make_pool(nblocks, BLOCK, **extra) if own_pool else \
        PagedKvPool(cfg.num_layers, nblocks, model.hkv, cfg.head_dim, BLOCK, device=dev)
    return GpuBackend(ModelRunner(model, pool, max_batch=max_batch, max_seq_len=ctx))
