"""Which decoder class serves a configuration on the GPU."""
from __future__ import annotations

import torch

from ..contracts.errors import Unsupported
from .config import Architecture, ModelConfig


def gpu_supported(cfg: ModelConfig) -> bool:
    """True when a paged sm_100a decoder exists for this configuration."""
    if cfg.stack is not None:
        return True
    return (cfg.head_dim == 128 and cfg.mla is None and
            cfg.architecture not in (Architecture.QWEN35, Architecture.DEEPSEEK_V2))


def gpu_model(cfg: ModelConfig, comm=None, device: torch.device | None = None, dtype: torch.dtype = torch.bfloat16):
    """An empty paged decoder for `cfg` (load_state_dict or init_random fills it). The Llama family computes in bf16 only."""
    if not gpu_supported(cfg):
        raise Unsupported(f"{cfg.architecture.value} (head_dim {cfg.head_dim}) is not served by the sm_100a decoders; load it "
                          "through the cpu-llama provider")
    if cfg.architecture is Architecture.ZOBUNEX:
        from .zobunex import ZobunexGpu

        return ZobunexGpu(cfg, comm=comm, device=device, dtype=dtype)
    if cfg.architecture is Architecture.GUNEDRA:
        from .gunedra import GunedraGpu

        return GunedraGpu(cfg, comm=comm, device=device, dtype=dtype)
    if cfg.architecture is Architecture.ROTALORN:
        from .rotalorn import RotalornGpu

        return RotalornGpu(cfg, comm=comm, device=device, dtype=dtype)
    if cfg.architecture is Architecture.NAFELIX:
        from .nafelix import NafelixGpu

        return NafelixGpu(cfg, comm=comm, device=device, dtype=dtype)
    if dtype != torch.bfloat16:
        raise Unsupported(f"{cfg.architecture.value}: the sm_100a decoder computes in bfloat16")
    from .llama import LlamaGpu

    return LlamaGpu(cfg, comm=comm, device=device)
