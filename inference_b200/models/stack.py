"""What the decoders whose config lists its layers share: construction, rotary tables, padded weights, projections, logits."""
from __future__ import annotations

import torch

from .. import ops
from ..contracts.errors import LoadError, Unsupported
from ..engine.kv_pool import LayeredKvPool, StateGeometry
from ..parallel.comm import Communicator, single
from .config import ChannelDeltaSpec, ModelConfig, rescale_frequencies


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


def half_pairs(dim: int, rot: int) -> list[int]:
    """Order of a head's dimensions that makes the partners (i, i + rot / 2) of a rotation neighbours; the kernels rotate neighbours, and
    a head's scores do not depend on the order of its dimensions."""
    return [j for i in range(rot // 2) for j in (i, i + rot // 2)] + list(range(rot, dim))


class StackDecoder:
    """One GPU, bf16 or true 32-bit (numerical checks). Widths that are not multiples of eight are padded with zero rows /
    columns at load time, which changes no result."""
    name = "stack"
    recurrent = False      # the cache pool needs state slots

    def __init__(self, cfg: ModelConfig, comm: Communicator | None = None, device: torch.device | None = None,
                 dtype: torch.dtype = torch.bfloat16):
        if cfg.stack is None:
            raise Unsupported(f"{self.name} needs a config that lists its layers")
        if dtype not in (torch.bfloat16, torch.float32):
            raise Unsupported(f"dtype {dtype}: bfloat16 or float32")
        self.comm = comm or single(device)
        if self.comm.is_parallel:
            raise Unsupported(f"{self.name} runs on one GPU; tensor parallelism is not built for it")
        self.cfg, self.stack, self.dtype = cfg, cfg.stack, dtype
        self.device = device or self.comm.device
        self.width, self.hp = cfg.hidden_size, up8(cfg.hidden_size)
        self.layers: list = []
        self.embed = self.final = None
        self.head = None           # rows that give the logits, where they are not the embedding table
        self._rope: dict[tuple, tuple[torch.Tensor, torch.Tensor]] = {}
        self.max_positions = 0
        self.launches = 0

    # ---- cache geometry -----------------------------------------------------------------------------------------
    def kv_geometry(self) -> list:
        raise NotImplementedError

    def kv_block_bytes(self, block_size: int = 16) -> int:
        return LayeredKvPool.block_bytes(self.kv_geometry(), block_size, self.dtype.itemsize)

    def make_pool(self, num_blocks: int, block_size: int = 16, state_slots: int = 0) -> LayeredKvPool:
        return LayeredKvPool(self.kv_geometry(), num_blocks, block_size, device=self.device, dtype=self.dtype, state_slots=state_slots)

    # ---- rotary tables --------------------------------------------------------------------------------------------
    def rotations(self) -> set[tuple[int, float]]:
        """(rotated dimensions, base) or (rotated dimensions, base, rescaling) of every layer that rotates."""
        raise NotImplementedError

    def ensure_rope(self, max_positions: int) -> None:
        if max_positions <= self.max_positions:
            return
        for key in self.rotations():
            dims, base = key[:2]
            freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
            if len(key) > 2 and key[2] is not None:
                freq = rescale_frequencies(freq, key[2])
            ang = torch.arange(max_positions, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
            self._rope[key] = (ang.cos().float().to(self.device).contiguous(),
                                        ang.sin().float().to(self.device).contiguous())
        self.max_positions = max_positions

    # ---- weights ----------------------------------------------------------------------------------------------------
    @staticmethod
    def tensor(weights: dict[str, torch.Tensor], name: str, *shape: int | None) -> torch.Tensor:
        """A tensor by name, its shape checked (None: any extent)."""
        if name not in weights:
            raise LoadError(f"missing tensor {name}")
        t = weights[name]
        if len(t.shape) != len(shape) or any(b is not None and a != b for a, b in zip(t.shape, shape)):
            raise LoadError(f"tensor {name} has shape {tuple(t.shape)}, expected {shape}")
        return t

    def _mat(self, t: torch.Tensor) -> torch.Tensor:
        """A matrix whose columns are stream columns: padded to the padded width, in the compute type, on the device."""
        return torch.nn.functional.pad(t.to(self.device, self.dtype), (0, self.hp - self.width)).contiguous()

    def _fp32(self, t: torch.Tensor, pad_to: int | None = None) -> torch.Tensor:
        t = t.to(self.device, torch.float32)
        return torch.nn.functional.pad(t, (0, (pad_to or t.shape[-1]) - t.shape[-1])).contiguous()

    def _heads(self, t: torch.Tensor, n: int, parts: list[tuple[int, int]], cols: int | None = None) -> torch.Tensor:
        """Rows laid out head by head in parts of the given (size, padded size) -> the same with every part padded; columns
        padded to `cols` (default: the stream's padded width)."""
        t = t.to(self.device, self.dtype).reshape(n, sum(a for a, _ in parts), -1)
        out = torch.zeros((n, sum(b for _, b in parts), cols or self.hp), dtype=self.dtype, device=self.device)
        src = dst = 0
        for a, b in parts:
            out[:, dst:dst + a, :t.shape[2]] = t[:, src:src + a]
            src, dst = src + a, dst + b
        return out.reshape(-1, out.shape[2])

    def _out(self, o: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
        out = torch.zeros((self.hp, heads, dp), dtype=self.dtype, device=self.device)
        out[:self.width, :, :d] = o.to(self.device, self.dtype).reshape(self.width, heads, d)
        return out.reshape(self.hp, heads * dp)

    def _pairs(self, gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
        """Rows (gate_0, up_0, gate_1, ...), padded."""
        ff = gate.shape[0]
        out = torch.zeros((up8(ff), 2, self.hp), dtype=self.dtype, device=self.device)
        out[:ff, 0, :self.width], out[:ff, 1, :self.width] = gate.to(self.device, self.dtype), up.to(self.device, self.dtype)
        return out.view(-1, self.hp)

    def _delta_inputs(self, m: ChannelDeltaSpec, p: str, get) -> tuple[list[torch.Tensor], torch.Tensor]:
        """Delta rule: (the projections q, k, v with every head padded, fp32 convolution weights [taps, their rows])."""
        dp, vp = ops.delta_key_width(m.dim), up8(m.vdim)
        parts = {"q": (m.kv_heads, m.dim, dp), "k": (m.kv_heads, m.dim, dp), "v": (m.heads, m.vdim, vp)}
        rows = [self._heads(get(p + n, h * d, self.width), h, [(d, padded)]) for n, (h, d, padded) in parts.items()]
        conv = torch.cat([torch.nn.functional.pad(self._fp32(get(f"{p}{n}.conv", h * d, m.conv)).view(h, d, m.conv),
                                                  (0, 0, 0, padded - d)).reshape(-1, m.conv) for n, (h, d, padded) in parts.items()])
        return rows, conv.t().contiguous()

    @staticmethod
    def _delta_geometry(m: ChannelDeltaSpec) -> StateGeometry:
        dp, vp = ops.delta_key_width(m.dim), up8(m.vdim)
        return StateGeometry((m.heads, vp, dp), (m.conv - 1, 2 * m.kv_heads * dp + m.heads * vp))

    # ---- forward ----------------------------------------------------------------------------------------------------
    def _linear(self, a: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype | None = None, out: torch.Tensor | None = None,
                bias: torch.Tensor | None = None, act: str | None = None, act_params: tuple[float, float] = (0.0, 0.0)) -> torch.Tensor:
        self.launches += 1
        if self.dtype == torch.float32:
            return ops.gemm_f32(a, w, out=out, bias=bias, act=act, act_params=act_params)
        return ops.gemm_bf16(a, w, out=out, out_dtype=out_dtype or torch.bfloat16, bias=bias, act=act, act_params=act_params)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        if hidden.shape[0] == 0:
            return torch.empty((0, self.cfg.vocab_size), dtype=torch.float32, device=self.device)
        return self._linear(hidden, self.embed if self.head is None else self.head, torch.float32)

    def greedy_tokens(self, hidden: torch.Tensor) -> torch.Tensor:
        self.launches += 1
        return ops.argmax(self.logits(hidden))
