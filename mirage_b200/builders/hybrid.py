"""What the builders of hybrid graphs share: buffers and weights padded for the tensor path, rotary tables, the mLSTM mixer, the head.

Linear weights of a bf16 graph are padded to a multiple of 64 input columns (the tensor path's k granularity), the activation
buffers in front of them likewise: what the padding columns hold is finite and meets zero weights.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..persistent_kernel import DTensor, PersistentKernel, bfloat16, float32, int32, int64


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def k_padded(k: int, dtype: torch.dtype) -> int:
    """Input columns a linear of a graph with activations of this type gives a weight of `k` columns."""
    return round_up(k, 64) if dtype == torch.bfloat16 else k


@dataclass(frozen=True)
class RotaryScaling:
    """Frequencies for longer contexts as in Llama 3.1: wavelengths longer than original / low positions are stretched by `factor`,
    those shorter than original / high are kept, the ones between are blended."""
    factor: float
    low: float
    high: float
    original: float

    def apply(self, f: torch.Tensor) -> torch.Tensor:
        turns = self.original * f / (2.0 * math.pi)           # original / wavelength
        s = (turns - self.low) / (self.high - self.low)
        blend = (1.0 - s) * f / self.factor + s * f
        return torch.where(turns > self.high, f, torch.where(turns < self.low, f / self.factor, blend))


def rotary_tables(base: float, dims: int, positions: int, device, scaling: Optional[RotaryScaling] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """float32 cos / sin [positions, dims / 2] of position * base^(-2i / dims); the angles are formed in 64-bit."""
    if dims == 0:
        z = torch.zeros(1, 1, dtype=torch.float32, device=device)
        return z, z.clone()
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if scaling is not None:
        f = scaling.apply(f)
    a = torch.arange(positions, dtype=torch.float64)[:, None] * f
    return a.cos().float().to(device), a.sin().float().to(device)


@dataclass(frozen=True)
class MlstmSpec:
    """Sizes of a matrix-memory mixer."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, m: Dict[str, Any]) -> "MlstmSpec":
        return cls(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))

    def state(self, slots: int, num_workers: int, device) -> Dict[str, torch.Tensor]:
        """float32, indexed by state slot: the memory, and normaliser and running maximum of every task of a head."""
        chunks = PersistentKernel.mlstm_chunks(num_workers, slots, self.heads, self.dim, self.vdim)
        z = lambda *s: torch.zeros(*s, dtype=torch.float32, device=device)
        return {"memory": z(slots, self.heads, self.dim, round_up(self.vdim, 4)), "normaliser": z(slots, self.heads, chunks, self.dim + 1)}


@dataclass
class HybridModelConfig:
    """What a builder needs beside the kernel: shapes, weights under their checkpoint names, state, activation type."""
    config: Any
    state_dict: Dict[str, torch.Tensor]
    state: List[Dict[str, torch.Tensor]]   # one entry per layer run
    dtype: torch.dtype = torch.bfloat16
    sampling_seed: Optional[int] = None    # None: greedy argmax; an int: Gumbel-max sampling

    def check_valid(self):
        assert self.state_dict is not None and len(self.state) >= len(self.config.layers)
        assert self.dtype in (torch.bfloat16, torch.float32)


class HybridBuilder:
    def __init__(self, mpk: PersistentKernel):
        self.mpk = mpk
        self.logits: Optional[DTensor] = None
        self.hidden: Optional[DTensor] = None      # float32 residual stream
        self._buffers: Dict[Tuple[str, tuple], DTensor] = {}
        self._tables: Dict[tuple, Tuple[DTensor, DTensor]] = {}
        self._attached: Dict[str, DTensor] = {}

    def _begin(self, mc: HybridModelConfig):
        self.sd, self.eps, self.width, self.dtype = mc.state_dict, mc.config.eps, mc.config.width, mc.dtype
        self.act = float32 if mc.dtype == torch.float32 else bfloat16

    def _buf(self, tag: str, width, dt) -> DTensor:
        """One buffer per purpose and row shape, shared by all layers."""
        shape = width if isinstance(width, tuple) else (width,)
        key = (tag, shape)
        if key not in self._buffers:
            self._buffers[key] = self.mpk.new_tensor(dims=(self.mpk.max_num_batched_tokens, *shape), dtype=dt,
                                                     name="_".join([tag, *map(str, shape)]))
        return self._buffers[key]

    def _kpad(self, k: int) -> int:
        return k_padded(k, self.dtype)

    def _attach(self, name: str, make) -> DTensor:
        """The tensor `make()` gives, once per name: a layer that runs several times has one set of weights."""
        if name not in self._attached:
            self._attached[name] = self.mpk.attach_input(make().contiguous(), name=name)
        return self._attached[name]

    def _weight(self, name: str, parts: List[torch.Tensor], dim: int = 0) -> DTensor:
        """The parts side by side along `dim`, input columns padded."""
        return self._attach(name, lambda: self._pad_k(torch.cat(parts, dim) if len(parts) > 1 else parts[0]))

    def _pad_k(self, w: torch.Tensor) -> torch.Tensor:
        pad = self._kpad(w.shape[-1]) - w.shape[-1]
        return torch.nn.functional.pad(w, (0, pad)) if pad else w

    def _att(self, name: str) -> DTensor:
        return self._attach(name, lambda: self.sd[name])

    def _linear(self, x: DTensor, w: DTensor, y: DTensor, activation: str = None, **kw):
        self.mpk.linear_layer(input=x, weight=w, output=y, grid_dim=(96, 1, 1), block_dim=(128, 1, 1), activation=activation, **kw)

    def _sublayer(self, x: DTensor, name: str, parts: List[torch.Tensor], bias: Optional[DTensor] = None) -> DTensor:
        """A sublayer's output linear, float32."""
        y = self._buf("sublayer", self.width, float32)
        self._linear(x, self._weight(name + ".padded", parts), y, bias=bias)
        return y

    def _mlstm(self, p: str, m: MlstmSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        """[q | k | v | gate | i | f] in one linear -> recurrence with its head norm and gate -> output linear."""
        mpk, sd = self.mpk, self.sd
        qk, v = m.heads * m.dim, m.heads * m.vdim
        proj = self._buf("proj", 2 * qk + 2 * v + 2 * m.heads, float32)
        self._linear(h, self._weight(p + "qkvgif", [sd[p + n] for n in ("q", "k", "v", "g", "i", "f")]), proj)
        out = self._buf("mixed", self._kpad(v), self.act)
        mpk.mlstm_layer(proj, self._att(p + "i.b"), self._att(p + "f.b"), self._att(p + "norm"), mpk.attach_input(st["memory"], name=p + "memory"),
                        mpk.attach_input(st["normaliser"], name=p + "normaliser"), self._buf("readout", v, float32), out,
                        heads=m.heads, dim=m.dim, vdim=m.vdim, q_col=0, k_col=qk, v_col=2 * qk, gate_col=2 * qk + v,
                        i_col=2 * qk + 2 * v, f_col=2 * qk + 2 * v + m.heads, gate_cap=m.gate_cap, eps=self.eps, q_scale=m.dim ** -0.5)
        return self._sublayer(out, p + "o", [sd[p + "o"]])

    def _gated(self, x: DTensor, p: str, ff: int, activation: str) -> DTensor:
        """down(act(gate x) * (up x)) for weights `p`gate / up / down."""
        sd, mid = self.sd, self._buf("ff", self._kpad(round_up(ff, 2)), self.act)
        even = lambda w: torch.nn.functional.pad(w, (0, 0, 0, ff % 2))
        w = self._attach(p + "gate_up", lambda: self._pad_k(self.mpk.interleave_gated(even(sd[p + "gate"]), even(sd[p + "up"]))))
        self._linear(x, w, mid, activation=activation)
        return self._sublayer(mid, p + "down", [torch.nn.functional.pad(sd[p + "down"], (0, ff % 2))])

    def _routing(self, experts: int, top: int) -> Tuple[DTensor, DTensor, DTensor]:
        """(expert weights, routing table, active list) a routing layer fills."""
        weights = self._buf("expert_weights", top, float32)
        key = ("routing", (experts,))
        if key not in self._buffers:
            self._buffers[key] = (self.mpk.new_tensor(dims=(experts, self.mpk.max_num_batched_tokens), dtype=int32, name=f"routing_{experts}"),
                                  self.mpk.new_tensor(dims=(experts + 1,), dtype=int32, name=f"active_{experts}"))
        return (weights, *self._buffers[key])

    def _experts(self, h: DTensor, routing: Tuple[DTensor, DTensor, DTensor], first: DTensor, second: DTensor, ff: int, top: int,
                 activation: str) -> DTensor:
        """Outputs [tokens, slots, width] of the chosen experts: second(act(first h)), `ff` columns in between (padded)."""
        grid = dict(grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
        mid = self._buf("expert_mid", (top, ff), self.act)
        self.mpk.moe_w13_linear_layer(h, first, *routing[1:], mid, **grid, activation=activation)
        out = self._buf("expert_out", (top, self.width), float32)
        self.mpk.moe_w2_linear_layer(mid, second, *routing[1:], out, **grid)
        return out

    def _rotary(self, base: float, dims: int, scaling: Optional[RotaryScaling] = None) -> Tuple[DTensor, DTensor]:
        key = (base, dims, scaling)
        if key not in self._tables:
            dev = self.sd["embed"].device
            cos, sin = rotary_tables(base, dims, self.mpk.max_seq_length, dev, scaling)
            n = len(self._tables)
            self._tables[key] = (self.mpk.attach_input(cos, name=f"cos_{n}"), self.mpk.attach_input(sin, name=f"sin_{n}"))
        return self._tables[key]

    def _head(self, h: DTensor, table: DTensor, vocab: int, sampling_seed: Optional[int], **linear):
        """Logits from the normed stream, and the layers that choose the next token."""
        mpk, mbt = self.mpk, self.mpk.max_num_batched_tokens
        self.logits = mpk.new_tensor(dims=(mbt, vocab), dtype=float32, name="logits")
        self._linear(h, table, self.logits, **linear)
        out = mpk.attach_input(mpk.meta_tensors["output_tokens"], name="output_token")
        if sampling_seed is not None:
            mpk.sampling_sm100_layer(logits=self.logits, output=out, grid_dim=(mbt, 1, 1), block_dim=(256, 1, 1),
                                     seed=sampling_seed)
            return
        parts = max(1, min(mpk.num_workers, vocab // 64))
        part_v = mpk.new_tensor(dims=(mbt, parts), dtype=float32, name="argmax_part_value")
        part_i = mpk.new_tensor(dims=(mbt, parts), dtype=int64, name="argmax_part_index")
        mpk.argmax_partial_layer(input=self.logits, output=(part_v, part_i), grid_dim=(parts, 1, 1), block_dim=(128, 1, 1))
        mpk.argmax_reduce_layer(input=(part_v, part_i), output=out, grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
