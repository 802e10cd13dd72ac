"""Palarax decoder on a `PersistentKernel`: configuration, weight preparation, recurrent state and layer sequence.

A float32 residual stream with a norm before and after every sublayer.  Two kinds of mixers:

  mlstm     [q | k | v | gate | i | f] in one linear -> matrix-memory recurrence with its head norm and gate -> output linear
  parallel  [q | k | y | x] in one linear -> { rotation, unit norms, cache rows -> attention with soft cap and sink } beside
            { short convolution -> gated diagonal recurrence }; both write their columns of one buffer, already scaled,
            and one linear over [left.o | right.o] adds them up

and a squared-relu feed-forward.  Linear weights of the bf16 graph are padded to a multiple of 64 input columns (the
tensor path's k granularity), the activation buffers in front of them likewise: the padding columns stay zero.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..mpk import register_model_builder
from ..persistent_kernel import DTensor, float32
from .hybrid import HybridBuilder, HybridModelConfig, MlstmSpec, round_up


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_base: float
    rot_dims: int
    scale: float
    softcap: float


@dataclass(frozen=True)
class RgLruSpec:
    width: int
    blocks: int
    taps: int


@dataclass(frozen=True)
class ParallelSpec:
    left: AttentionSpec
    right: RgLruSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                # MlstmSpec or ParallelSpec
    ff: Optional[int]         # width of the feed-forward, None: the layer has none


@dataclass(frozen=True)
class PalaraxConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerSpec, ...]

    DECAY = 8.0               # constant of the diagonal recurrence's log decay

    @classmethod
    def from_dict(cls, c: Dict[str, Any]) -> "PalaraxConfig":
        layers = []
        for n, entry in enumerate(c["layers"]):
            m = entry["mixer"]
            if entry["type"] == "mlstm":
                mixer = MlstmSpec.from_dict(m)
            elif entry["type"] == "parallel":
                l, r = m["left"], m["right"]
                left = AttentionSpec(int(l["heads"]), int(l["kv_heads"]), int(l["dim"]), int(l["vdim"]),
                                     float(l["rot"]["base"]), int(l["rot"]["dims"]), float(l["scale"]), float(l["softcap"]))
                right = RgLruSpec(int(r["width"]), int(r["blocks"]), int(r["conv"]))
                if left.heads % left.kv_heads or left.rot_dims % 2 or left.rot_dims > left.dim or right.width % right.blocks:
                    raise ValueError(f"layer {n}: sizes do not divide")
                if left.vdim != left.dim:
                    raise ValueError(f"layer {n}: keys serve as values, but dim {left.dim} != vdim {left.vdim}")
                mixer = ParallelSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))
            else:
                raise ValueError(f"layer {n}: unknown mixer {entry['type']!r}")
            mlp = entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {n}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(mixer, None if mlp is None else int(mlp["ff"])))
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), tuple(layers))

    @classmethod
    def from_checkpoint(cls, path: str) -> "PalaraxConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))


def allocate_state(c: PalaraxConfig, *, slots: int, max_num_pages: int, page_size: int, dtype: torch.dtype, device,
                   num_workers: int) -> List[Dict[str, torch.Tensor]]:
    """Per layer: what a sequence leaves behind.  Attention caches are paged [pages, page, kv heads, head size rounded up
    to 8] in the activation type; recurrent state is float32 and indexed by state slot."""
    z32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=device)
    out = []
    for layer in c.layers:
        m = layer.mixer
        if isinstance(m, MlstmSpec):
            out.append(m.state(slots, num_workers, device))
        else:
            shape = lambda d: (max_num_pages, page_size, m.left.kv_heads, round_up(d, 8))
            out.append({"k": torch.zeros(shape(m.left.dim), dtype=dtype, device=device),
                        "v": torch.zeros(shape(m.left.vdim), dtype=dtype, device=device),
                        "conv": z32(slots, max(m.right.taps - 1, 1), m.right.width),
                        "diag": z32(slots, m.right.width)})
    return out


PalaraxModelConfig = HybridModelConfig


@register_model_builder("palarax")
class PalaraxBuilder(HybridBuilder):
    # -- mixers: `h` is the normed input; return the mixer's float32 output
    def _parallel(self, p: str, m: ParallelSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd = self.mpk, self.sd
        l, r, pl, pr = m.left, m.right, p + "left.", p + "right."
        nq, nk = l.heads * l.dim, l.kv_heads * l.dim
        k_col, y_col, x_col = nq, nq + nk, nq + nk + r.width
        proj = self._buf("proj", x_col + r.width, float32)
        self._linear(h, self._weight(p + "qkyx", [sd[pl + "q"], sd[pl + "k"], sd[pr + "y"], sd[pr + "x"]]), proj)
        left_out = l.heads * l.vdim
        mixed = self._buf("mixed", self._kpad(left_out + r.width), self.act)
        # right branch, first half: a worker runs its tasks in layer order, so what is short and early in both branches comes
        # first, and no branch waits behind the other's long task
        u = self._buf("conv_out", r.width, float32)
        mpk.short_conv_layer(proj, self._att(pr + "conv"), mpk.attach_input(st["conv"], name=pr + "conv_state"), u,
                             input_bias=self._att(pr + "x.b"), bias=self._att(pr + "conv.b"), in_col=x_col)
        # left branch
        kc, vc = mpk.attach_input(st["k"], name=pl + "k_cache"), mpk.attach_input(st["v"], name=pl + "v_cache")
        q = self._buf("q", l.heads * kc.dim(3), self.act)
        cos, sin = self._rotary(l.rot_base, l.rot_dims)
        mpk.qkv_append_layer(proj, q, kc, vc, cos, sin, heads=l.heads, kv_heads=l.kv_heads, dim=l.dim, vdim=l.vdim, q_col=0,
                             k_col=k_col, v_col=k_col, rot_dims=l.rot_dims, unit_norm=True, eps=self.eps)
        mpk.ext_attention_layer(q, kc, vc, mixed, heads=l.heads, kv_heads=l.kv_heads, vdim=l.vdim, scale=l.scale,
                                softcap=l.softcap, sink=True, out_col=0, out_scale=m.left_scale)
        # right branch, second half
        mpk.rglru_layer(u, proj, self._att(pr + "y.b"), self._att(pr + "ra"), self._att(pr + "ra.b"), self._att(pr + "ri"),
                        self._att(pr + "ri.b"), self._att(pr + "lam"), mpk.attach_input(st["diag"], name=pr + "state"), mixed,
                        y_col=y_col, out_col=left_out, out_scale=m.right_scale, decay=PalaraxConfig.DECAY)
        y = self._buf("sublayer", self.width, float32)
        self._linear(mixed, self._weight(p + "o", [sd[pl + "o"], sd[pr + "o"]], dim=1), y)
        return y

    def build_from_config(self, mc: PalaraxModelConfig):
        mpk, c, sd = self.mpk, mc.config, mc.state_dict
        self._begin(mc)
        if tuple(sd["embed"].shape) != (c.vocab, c.width):
            raise ValueError(f"embedding is {tuple(sd['embed'].shape)}, configuration says {(c.vocab, c.width)}")
        table = self._weight("embed", [sd["embed"]])
        # two stream buffers in turn: a norm reads one and writes the other
        x, other = self._buf("stream", c.width, float32), self._buf("stream_b", c.width, float32)
        h = self._buf("normed", self._kpad(c.width), self.act)
        mpk.embed_layer(input=mpk.attach_input(mpk.meta_tensors["input_tokens"], name="input_token"), weight=table, output=x,
                        grid_dim=(1, 1, 1), block_dim=(128, 1, 1), input_source=1)

        def norm(y: Optional[DTensor], post: Optional[str], nxt: str):
            nonlocal x, other
            mpk.residual_norm_layer(x, y, self._att(post) if post else None, self._att(nxt), h, eps=c.eps, zero_centered=True,
                                    x_out=other if y is not None else None)
            if y is not None:
                x, other = other, x

        # a sublayer's closing norm and the next one's opening norm are one task
        y, post = None, None
        for n, layer in enumerate(c.layers):
            p = f"l{n}."
            norm(y, post, p + "norm1")
            mixer = self._mlstm if isinstance(layer.mixer, MlstmSpec) else self._parallel
            y, post = mixer(p + "mix.", layer.mixer, mc.state[n], h), p + "norm1b"
            if layer.ff is not None:
                norm(y, post, p + "norm2")
                mid = self._buf("ff", self._kpad(layer.ff), self.act)
                # (a padded buffer is wider than the weight has rows: the linear fills its leading columns)
                self._linear(h, self._weight(p + "mlp.up.padded", [sd[p + "mlp.up"]]), mid, activation="relu2")
                y, post = self._buf("sublayer", c.width, float32), p + "norm2b"
                self._linear(mid, self._weight(p + "mlp.down.padded", [sd[p + "mlp.down"]]), y)
        norm(y, post, "final.norm")
        self.hidden = x
        self._head(h, table, c.vocab, mc.sampling_seed)
