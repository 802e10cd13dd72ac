"""Bebuzen decoder on a `PersistentKernel`: configuration, weight preparation, recurrent state and layer sequence.

A float32 residual stream that the sublayers read as it is; a norm on every sublayer's output, which joins the stream times a
factor.  Mixers:

  mamba1       [x | z] in one linear -> short convolution -> [step sizes' low-rank part | B | C] linear -> selective scan with
               its gate -> output linear
  attention    differential attention: [q | k | v] in one linear -> short convolution over all of them -> norms, rotation, cache
               rows that hold both maps' keys -> windowed attention of both maps over the same values -> their difference ->
               output linear.  A layer may read the keys and values of an earlier one; it then has queries only
  attention_2  [q | k | v] in one linear -> norms, rotation, cache rows -> windowed attention that keeps the first tokens and has
               one in its denominator -> output linear

and feed-forwards: dense with a gated silu, or a mixture of squared-relu experts (softmax routing; the experts' weighted sum joins
the shared expert in the next norm's task).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..mpk import register_model_builder
from ..persistent_kernel import DTensor, float32
from .hybrid import HybridBuilder, HybridModelConfig, RotaryScaling, round_up


@dataclass(frozen=True)
class MambaSpec:
    inner: int
    state: int
    dt_rank: int
    taps: int


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_base: float
    rot_dims: int
    scaling: Optional[RotaryScaling]
    scale: float
    window: int                       # 0: every earlier position is seen
    keep_first: int

    MAPS = 1

    @property
    def q_rows(self) -> int:
        return self.heads * self.MAPS * self.dim

    @property
    def k_rows(self) -> int:
        return self.kv_heads * self.MAPS * self.dim

    @property
    def v_rows(self) -> int:
        return self.kv_heads * self.vdim


@dataclass(frozen=True)
class DiffAttentionSpec(AttentionSpec):
    diff: float = 0.0
    taps: int = 1
    kv_from: Optional[int] = None     # layer whose keys and values are read

    MAPS = 2


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    scale: float
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                # MambaSpec, AttentionSpec or DiffAttentionSpec
    ff: Any                   # width of a dense feed-forward, MoeSpec, or None: the layer has none


@dataclass(frozen=True)
class BebuzenConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: Tuple[LayerSpec, ...]

    @staticmethod
    def _mixer(n: int, entry: Dict[str, Any]):
        m = entry["mixer"]
        if entry["type"] == "mamba1":
            return MambaSpec(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
        if entry["type"] not in ("attention", "attention_2"):
            raise ValueError(f"layer {n}: unknown mixer {entry['type']!r}")
        rot, mask = m["rot"], m.get("mask") or {}
        s = rot.get("scaling")
        kw = dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), rot_base=float(rot["base"]),
                  rot_dims=int(rot["dims"]), scale=float(m["scale"]), window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0),
                  scaling=RotaryScaling(*(float(s[k]) for k in ("factor", "low", "high", "original"))) if s else None)
        if entry["type"] == "attention_2":
            spec = AttentionSpec(**kw)
        else:
            spec = DiffAttentionSpec(**kw, diff=float(m["diff"]), taps=int(m["conv"]), kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        if spec.heads % spec.kv_heads or spec.rot_dims % 2 or spec.rot_dims > spec.dim:
            raise ValueError(f"layer {n}: {spec.heads} heads over {spec.kv_heads}, {spec.rot_dims} of {spec.dim} dimensions rotated")
        return spec

    @staticmethod
    def _ff(n: int, mlp: Optional[Dict[str, Any]]):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return int(mlp["ff"])
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {n}: unknown feed-forward {mlp['kind']!r}")
        r, shared = mlp["router"], mlp.get("shared")
        spec = MoeSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), float(r.get("scale", 1.0)), int(shared["ff"]) if shared else None)
        if not 1 <= spec.top <= spec.experts:
            raise ValueError(f"layer {n}: {spec.top} of {spec.experts} experts")
        return spec

    @classmethod
    def from_dict(cls, c: Dict[str, Any]) -> "BebuzenConfig":
        layers = tuple(LayerSpec(cls._mixer(n, e), cls._ff(n, e.get("mlp"))) for n, e in enumerate(c["layers"]))
        for n, layer in enumerate(layers):
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            src = layers[j].mixer if 0 <= j < n else None
            if not isinstance(src, DiffAttentionSpec) or src.kv_from is not None or \
                    any(getattr(src, f) != getattr(layer.mixer, f) for f in ("kv_heads", "dim", "vdim")):
                raise ValueError(f"layer {n}: keys and values of layer {j}, which has none of this layer's sizes")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c.get("residual_mult", 1.0)), layers)

    @classmethod
    def from_checkpoint(cls, path: str) -> "BebuzenConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))


def allocate_state(c: BebuzenConfig, *, slots: int, max_num_pages: int, page_size: int, dtype: torch.dtype, device,
                   num_workers: int) -> List[Dict[str, torch.Tensor]]:
    """Per layer: what a sequence leaves behind.  Keys (both maps of a head side by side) and values are paged [pages, page,
    kv heads, size rounded up to 8] in the activation type; carried convolution inputs and scan states are float32 and indexed by
    state slot.  A layer that reads another layer's keys and values has only the convolution's inputs."""
    z32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=device)
    out = []
    for layer in c.layers:
        m, st = layer.mixer, {}
        if isinstance(m, MambaSpec):
            st["conv"], st["scan"] = z32(slots, max(m.taps - 1, 1), m.inner), z32(slots, m.inner, round_up(m.state, 4))
        else:
            own = getattr(m, "kv_from", None) is None
            if own:
                for name, size in (("k", m.MAPS * m.dim), ("v", m.vdim)):
                    st[name] = torch.zeros(max_num_pages, page_size, m.kv_heads, round_up(size, 8), dtype=dtype, device=device)
            if isinstance(m, DiffAttentionSpec):
                st["conv"] = z32(slots, max(m.taps - 1, 1), m.q_rows + (m.k_rows + m.v_rows if own else 0))
        out.append(st)
    return out


BebuzenModelConfig = HybridModelConfig


@register_model_builder("bebuzen")
class BebuzenBuilder(HybridBuilder):
    # -- mixers: `h` is the stream in the activation type; return the mixer's float32 output
    def _mamba(self, n: int, p: str, m: MambaSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd = self.mpk, self.sd
        proj = self._buf("proj", 2 * m.inner, float32)
        self._linear(h, self._weight(p + "in.padded", [sd[p + "in"]]), proj)
        u = self._buf("conv_out", m.inner, float32)
        # the [steps | B | C] linear reads the convolution in the activation type, the recurrence in 32-bit
        operand = u if self.act is float32 else self._buf("conv_operand", self._kpad(m.inner), self.act)
        mpk.short_conv_layer(proj, self._att(p + "conv"), mpk.attach_input(st["conv"], name=p + "conv_state"), u,
                             bias=self._att(p + "conv.b"), activation="silu", copy=None if operand is u else operand)
        low = self._buf("scan_low", m.dt_rank + 2 * m.state, float32)
        self._linear(operand, self._weight(p + "x.padded", [sd[p + "x"]]), low)
        out = self._buf("mixed", self._kpad(m.inner), self.act)
        mpk.selective_scan_layer(u, low, proj, self._att(p + "dt"), self._att(p + "dt.b"), self._att(p + "A_log"), self._att(p + "D"),
                                 mpk.attach_input(st["scan"], name=p + "scan_state"), out, rank=m.dt_rank, n=m.state, gate_col=m.inner)
        return self._sublayer(out, p + "o", [sd[p + "o"]])

    def _attention(self, n: int, p: str, m: AttentionSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd = self.mpk, self.sd
        diff = m if isinstance(m, DiffAttentionSpec) else None
        names = ("q", "k", "v") if diff is None or diff.kv_from is None else ("q",)
        cols = m.q_rows + (m.k_rows + m.v_rows if len(names) > 1 else 0)
        join = lambda suffix: self._attach(p + "".join(names) + suffix, lambda: torch.cat([sd[p + nm + suffix] for nm in names]))
        proj = self._buf("proj", cols, float32)
        weight = self._weight(p + "".join(names), [sd[p + nm] for nm in names])
        if diff is None:
            self._linear(h, weight, proj, bias=join(".b"))
        else:   # the biases enter with the convolution's inputs
            self._linear(h, weight, proj)
            conv = self._buf("conv_out", cols, float32)
            mpk.short_conv_layer(proj, join(".conv"), mpk.attach_input(st["conv"], name=p + "conv_state"), conv, input_bias=join(".b"))
            proj = conv
        if len(names) > 1:
            self._kv[n] = tuple(mpk.attach_input(st[nm], name=f"{p}{nm}_cache") for nm in ("k", "v"))
        k_cache, v_cache = self._kv[n if len(names) > 1 else diff.kv_from]
        own = (k_cache, v_cache) if len(names) > 1 else (None, None)
        q = self._buf("q", m.heads * m.MAPS * k_cache.dim(3), self.act)
        cos, sin = self._rotary(m.rot_base, m.rot_dims, m.scaling)
        mpk.qkv_append_layer(proj, q, *own, cos, sin, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, q_col=0, k_col=m.q_rows,
                             v_col=m.q_rows + m.k_rows, rot_dims=m.rot_dims, eps=self.eps, q_norm=self._att(p + "q.norm"),
                             k_norm=self._att(p + "k.norm") if own[0] is not None else None, interleaved=diff is None, maps=m.MAPS)
        mixed = self._buf("mixed", self._kpad(m.heads * m.vdim), self.act)
        out = mixed if diff is None else self._buf("maps", 2 * m.heads * m.vdim, float32)
        mpk.ext_attention_layer(q, k_cache, v_cache, out, heads=m.heads * m.MAPS, kv_heads=m.kv_heads, vdim=m.vdim, scale=m.scale,
                                sink=diff is None, window=m.window, keep_first=m.keep_first)
        if diff is None:
            return self._sublayer(mixed, p + "o", [sd[p + "o"]], bias=self._att(p + "o.b"))
        dot = lambda a, b: math.exp(float((sd[p + a].double() * sd[p + b].double()).sum()))
        mpk.diff_combine_layer(out, mixed, heads=m.heads, vdim=m.vdim, lam=dot("lq1", "lk1") - dot("lq2", "lk2") + diff.diff,
                               factor=1.0 - diff.diff, eps=self.eps)
        return self._sublayer(mixed, p + "o", [sd[p + "o"]])

    # -- feed-forwards: return the terms whose normed sum joins the stream (arguments of residual_norm_layer)
    def _moe(self, h: DTensor, p: str, m: MoeSpec) -> Dict[str, Any]:
        mpk, sd = self.mpk, self.sd
        E, F = m.experts, self._kpad(m.ff)
        logits = self._buf("router", E, float32)
        self._linear(h, self._weight(p + "router.padded", [sd[p + "router"]]), logits)
        routing = self._routing(E, m.top)
        mpk.moe_topk_softmax_routing_layer(logits, routing, grid_dim=(1, 1, 1), block_dim=(128, 1, 1), renormalize=False, scale=m.scale)
        y = None
        if m.shared_ff is not None:
            mid = self._buf("ff", self._kpad(m.shared_ff), self.act)
            self._linear(h, self._weight(p + "shared.up.padded", [sd[p + "shared.up"]]), mid, activation="relu2")
            y = self._sublayer(mid, p + "shared.down", [sd[p + "shared.down"]])
        first = self._attach(p + "experts.up", lambda: torch.stack([self._pad_k(sd[f"{p}e{e}.up"]) for e in range(E)]))
        second = self._attach(p + "experts.down", lambda: torch.stack([self._pad_k(sd[f"{p}e{e}.down"]) for e in range(E)]))
        return {"y": y, "experts": (self._experts(h, routing, first, second, F, m.top, "relu2"), routing[0])}

    def build_from_config(self, mc: BebuzenModelConfig):
        mpk, c, sd = self.mpk, mc.config, mc.state_dict
        self._begin(mc)
        self._kv: Dict[int, Tuple[DTensor, DTensor]] = {}          # layer -> its key and value caches
        if tuple(sd["embed"].shape) != (c.vocab, c.width) or tuple(sd["head"].shape) != (c.vocab, c.width):
            raise ValueError(f"embedding {tuple(sd['embed'].shape)}, head {tuple(sd['head'].shape)}, configuration {(c.vocab, c.width)}")
        # two stream buffers in turn: a norm's task reads one and writes the other
        x, other = self._buf("stream", c.width, float32), self._buf("stream_b", c.width, float32)
        h = self._buf("operand", self._kpad(c.width), self.act)
        mpk.embed_layer(input=mpk.attach_input(mpk.meta_tensors["input_tokens"], name="input_token"), weight=self._att("embed"),
                        output=x, grid_dim=(1, 1, 1), block_dim=(128, 1, 1), input_source=1)
        mpk.residual_norm_layer(x, output=h, eps=c.eps)

        def join(name: str, terms: Dict[str, Any], closing: Optional[DTensor] = None):
            """The sublayer's normed output joins the stream; `h` is the new stream, or its norm with the weight `closing`."""
            nonlocal x, other
            mpk.residual_norm_layer(x, post_weight=self._att(name), norm_weight=closing, output=h, eps=c.eps, x_out=other,
                                    post_factor=c.residual_mult, **terms)
            x, other = other, x

        sublayers = [(n, part) for n, layer in enumerate(c.layers) for part in ("mixer", "ff") if part == "mixer" or layer.ff is not None]
        for n, part in sublayers:
            layer, p = c.layers[n], f"l{n}."
            if part == "mixer":
                mixer = self._mamba if isinstance(layer.mixer, MambaSpec) else self._attention
                terms = {"y": mixer(n, p + "mix.", layer.mixer, mc.state[n], h)}
            elif isinstance(layer.ff, MoeSpec):
                terms = self._moe(h, p + "mlp.", layer.ff)
            else:
                terms = {"y": self._gated(h, p + "mlp.", layer.ff, "gated_silu")}
            join(p + ("norm1" if part == "mixer" else "norm2"), terms, self._att("final.norm") if (n, part) == sublayers[-1] else None)
        self.hidden = x
        self._head(h, self._weight("head", [sd["head"]]), c.vocab, mc.sampling_seed)
