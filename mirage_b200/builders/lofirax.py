"""Lofirax decoder on a `PersistentKernel`: configuration, weight preparation, recurrent state and layer sequence.

A float32 residual stream with a layer norm in front of every sublayer; a range of layers may run several times.  Mixers:

  gla     [q | k | v | gate | a1] in one linear -> gated linear attention with its head norm and gate -> output linear
  latent  two linears over the normed stream: the unrotated query parts, and [rotated query parts | latent | shared key part].
          Keys and values are never expanded: a grouped linear per head takes the unrotated queries into the latent space
          (W_uk^T q) while the cache rows are written, attention runs over the latent rows as one shared key / value head,
          another grouped linear takes its output from the latent space to the values (W_uv o) -> output linear

and feed-forwards: dense with a gated tanh-gelu, or a mixture of experts (group-limited sigmoid routing; the experts' weighted sum
and the gated shared expert join the stream in the next norm's task).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..mpk import register_model_builder
from ..persistent_kernel import DTensor, float32
from .hybrid import HybridBuilder, HybridModelConfig, k_padded, round_up


@dataclass(frozen=True)
class GlaSpec:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int                  # unrotated query / key size of a head
    rot_dim: int
    vdim: int
    kv_rank: int
    rot_base: float
    scale: float

    def row(self, dtype: torch.dtype) -> int:
        """Width of a cache row: latent and rotated part, and the latent's padding where values are read with it."""
        return round_up(max(self.kv_rank + self.rot_dim, k_padded(self.kv_rank, dtype)), 8)


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    groups: int
    keep: int
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                # GlaSpec or LatentSpec
    ff: Any                   # width of a dense feed-forward, MoeSpec, or None: the layer has none


@dataclass(frozen=True)
class LofiraxConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    logit_softcap: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Tuple[int, int, int]]      # (start, stop, times)

    @staticmethod
    def _mixer(n: int, entry: Dict[str, Any]):
        m = entry["mixer"]
        if entry["type"] == "gla":
            return GlaSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))
        if entry["type"] != "latent_attention":
            raise ValueError(f"layer {n}: unknown mixer {entry['type']!r}")
        spec = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                          float(m["rot"]["base"]), float(m["scale"]))
        if int(m["rot"]["dims"]) != spec.rot_dim or spec.rot_dim % 2:
            raise ValueError(f"layer {n}: the rotary part has {spec.rot_dim} dimensions, the rotation {m['rot']['dims']}")
        return spec

    @staticmethod
    def _ff(n: int, mlp: Optional[Dict[str, Any]]):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return int(mlp["ff"])
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {n}: unknown feed-forward {mlp['kind']!r}")
        r = mlp["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        spec = MoeSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(g["count"]), int(g["keep"]),
                       int(shared["ff"]) if shared else None)
        if spec.experts % spec.groups or not 1 <= spec.keep <= spec.groups or spec.top > spec.keep * (spec.experts // spec.groups):
            raise ValueError(f"layer {n}: {spec.experts} experts, {spec.groups} groups, {spec.keep} kept, {spec.top} chosen")
        return spec

    @classmethod
    def from_dict(cls, c: Dict[str, Any]) -> "LofiraxConfig":
        layers = tuple(LayerSpec(cls._mixer(n, e), cls._ff(n, e.get("mlp"))) for n, e in enumerate(c["layers"]))
        loop = c.get("loop")
        if loop:
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ValueError(f"loop {loop} over {len(layers)} layers")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float((c.get("embedding") or {}).get("scale", 1.0)),
                   float(c.get("logit_softcap") or 0.0), layers, loop or None)

    @classmethod
    def from_checkpoint(cls, path: str) -> "LofiraxConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) in execution order; the pass's number is given with its first layer, None elsewhere."""
        start, stop, times = self.loop or (0, 0, 0)
        out: List[Tuple[int, Optional[int]]] = [(n, None) for n in range(start)]
        for t in range(times):
            out += [(n, t if n == start else None) for n in range(start, stop)]
        return out + [(n, None) for n in range(stop, len(self.layers))]


def allocate_state(c: LofiraxConfig, *, slots: int, max_num_pages: int, page_size: int, dtype: torch.dtype, device,
                   num_workers: int) -> List[Dict[str, torch.Tensor]]:
    """Per layer run: what a sequence leaves behind.  Latent rows are paged [pages, page, 1, row] in the activation type; the
    matrix memories are float32 and indexed by state slot."""
    out = []
    for n, _ in c.runs():
        m = c.layers[n].mixer
        if isinstance(m, GlaSpec):
            out.append({"memory": torch.zeros(slots, m.heads, m.dim, round_up(m.vdim, 4), dtype=torch.float32, device=device)})
        else:
            out.append({"latent": torch.zeros(max_num_pages, page_size, 1, m.row(dtype), dtype=dtype, device=device)})
    return out


LofiraxModelConfig = HybridModelConfig


@register_model_builder("lofirax")
class LofiraxBuilder(HybridBuilder):
    # -- mixers: `h` is the normed input, `run` names the layer run; return the mixer's float32 output
    def _gla(self, p: str, run: str, m: GlaSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd = self.mpk, self.sd
        qk, v, rank = m.heads * m.dim, m.heads * m.vdim, sd[p + "a1"].shape[0]
        proj = self._buf("proj", 2 * qk + 2 * v + rank, float32)
        self._linear(h, self._weight(p + "qkvga", [sd[p + n] for n in ("q", "k", "v", "g", "a1")]), proj)
        out = self._buf("mixed", self._kpad(v), self.act)
        chunks = mpk.mlstm_chunks(mpk.num_workers, mpk.max_num_batched_requests, m.heads, m.dim, m.vdim)
        mpk.gla_layer(proj, self._att(p + "a2"), self._att(p + "a2.b"), self._att(p + "norm"),
                      mpk.attach_input(st["memory"], name=run + "memory"), self._buf("readout", v, float32), out, heads=m.heads,
                      dim=m.dim, vdim=m.vdim, q_col=0, k_col=qk, v_col=2 * qk, gate_col=2 * qk + v, a1_col=2 * qk + 2 * v,
                      tau=m.tau, eps=self.eps, q_scale=m.dim ** -0.5, chunks=chunks)
        return self._sublayer(out, p + "o", [sd[p + "o"]])

    def _latent(self, p: str, run: str, m: LatentSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd, pad = self.mpk, self.sd, torch.nn.functional.pad
        H, dim, rot, rank = m.heads, m.dim, m.rot_dim, m.kv_rank
        dim_p, rank_p, row = self._kpad(dim), self._kpad(rank), m.row(self.dtype)
        by_head = sd[p + "q"].view(H, dim + rot, self.width)
        q_un = self._buf("q_unrotated", H * dim_p, self.act)
        self._linear(h, self._attach(p + "q.unrotated", lambda: self._pad_k(pad(by_head[:, :dim], (0, 0, 0, dim_p - dim)).flatten(0, 1))), q_un)
        proj = self._buf("proj", (H + 1) * rot + rank, float32)
        self._linear(h, self._weight(p + "q.rotated.dkv", [by_head[:, dim:].flatten(0, 1), sd[p + "dkv"]]), proj)
        q = self._buf("q_latent", H * row, self.act)
        cache = mpk.attach_input(st["latent"], name=run + "latent")
        uk = self._attach(p + "uk.absorbed", lambda: self._pad_k(sd[p + "uk"].view(H, dim, rank).transpose(1, 2)))
        mpk.grouped_linear_layer(q_un, uk, q, in_stride=dim_p, out_stride=row)
        cos, sin = self._rotary(m.rot_base, rot)
        mpk.latent_append_layer(proj, self._att(p + "dkv.norm"), q, cache, cos, sin, heads=H, rank=rank, rot_dims=rot, q_col=0,
                                kv_col=H * rot, eps=self.eps)
        mixed = self._buf("latent_out", H * rank_p, self.act)
        mpk.ext_attention_layer(q, cache, cache, mixed, heads=H, kv_heads=1, vdim=rank_p, scale=m.scale, sinks=self._att(p + "sink"),
                                separate_merge=True)
        values = self._buf("mixed", self._kpad(H * m.vdim), self.act)
        uv = self._attach(p + "uv.heads", lambda: self._pad_k(sd[p + "uv"].view(H, m.vdim, rank)))
        mpk.grouped_linear_layer(mixed, uv, values, in_stride=rank_p, out_stride=m.vdim)
        return self._sublayer(values, p + "o", [sd[p + "o"]])

    # -- feed-forwards: return the terms that join the stream (arguments of residual_norm_layer)
    def _moe(self, h: DTensor, p: str, m: MoeSpec) -> Dict[str, Any]:
        mpk, sd = self.mpk, self.sd
        E, F = m.experts, self._kpad(round_up(m.ff, 2))
        shared = m.shared_ff is not None
        logits = self._buf("router", E + int(shared), float32)
        self._linear(h, self._weight(p + "router.sg", [sd[p + "router"]] + ([sd[p + "shared.sg"]] if shared else [])), logits)
        routing = self._routing(E, m.top)
        grid = dict(grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
        mpk.moe_topk_sigmoid_routing_layer(logits, self._attach(p + "correction.f32", lambda: sd[p + "correction"].float()),
                                           routing, **grid, num_groups=m.groups, topk_group=m.keep,
                                           routed_scaling_factor=1.0, keep_logits=True)
        y = self._gated(h, p + "shared.", m.shared_ff, "gated_silu") if shared else None
        rows = lambda n, r: torch.nn.functional.pad(n, (0, 0, 0, r - n.shape[0]))
        w13 = self._attach(p + "experts.gate_up", lambda: torch.stack(
            [self._pad_k(mpk.interleave_gated(rows(sd[f"{p}e{e}.gate"], F), rows(sd[f"{p}e{e}.up"], F))) for e in range(E)]))
        w2 = self._attach(p + "experts.down", lambda: torch.stack(
            [torch.nn.functional.pad(sd[f"{p}e{e}.down"], (0, F - m.ff)) for e in range(E)]))
        out = self._experts(h, routing, w13, w2, F, m.top, "gated_silu")
        return {"y": y, "experts": (out, routing[0]), "y_gate": (logits, E) if shared else None}

    def build_from_config(self, mc: LofiraxModelConfig):
        mpk, c, sd = self.mpk, mc.config, mc.state_dict
        self._begin(mc)
        if tuple(sd["embed"].shape) != (c.vocab, c.width) or tuple(sd["head"].shape) != (c.vocab, c.width):
            raise ValueError(f"embedding {tuple(sd['embed'].shape)}, head {tuple(sd['head'].shape)}, configuration {(c.vocab, c.width)}")
        # the embedding output stays for the passes of the loop; two further stream buffers in turn: a norm reads one and writes the other
        embedded = self._buf("embedded", c.width, float32)
        streams = [self._buf("stream", c.width, float32), self._buf("stream_b", c.width, float32)]
        x = embedded
        h = self._buf("normed", self._kpad(c.width), self.act)
        mpk.embed_layer(input=mpk.attach_input(mpk.meta_tensors["input_tokens"], name="input_token"), weight=self._att("embed"),
                        output=x, grid_dim=(1, 1, 1), block_dim=(128, 1, 1), input_source=1, factor=c.embed_scale)

        def norm(name: str, terms: Dict[str, Any]):
            nonlocal x
            to = streams[0] if x is not streams[0] else streams[1]
            mpk.residual_norm_layer(x, norm_weight=self._att(name), norm_bias=self._att(name + ".b"), output=h, eps=c.eps,
                                    layer_norm=True, x_out=to if terms else None, **terms)
            x = to if terms else x

        terms: Dict[str, Any] = {}       # what the next norm's task adds to the stream first
        for r, (n, t) in enumerate(c.runs()):
            layer, p = c.layers[n], f"l{n}."
            if t is not None:
                terms["added_row"] = self._attach(f"loop.step.{t}", lambda: sd["loop.step"][t].clone())
                if t > 0:
                    terms["added"] = embedded
            norm(p + "norm1", terms)
            mixer = self._gla if isinstance(layer.mixer, GlaSpec) else self._latent
            terms = {"y": mixer(p + "mix.", f"run{r}.", layer.mixer, mc.state[r], h)}
            if layer.ff is not None:
                norm(p + "norm2", terms)
                if isinstance(layer.ff, MoeSpec):
                    terms = self._moe(h, p + "mlp.", layer.ff)
                else:
                    terms = {"y": self._gated(h, p + "mlp.", layer.ff, "gated_gelu_tanh")}
        norm("final.norm", terms)
        self.hidden = x
        cap = dict(activation="softcap", softcap=c.logit_softcap) if c.logit_softcap else {}
        self._head(h, self._weight("head", [sd["head"]]), c.vocab, mc.sampling_seed, **cap)
