"""Ruludra decoder on a `PersistentKernel`: configuration, weight preparation, state and layer sequence.

The stream starts as the sum of a token's embedding, a row for the token and the one before it, and sines and cosines of the position.
Norms before and after every sublayer; behind a layer the stream is replaced by a weighted sum of the embedding output and all layers'
results so far, formed in the task of the layer's closing norm.  Mixers:

  mlstm      matrix-memory recurrence (`HybridBuilder._mlstm`)
  attention  [q | k] in one linear -> norms over all heads, query temperature, cache rows (the keys as projected are the values) ->
             windowed attention with a distance bias -> output linear
  latent     [query latent | latent | gate] in one linear -> norm of the query latent, cache rows of the normed latent -> queries ->
             a grouped linear per head takes them into the latent space (W_uk^T q), windowed attention runs over the latent rows as
             one shared key / value head, another grouped linear takes its output to the values (W_uv o) and multiplies the gate in ->
             output linear.  A layer may read the latents of an earlier one; it then has queries and gate only

and a feed-forward whose activation is a sum of normed powers.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..mpk import register_model_builder
from ..persistent_kernel import DTensor, float32
from .hybrid import HybridBuilder, HybridModelConfig, MlstmSpec, k_padded, round_up


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int                               # 0: every earlier position is seen
    temperature: Optional[Tuple[float, int]]  # (coefficient, positions of a step)


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int
    kv_from: Optional[int]                    # layer whose latents are read

    def row(self, dtype: torch.dtype) -> int:
        """Width of a cache row: the latent, and its padding where values are read with it."""
        return round_up(k_padded(self.kv_rank, dtype), 8)


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                # MlstmSpec, AttentionSpec or LatentSpec
    ff: Optional[int]         # width of the feed-forward, None: the layer has none


@dataclass(frozen=True)
class RuludraConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    bigram: Optional[Tuple[int, int, int]]    # (buckets, multiplier of the previous id, multiplier of the id)
    layers: Tuple[LayerSpec, ...]

    @staticmethod
    def _mixer(n: int, entry: Dict[str, Any]):
        m = entry["mixer"]
        if entry["type"] == "mlstm":
            return MlstmSpec.from_dict(m)
        window = int((m.get("mask") or {}).get("size") or 0)
        if entry["type"] == "attention":
            t = m.get("q_temp")
            spec = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]), window,
                                 (float(t["coef"]), int(t["every"])) if t else None)
            if spec.heads % spec.kv_heads:
                raise ValueError(f"layer {n}: {spec.heads} heads over {spec.kv_heads}")
            if int(m.get("vdim", spec.dim)) != spec.dim:
                raise ValueError(f"layer {n}: keys serve as values, but dim {spec.dim} != vdim {m['vdim']}")
            return spec
        if entry["type"] == "latent_attention":
            j = m.get("kv_from")
            return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]), window,
                              None if j is None else int(j))
        raise ValueError(f"layer {n}: unknown mixer {entry['type']!r}")

    @staticmethod
    def _ff(n: int, mlp: Optional[Dict[str, Any]]) -> Optional[int]:
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {n}: unknown feed-forward {mlp['kind']!r}")
        return None if mlp is None else int(mlp["ff"])

    @classmethod
    def from_dict(cls, c: Dict[str, Any]) -> "RuludraConfig":
        layers = tuple(LayerSpec(cls._mixer(n, e), cls._ff(n, e.get("mlp"))) for n, e in enumerate(c["layers"]))
        for n, layer in enumerate(layers):
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            src = layers[j].mixer if 0 <= j < n else None
            if not isinstance(src, LatentSpec) or src.kv_from is not None or src.kv_rank != layer.mixer.kv_rank:
                raise ValueError(f"layer {n}: no latents of {layer.mixer.kv_rank} in layer {j}")
        b = (c.get("embedding") or {}).get("bigram")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c.get("logit_scale", 1.0)),
                   (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None, layers)

    @classmethod
    def from_checkpoint(cls, path: str) -> "RuludraConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))


def allocate_state(c: RuludraConfig, *, slots: int, max_num_pages: int, page_size: int, dtype: torch.dtype, device,
                   num_workers: int) -> List[Dict[str, torch.Tensor]]:
    """Per layer: what a sequence leaves behind.  Keys, values [pages, page, kv heads, size rounded up to 8] and latent rows [pages,
    page, 1, row] are paged, in the activation type; matrix memories are float32 and indexed by state slot.  A layer that reads another
    one's latents has nothing of its own.  (The previous token, which the embedding needs, is in the scheduler's token table.)"""
    out = []
    for layer in c.layers:
        m = layer.mixer
        pages = lambda heads, size: torch.zeros(max_num_pages, page_size, heads, size, dtype=dtype, device=device)
        if isinstance(m, MlstmSpec):
            out.append(m.state(slots, num_workers, device))
        elif isinstance(m, AttentionSpec):
            out.append({nm: pages(m.kv_heads, round_up(m.dim, 8)) for nm in ("k", "v")})
        else:
            out.append({"latent": pages(1, m.row(dtype))} if m.kv_from is None else {})
    return out


RuludraModelConfig = HybridModelConfig


@register_model_builder("ruludra")
class RuludraBuilder(HybridBuilder):
    # -- mixers: `h` is the normed input; return the mixer's float32 output
    def _attention(self, p: str, m: AttentionSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd = self.mpk, self.sd
        nq, nk = m.heads * m.dim, m.kv_heads * m.dim
        proj = self._buf("proj", nq + nk, float32)
        self._linear(h, self._weight(p + "qk", [sd[p + "q"], sd[p + "k"]]), proj)
        kc, vc = (mpk.attach_input(st[nm], name=f"{p}{nm}_cache") for nm in ("k", "v"))
        q = self._buf("q", m.heads * kc.dim(3), self.act)
        mpk.qkv_append_layer(proj, q, kc, vc, None, None, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.dim, q_col=0, k_col=nq, v_col=nq,
                             rot_dims=0, eps=self.eps, q_norm=self._att(p + "q.norm"), k_norm=self._att(p + "k.norm"), whole_norm=True,
                             temperature=m.temperature)
        mixed = self._buf("mixed", self._kpad(nq), self.act)
        mpk.ext_attention_layer(q, kc, vc, mixed, heads=m.heads, kv_heads=m.kv_heads, vdim=m.dim, scale=m.scale, window=m.window,
                                distance_bias=(self._att(p + "r1"), self._att(p + "r2")))
        return self._sublayer(mixed, p + "o", [sd[p + "o"]])

    def _latent(self, n: int, p: str, m: LatentSpec, st: Dict[str, torch.Tensor], h: DTensor) -> DTensor:
        mpk, sd, pad = self.mpk, self.sd, torch.nn.functional.pad
        H, dim, rank = m.heads, m.dim, m.kv_rank
        dim_p, rank_p, row = self._kpad(dim), self._kpad(rank), m.row(self.dtype)
        names = ("dq", "dkv", "g") if m.kv_from is None else ("dq", "g")
        gate_col = m.q_rank + (rank if m.kv_from is None else 0)
        proj = self._buf("proj", gate_col + H * m.vdim, float32)
        self._linear(h, self._weight(p + "".join(names), [sd[p + nm] for nm in names]), proj)
        low = self._buf("q_low", self._kpad(m.q_rank), self.act)
        mpk.residual_norm_layer(proj, norm_weight=self._att(p + "dq.norm"), output=low, eps=self.eps, columns=m.q_rank)
        if m.kv_from is None:
            self._latents[n] = mpk.attach_input(st["latent"], name=p + "latent")
            mpk.latent_append_layer(proj, self._att(p + "dkv.norm"), None, self._latents[n], None, None, heads=H, rank=rank, rot_dims=0,
                                    q_col=0, kv_col=m.q_rank, eps=self.eps)
        cache = self._latents[n if m.kv_from is None else m.kv_from]
        expanded = self._buf("q_expanded", H * dim_p, self.act)
        uq = lambda: self._pad_k(pad(sd[p + "uq"].view(H, dim, m.q_rank), (0, 0, 0, dim_p - dim)).flatten(0, 1))
        self._linear(low, self._attach(p + "uq.heads", uq), expanded)
        q = self._buf("q_latent", H * row, self.act)
        uk = self._attach(p + "uk.absorbed", lambda: self._pad_k(sd[p + "uk"].view(H, dim, rank).transpose(1, 2)))
        mpk.grouped_linear_layer(expanded, uk, q, in_stride=dim_p, out_stride=row)
        mixed = self._buf("latent_out", H * rank_p, self.act)
        mpk.ext_attention_layer(q, cache, cache, mixed, heads=H, kv_heads=1, vdim=rank_p, scale=m.scale, window=m.window, separate_merge=True)
        values = self._buf("mixed", self._kpad(H * m.vdim), self.act)
        uv = self._attach(p + "uv.heads", lambda: self._pad_k(sd[p + "uv"].view(H, m.vdim, rank)))
        mpk.grouped_linear_layer(mixed, uv, values, in_stride=rank_p, out_stride=m.vdim, gate=proj, gate_col=gate_col)
        return self._sublayer(values, p + "o", [sd[p + "o"]])

    def _poly(self, p: str, ff: int, h: DTensor) -> DTensor:
        z = self._buf("ff_in", ff, float32)
        self._linear(h, self._weight(p + "up.padded", [self.sd[p + "up"]]), z)
        mid = self._buf("ff", self._kpad(ff), self.act)
        self.mpk.poly_norm_layer(z, self._att(p + "act"), mid, eps=self.eps)
        return self._sublayer(mid, p + "down", [self.sd[p + "down"]])

    def build_from_config(self, mc: RuludraModelConfig):
        mpk, c, sd = self.mpk, mc.config, mc.state_dict
        self._begin(mc)
        self._latents: Dict[int, DTensor] = {}                     # layer -> its latent cache
        if tuple(sd["embed"].shape) != (c.vocab, c.width) or tuple(sd["head"].shape) != (c.vocab, c.width):
            raise ValueError(f"embedding {tuple(sd['embed'].shape)}, head {tuple(sd['head'].shape)}, configuration {(c.vocab, c.width)}")
        if c.bigram and tuple(sd["bigram"].shape) != (c.bigram[0] + 1, c.width):
            raise ValueError(f"bigram table {tuple(sd['bigram'].shape)}, configuration {c.bigram[0]} buckets")
        # two stream buffers in turn: a norm's task reads one and writes the other
        x, other = self._buf("stream", c.width, float32), self._buf("stream_b", c.width, float32)
        h = self._buf("normed", self._kpad(c.width), self.act)
        results = mpk.new_tensor(dims=(len(c.layers) + 1, mpk.max_num_batched_tokens, c.width), dtype=float32, name="results")
        freq = self._attach("position_frequencies", lambda: mpk.position_frequencies(c.width).to(sd["embed"].device))
        mpk.embed_layer(input=mpk.attach_input(mpk.meta_tensors["input_tokens"], name="input_token"), weight=self._att("embed"), output=x,
                        grid_dim=(1, 1, 1), block_dim=(128, 1, 1), input_source=1, positions=freq, copy=results,
                        bigram=(self._att("bigram"), *c.bigram[1:]) if c.bigram else None)

        def norm(y: Optional[DTensor], post: Optional[str], nxt: str, average: Optional[Tuple[DTensor, DTensor]] = None):
            nonlocal x, other
            mpk.residual_norm_layer(x, y, self._att(post) if post else None, self._att(nxt), h, eps=c.eps, x_out=other if y is not None else None,
                                    average=average)
            if y is not None:
                x, other = other, x

        # a sublayer's closing norm, the average behind a layer and the next opening norm are one task
        norm(None, None, "l0.norm1" if c.layers else "final.norm")
        for n, layer in enumerate(c.layers):
            p, st = f"l{n}.", mc.state[n]
            if isinstance(layer.mixer, MlstmSpec):
                y = self._mlstm(p + "mix.", layer.mixer, st, h)
            elif isinstance(layer.mixer, AttentionSpec):
                y = self._attention(p + "mix.", layer.mixer, st, h)
            else:
                y = self._latent(n, p + "mix.", layer.mixer, st, h)
            post = p + "norm1b"
            if layer.ff is not None:
                norm(y, post, p + "norm2")
                y, post = self._poly(p + "mlp.", layer.ff, h), p + "norm2b"
            norm(y, post, f"l{n + 1}.norm1" if n + 1 < len(c.layers) else "final.norm", (results, self._att(p + "dwa")))
        self.hidden = x
        self._head(h, self._weight("head", [sd["head"]]), c.vocab, mc.sampling_seed, activation="scale", scale=c.logit_scale)
