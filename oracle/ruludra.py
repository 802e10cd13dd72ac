"""CPU oracle of the Ruludra decoder: the mechanisms of oracle/hybrid_ops.py in the design's order, over whole sequences.

TEST INFRASTRUCTURE ONLY.  Configurations are plain dictionaries in the checkpoint's format; weights are made here from a
seed, bf16-valued, so that the product and the oracle start from the same numbers.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch

from . import hybrid_ops as ops

Tensor = torch.Tensor


def _mlp(ff: Optional[int]) -> Optional[Dict[str, Any]]:
    return None if ff is None else {"kind": "dense", "ff": ff}


def mlstm_layer(heads: int, dim: int, vdim: int, cap: float = 9.0, ff: Optional[int] = 64) -> Dict[str, Any]:
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": _mlp(ff)}


def attention_layer(heads: int, kv_heads: int, dim: int, window: int, ff: Optional[int] = 64, *, scale: float = 0.2, coef: float = 0.4,
                    every: int = 50) -> Dict[str, Any]:
    """Windowed attention with a distance bias; the keys as projected are the values."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": window}, "q_temp": {"coef": coef, "every": every}}, "mlp": _mlp(ff)}


def latent_layer(heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int, window: int, ff: Optional[int] = 64, *, scale: float = 0.25,
                 kv_from: Optional[int] = None) -> Dict[str, Any]:
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": _mlp(ff)}


def config(vocab: int, width: int, layers: Sequence[Dict[str, Any]], *, eps: float = 1e-5, logit_scale: float = 0.6, buckets: int = 83,
           mul_prev: int = 31, mul_cur: int = 7) -> Dict[str, Any]:
    return {"architecture": "Ruludra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": list(layers)}


def make_weights(c: Dict[str, Any], seed: int) -> Dict[str, Tensor]:
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, Tensor] = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    D = c["width"]
    put("embed", c["vocab"], D, std=1.0)
    put("bigram", c["embedding"]["bigram"]["buckets"] + 1, D, std=0.7)
    for n, layer in enumerate(c["layers"]):
        p, m, mlp = f"l{n}.", layer["mixer"], layer["mlp"]
        mix = p + "mix."
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            put(p + nm, D, std=0.2, mean=1.0)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "mlstm":
            for nm, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv), ("i", H), ("f", H)):
                put(mix + nm, rows, D)
            put(mix + "o", D, H * dv)
            put(mix + "norm", H * dv, std=0.2, mean=1.0)
            put(mix + "i.b", H, std=1.0)
            put(mix + "f.b", H, std=1.0, mean=4.0)           # forget gates near one: a long memory
        elif layer["type"] == "attention":
            for nm, rows in (("q", H * d), ("k", m["kv_heads"] * d)):
                put(mix + nm, rows, D)
                put(f"{mix}{nm}.norm", rows, std=0.3, mean=1.2)
            w[mix + "r1"] = torch.rand(H, generator=g).mul(0.8).to(torch.bfloat16)
            w[mix + "r2"] = torch.rand(H, generator=g).mul(1.5).to(torch.bfloat16)
            put(mix + "o", D, H * d)
        else:
            r = m["kv_rank"]
            put(mix + "dq", m["q_rank"], D)
            put(mix + "dq.norm", m["q_rank"], std=0.3, mean=1.2)
            put(mix + "uq", H * d, m["q_rank"])
            if m.get("kv_from") is None:
                put(mix + "dkv", r, D)
                put(mix + "dkv.norm", r, std=0.3, mean=1.2)
            put(mix + "uk", H * d, r)
            put(mix + "uv", H * dv, r)
            put(mix + "g", H * dv, D)
            put(mix + "o", D, H * dv)
        if mlp:
            put(p + "mlp.up", mlp["ff"], D)
            put(p + "mlp.down", D, mlp["ff"])
            put(p + "mlp.act", 4, std=0.3, mean=0.5)
        put(p + "dwa", n + 2, std=0.2)
        w[p + "dwa"][-1] += 0.8
    put("final.norm", D, std=0.2, mean=1.0)
    put("head", c["vocab"], D)
    return w


class RuludraOracle:
    def __init__(self, c: Dict[str, Any], weights: Dict[str, Tensor], dtype: torch.dtype = torch.float64):
        self.c, self.dtype = c, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}
        self.eps = c["norm"]["eps"]

    def embedding(self, tokens: Sequence[int]) -> Tensor:
        b = self.c["embedding"]["bigram"]
        rows = ops.bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])
        return self.w["embed"][torch.tensor(list(tokens))] + self.w["bigram"][torch.tensor(rows)] + \
            ops.sinusoids(len(tokens), self.c["width"], self.dtype)

    def mlstm(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, T, H, d = self.w, h.shape[0], m["heads"], m["dim"]
        q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
        k = (h @ w[p + "k"].T).view(T, H, d)
        v = (h @ w[p + "v"].T).view(T, H, m["vdim"])
        o = ops.mlstm(q, k, v, h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"])
        return ops.mlstm_output(o, w[p + "norm"], h @ w[p + "g"].T, self.eps) @ w[p + "o"].T

    def attention(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, T = self.w, h.shape[0]
        heads = lambda y: y.view(T, -1, m["dim"])
        v = h @ w[p + "k"].T
        q, k = ops.rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], self.eps), ops.rms_norm(v, w[p + "k.norm"], self.eps)
        t = m.get("q_temp")
        if t:
            q = q * torch.tensor([ops.query_temperature(i, t["coef"], t["every"]) for i in range(T)], dtype=self.dtype)[:, None]
        o = ops.biased_attention(heads(q), heads(k), heads(v), m["scale"], (m.get("mask") or {}).get("size") or 0, w[p + "r1"], w[p + "r2"])
        return o.flatten(1) @ w[p + "o"].T

    def latent(self, p: str, m: Dict[str, Any], h: Tensor, latents: Dict[int, Tensor], n: int) -> Tensor:
        w, T = self.w, h.shape[0]
        q = ops.rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], self.eps) @ w[p + "uq"].T
        if m.get("kv_from") is None:
            latents[n] = ops.rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], self.eps)
            src = n
        else:
            src = m["kv_from"]
        o = ops.latent_window_attention(q.view(T, m["heads"], m["dim"]), latents[src], w[p + "uk"], w[p + "uv"], m["scale"],
                                        (m.get("mask") or {}).get("size") or 0)
        return (o.flatten(1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def hidden(self, tokens: Sequence[int], trace: Optional[list] = None) -> Tensor:
        w = self.w
        x = self.embedding(tokens)
        history, latents = [x], {}
        for n, layer in enumerate(self.c["layers"]):
            p, m, mlp = f"l{n}.", layer["mixer"], layer["mlp"]
            norm = lambda v, name: ops.rms_norm(v, w[p + name], self.eps)
            h = norm(x, "norm1")
            if layer["type"] == "mlstm":
                y = self.mlstm(p + "mix.", m, h)
            elif layer["type"] == "attention":
                y = self.attention(p + "mix.", m, h)
            else:
                y = self.latent(p + "mix.", m, h, latents, n)
            x = x + norm(y, "norm1b")
            if mlp:
                y = ops.poly_norm(norm(x, "norm2") @ w[p + "mlp.up"].T, w[p + "mlp.act"], self.eps) @ w[p + "mlp.down"].T
                x = x + norm(y, "norm2b")
            history.append(x)
            x = ops.depth_average(history, w[p + "dwa"])
            if trace is not None:
                trace.append(x.clone())
        return x

    def logits(self, tokens: Sequence[int]) -> Tensor:
        """[tokens, vocab]"""
        return ops.rms_norm(self.hidden(tokens), self.w["final.norm"], self.eps) @ self.w["head"].T * self.c["logit_scale"]

    def greedy(self, prompt: Sequence[int], new_tokens: int) -> List[int]:
        out = list(prompt)
        for _ in range(new_tokens):
            out.append(int(self.logits(out)[-1].argmax()))
        return out
