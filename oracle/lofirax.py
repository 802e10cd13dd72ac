"""CPU oracle of the Lofirax decoder: the mechanisms of oracle/hybrid_ops.py in the design's order, over whole sequences.

TEST INFRASTRUCTURE ONLY.  Configurations are plain dictionaries in the checkpoint's format; weights are made here from a
seed, bf16-valued, so that the product and the oracle start from the same numbers.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch

from . import hybrid_ops as ops

Tensor = torch.Tensor


def dense(ff: int) -> Dict[str, Any]:
    return {"kind": "dense", "ff": ff}


def moe(experts: int, top: int, ff: int, groups: int, keep: int, shared: Optional[int]) -> Dict[str, Any]:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def gla_layer(heads: int, dim: int, vdim: int, tau: float, mlp: Optional[Dict[str, Any]]) -> Dict[str, Any]:
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def latent_layer(heads: int, dim: int, rot: int, vdim: int, rank: int, mlp: Optional[Dict[str, Any]], *, base: float = 5000.0,
                 scale: float = 0.2) -> Dict[str, Any]:
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def config(vocab: int, width: int, layers: Sequence[Dict[str, Any]], *, loop=None, eps: float = 1e-5, embed_scale: float = 3.0,
           softcap: float = 20.0) -> Dict[str, Any]:
    """loop: (start, stop, times) or None."""
    return {"architecture": "Lofirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers),
            "embedding": {"scale": embed_scale}, "logit_softcap": softcap,
            "loop": None if loop is None else {"start": loop[0], "stop": loop[1], "times": loop[2]}}


def make_weights(c: Dict[str, Any], seed: int, gate_rank: int = 8) -> Dict[str, Tensor]:
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, Tensor] = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def norm(name, width):
        put(name, width, std=0.2, mean=1.0)
        put(name + ".b", width, std=0.2)

    def ff(name, width, size):
        put(name + "gate", size, width)
        put(name + "up", size, width)
        put(name + "down", width, size)

    D = c["width"]
    put("embed", c["vocab"], D, std=0.3)
    if c.get("loop"):
        put("loop.step", c["loop"]["times"], D, std=0.4)
    for n, layer in enumerate(c["layers"]):
        p, m, mlp = f"l{n}.", layer["mixer"], layer["mlp"]
        norm(p + "norm1", D)
        mix = p + "mix."
        if layer["type"] == "gla":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            for nm, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv), ("a1", gate_rank)):
                put(mix + nm, rows, D)
            put(mix + "a2", H * d, gate_rank)
            put(mix + "a2.b", H * d, std=1.5, mean=1.0)      # decays from short to long
            put(mix + "norm", dv, std=0.2, mean=1.0)
            put(mix + "o", D, H * dv)
        else:
            H = m["heads"]
            put(mix + "q", H * (m["dim"] + m["rot_dim"]), D)
            put(mix + "dkv", m["kv_rank"] + m["rot_dim"], D)
            put(mix + "dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
            put(mix + "uk", H * m["dim"], m["kv_rank"])
            put(mix + "uv", H * m["vdim"], m["kv_rank"])
            put(mix + "sink", H, std=1.0)
            put(mix + "o", D, H * m["vdim"])
        if mlp is None:
            continue
        norm(p + "norm2", D)
        if mlp["kind"] == "dense":
            ff(p + "mlp.", D, mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        put(p + "mlp.router", E, D)
        put(p + "mlp.correction", E, std=0.3)
        for e in range(E):
            ff(f"{p}mlp.e{e}.", D, mlp["expert"]["ff"])
        if mlp.get("shared"):
            ff(p + "mlp.shared.", D, mlp["shared"]["ff"])
            put(p + "mlp.shared.sg", 1, D)
    norm("final.norm", D)
    put("head", c["vocab"], D)
    return w


class LofiraxOracle:
    def __init__(self, c: Dict[str, Any], weights: Dict[str, Tensor], dtype: torch.dtype = torch.float64):
        self.c, self.dtype = c, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}
        self.eps = c["norm"]["eps"]

    def _norm(self, x: Tensor, name: str) -> Tensor:
        return ops.layer_norm(x, self.w[name], self.w[name + ".b"], self.eps)

    def gla(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, T, H, d, dv = self.w, h.shape[0], m["heads"], m["dim"], m["vdim"]
        q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
        k = (h @ w[p + "k"].T).view(T, H, d)
        v = (h @ w[p + "v"].T).view(T, H, dv)
        z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).view(T, H, d)
        o = ops.rms_unit(ops.gla(q, k, v, z, m["tau"]), self.eps) * w[p + "norm"]
        return (o.reshape(T, H * dv) * ops.silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def latent(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w = self.w
        o = ops.latent_attention(h, w[p + "q"], w[p + "dkv"], w[p + "dkv.norm"], w[p + "uk"], w[p + "uv"], w[p + "sink"],
                                 heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                                 base=m["rot"]["base"], scale=m["scale"], eps=self.eps)
        return o @ w[p + "o"].T

    def moe(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, r = self.w, m["router"]
        scores = torch.sigmoid(h @ w[p + "router"].T)
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            chosen = ops.grouped_choice(scores[t], w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"])
            total = sum(scores[t, e] for e in chosen) + 1e-20
            for e in chosen:
                n = f"{p}e{e}."
                out[t] += scores[t, e] / total * ops.gated_ff(h[t], w[n + "gate"], w[n + "up"], w[n + "down"], ops.silu)
        if m.get("shared"):
            n = p + "shared."
            out = out + torch.sigmoid(h @ w[n + "sg"].T) * ops.gated_ff(h, w[n + "gate"], w[n + "up"], w[n + "down"], ops.silu)
        return out

    def order(self) -> List[tuple]:
        """(layer, pass or None) of every layer run; a pass's first run carries its number."""
        n, loop = len(self.c["layers"]), self.c.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        runs: List[tuple] = [(i, None) for i in range(loop["start"])]
        for t in range(loop["times"]):
            runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
        return runs + [(i, None) for i in range(loop["stop"], n)]

    def hidden(self, tokens: Sequence[int], trace: Optional[list] = None) -> Tensor:
        w, c = self.w, self.c
        embedded = w["embed"][torch.tensor(list(tokens))] * c["embedding"]["scale"]
        x = embedded.clone()
        for n, t in self.order():
            layer, p = c["layers"][n], f"l{n}."
            if t is not None:
                x = x + (embedded if t > 0 else 0.0) + w["loop.step"][t]
            h = self._norm(x, p + "norm1")
            x = x + (self.gla if layer["type"] == "gla" else self.latent)(p + "mix.", layer["mixer"], h)
            mlp = layer["mlp"]
            if mlp is not None:
                h = self._norm(x, p + "norm2")
                if mlp["kind"] == "dense":
                    q = p + "mlp."
                    x = x + ops.gated_ff(h, w[q + "gate"], w[q + "up"], w[q + "down"], ops.gelu_tanh)
                else:
                    x = x + self.moe(p + "mlp.", mlp, h)
            if trace is not None:
                trace.append(x.clone())
        return x

    def logits(self, tokens: Sequence[int]) -> Tensor:
        """[tokens, vocab]"""
        return ops.softcap(self._norm(self.hidden(tokens), "final.norm") @ self.w["head"].T, self.c["logit_softcap"])

    def greedy(self, prompt: Sequence[int], new_tokens: int) -> List[int]:
        out = list(prompt)
        for _ in range(new_tokens):
            out.append(int(self.logits(out)[-1].argmax()))
        return out
