"""CPU oracle of the Bebuzen decoder: the mechanisms of oracle/hybrid_ops.py in the design's order, over whole sequences.

TEST INFRASTRUCTURE ONLY.  Configurations are plain dictionaries in the checkpoint's format; weights are made here from a
seed, bf16-valued, so that the product and the oracle start from the same numbers.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch

from . import hybrid_ops as ops

Tensor = torch.Tensor


def dense(ff: int) -> Dict[str, Any]:
    return {"kind": "dense", "ff": ff}


def moe(experts: int, top: int, ff: int, scale: float, shared: Optional[int]) -> Dict[str, Any]:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def mamba_layer(inner: int, state: int, dt_rank: int, taps: int, mlp: Optional[Dict[str, Any]]) -> Dict[str, Any]:
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": taps}, "mlp": mlp}


def sink_layer(heads: int, kv_heads: int, dim: int, vdim: int, rot: int, window: int, keep: int, mlp: Optional[Dict[str, Any]], *,
               base: float = 3000.0, scale: float = 0.2) -> Dict[str, Any]:
    """Attention with a sliding window, kept first tokens and one in the softmax denominator."""
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                             "mask": {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def diff_layer(heads: int, kv_heads: int, dim: int, vdim: int, rot: int, window: int, taps: int, mlp: Optional[Dict[str, Any]], *,
               diff: float = 0.4, base: float = 20000.0, scale: float = 0.15, scaling: Tuple = (3.0, 1.0, 5.0, 300),
               kv_from: Optional[int] = None) -> Dict[str, Any]:
    """Differential attention; scaling: (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "diff": diff, "scale": scale, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(vocab: int, width: int, layers: Sequence[Dict[str, Any]], *, eps: float = 1e-5, mult: float = 0.8) -> Dict[str, Any]:
    return {"architecture": "Bebuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": list(layers)}


def make_weights(c: Dict[str, Any], seed: int) -> Dict[str, Tensor]:
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, Tensor] = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    D = c["width"]
    put("embed", c["vocab"], D, std=1.0)
    for n, layer in enumerate(c["layers"]):
        p, m, mlp = f"l{n}.", layer["mixer"], layer["mlp"]
        mix = p + "mix."
        put(p + "norm1", D, std=0.2, mean=1.0)
        if layer["type"] == "mamba1":
            inner, state, rank = m["inner"], m["state"], m["dt_rank"]
            put(mix + "in", 2 * inner, D)
            put(mix + "conv", inner, m["conv"])
            put(mix + "conv.b", inner, std=0.2)
            put(mix + "x", rank + 2 * state, inner, std=1.5 * inner ** -0.5)
            put(mix + "dt", inner, rank)
            put(mix + "dt.b", inner, std=2.0, mean=-2.0)           # step sizes, and with them memories, from short to long
            put(mix + "A_log", inner, state, std=0.8)
            put(mix + "D", inner, std=0.5, mean=1.0)
            put(mix + "o", D, inner)
        else:
            maps = 2 if layer["type"] == "attention" else 1
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for nm, rows in [("q", H * maps * d)] + ([("k", G * maps * d), ("v", G * dv)] if "kv_from" not in m else []):
                put(mix + nm, rows, D)
                put(mix + nm + ".b", rows, std=0.3)
                if maps == 2:
                    put(f"{mix}{nm}.conv", rows, m["conv"], std=0.6)
                if nm != "v":
                    put(f"{mix}{nm}.norm", d, std=0.3, mean=1.5)
            if maps == 2:
                for nm in ("lq1", "lk1", "lq2", "lk2"):
                    put(mix + nm, d, std=0.6 * d ** -0.25)
            put(mix + "o", D, H * dv)
            if maps == 1:
                put(mix + "o.b", D, std=0.3)
        if mlp is None:
            continue
        put(p + "norm2", D, std=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            put(p + "mlp.gate", mlp["ff"], D)
            put(p + "mlp.up", mlp["ff"], D)
            put(p + "mlp.down", D, mlp["ff"])
            continue
        put(p + "mlp.router", mlp["router"]["experts"], D, std=2.0 * D ** -0.5)
        for name, ff in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + \
                ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            put(f"{p}mlp.{name}.up", ff, D)
            put(f"{p}mlp.{name}.down", D, ff)
    put("final.norm", D, std=0.2, mean=1.0)
    put("head", c["vocab"], D)
    return w


class BebuzenOracle:
    def __init__(self, c: Dict[str, Any], weights: Dict[str, Tensor], dtype: torch.dtype = torch.float64):
        self.c, self.dtype = c, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}
        self.eps = c["norm"]["eps"]

    def mamba(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, inner, state, rank = self.w, m["inner"], m["state"], m["dt_rank"]
        xz = h @ w[p + "in"].T
        x = ops.silu(ops.short_conv(xz[:, :inner], w[p + "conv"], w[p + "conv.b"]))
        low = x @ w[p + "x"].T
        dt = torch.nn.functional.softplus(low[:, :rank] @ w[p + "dt"].T + w[p + "dt.b"])
        y = ops.selective_scan(x, dt, -torch.exp(w[p + "A_log"]), low[:, rank:rank + state], low[:, rank + state:], w[p + "D"])
        return (y * ops.silu(xz[:, inner:])) @ w[p + "o"].T

    def _heads(self, p: str, nm: str, h: Tensor, m: Dict[str, Any], size: int, maps: int, turn: bool) -> Tensor:
        """Projection, convolution, norm and rotation of q, k or v -> [tokens, heads * maps, size]."""
        w = self.w
        y = h @ w[p + nm].T + w[p + nm + ".b"]
        if maps == 2:
            y = ops.short_conv(y, w[f"{p}{nm}.conv"], None)
        y = y.view(h.shape[0], -1, size)
        if not turn:
            return y
        freqs = ops.rotary_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
        return ops.rotate_pairs(ops.rms_norm(y, w[f"{p}{nm}.norm"], self.eps), torch.arange(h.shape[0]), freqs, interleaved=maps == 1)

    def sink_attention(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w = self.w
        q, k = (self._heads(p, nm, h, m, m["dim"], 1, True) for nm in ("q", "k"))
        o = ops.window_attention(q, k, self._heads(p, "v", h, m, m["vdim"], 1, False), m["scale"], m["mask"]["size"],
                                 m["mask"]["keep_first"], sink=True)
        return o.flatten(1) @ w[p + "o"].T + w[p + "o.b"]

    def diff_attention(self, p: str, m: Dict[str, Any], h: Tensor, kv: Dict[int, tuple], n: int) -> Tensor:
        w, T, d = self.w, h.shape[0], m["dim"]
        pair = lambda y: y.view(T, -1, 2, d)
        if "kv_from" not in m:
            kv[n] = (pair(self._heads(p, "k", h, m, d, 2, True)), self._heads(p, "v", h, m, m["vdim"], 2, False))
        k, v = kv[m.get("kv_from", n)]
        lam = ops.diff_lambda(*(w[p + nm] for nm in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
        o = ops.diff_attention(pair(self._heads(p, "q", h, m, d, 2, True)), k, v, m["scale"], lam, m["diff"], self.eps, m["mask"]["size"])
        return o.flatten(1) @ w[p + "o"].T

    def moe(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, r = self.w, m["router"]
        expert = lambda x, n: ops.squared_relu(x @ w[n + ".up"].T) @ w[n + ".down"].T
        logits = h @ w[p + "router"].T
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            for e, s in zip(*ops.softmax_choice(logits[t], r["top"])):
                out[t] += s * r["scale"] * expert(h[t], f"{p}e{e}")
        return out + expert(h, p + "shared") if m.get("shared") else out

    def hidden(self, tokens: Sequence[int], trace: Optional[list] = None) -> Tensor:
        w, mult = self.w, self.c["residual_mult"]
        x = w["embed"][torch.tensor(list(tokens))]
        kv: Dict[int, tuple] = {}
        for n, layer in enumerate(self.c["layers"]):
            p, m, mlp = f"l{n}.", layer["mixer"], layer["mlp"]
            if layer["type"] == "mamba1":
                y = self.mamba(p + "mix.", m, x)
            elif layer["type"] == "attention":
                y = self.diff_attention(p + "mix.", m, x, kv, n)
            else:
                y = self.sink_attention(p + "mix.", m, x)
            x = x + mult * ops.rms_norm(y, w[p + "norm1"], self.eps)
            if mlp is not None:
                q = p + "mlp."
                y = self.moe(q, mlp, x) if mlp["kind"] == "moe" else ops.gated_ff(x, w[q + "gate"], w[q + "up"], w[q + "down"], ops.silu)
                x = x + mult * ops.rms_norm(y, w[p + "norm2"], self.eps)
            if trace is not None:
                trace.append(x.clone())
        return x

    def logits(self, tokens: Sequence[int]) -> Tensor:
        """[tokens, vocab]"""
        return ops.rms_norm(self.hidden(tokens), self.w["final.norm"], self.eps) @ self.w["head"].T

    def greedy(self, prompt: Sequence[int], new_tokens: int) -> List[int]:
        out = list(prompt)
        for _ in range(new_tokens):
            out.append(int(self.logits(out)[-1].argmax()))
        return out
