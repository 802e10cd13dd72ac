"""CPU oracle of the Palarax decoder: the mechanisms of oracle/hybrid_ops.py in the design's order, over whole sequences.

TEST INFRASTRUCTURE ONLY.  Configurations are plain dictionaries in the checkpoint's format; weights are made here from a
seed, bf16-valued, so that the product and the oracle start from the same numbers.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch

from . import hybrid_ops as ops

Tensor = torch.Tensor


def mlstm_layer(heads: int, dim: int, vdim: int, cap: float = 12.0, ff: Optional[int] = 64) -> Dict[str, Any]:
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def parallel_layer(heads: int, kv_heads: int, dim: int, rot: int, width: int, blocks: int, taps: int, *, base: float = 7000.0,
                   scale: float = 0.3, softcap: float = 20.0, left_scale: float = 0.7, right_scale: float = 0.9,
                   ff: Optional[int] = 64) -> Dict[str, Any]:
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                               "softcap": softcap, "rot": {"base": base, "dims": rot}},
                      "right": {"width": width, "blocks": blocks, "conv": taps},
                      "left_scale": left_scale, "right_scale": right_scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab: int, width: int, layers: Sequence[Dict[str, Any]], eps: float = 1e-5) -> Dict[str, Any]:
    return {"architecture": "Palarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}


def make_weights(c: Dict[str, Any], seed: int) -> Dict[str, Tensor]:
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, Tensor] = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    D = c["width"]
    put("embed", c["vocab"], D, std=1.0)
    for n, layer in enumerate(c["layers"]):
        p, m = f"l{n}.", layer["mixer"]
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            put(p + nm, D, std=0.1)
        if layer["type"] == "mlstm":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            for nm, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv), ("i", H), ("f", H)):
                put(p + "mix." + nm, rows, D)
            put(p + "mix.o", D, H * dv)
            put(p + "mix.norm", H * dv, std=0.2, mean=1.0)
            put(p + "mix.i.b", H, std=1.0)
            put(p + "mix.f.b", H, std=1.0, mean=4.0)       # forget gates near one: a long memory
        else:
            l, r = m["left"], m["right"]
            pl, pr = p + "mix.left.", p + "mix.right."
            put(pl + "q", l["heads"] * l["dim"], D)
            put(pl + "k", l["kv_heads"] * l["dim"], D)
            put(pl + "o", D, l["heads"] * l["vdim"])
            W, nb = r["width"], r["blocks"]
            for nm in ("y", "x"):
                put(pr + nm, W, D)
                put(pr + nm + ".b", W, std=0.3)
            put(pr + "conv", W, r["conv"], std=0.5)
            put(pr + "conv.b", W, std=0.2)
            for nm in ("ra", "ri"):
                put(pr + nm, nb, W // nb, W // nb)
                put(pr + nm + ".b", nb, W // nb, std=0.5)
            put(pr + "lam", W, std=1.0, mean=-5.0)         # decays near one: a long memory
            put(pr + "o", D, W)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            put(p + "mlp.up", ff, D)
            put(p + "mlp.down", D, ff)
    put("final.norm", D, std=0.1)
    return w


class PalaraxOracle:
    def __init__(self, c: Dict[str, Any], weights: Dict[str, Tensor], dtype: torch.dtype = torch.float64):
        self.c, self.dtype = c, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}
        self.eps = c["norm"]["eps"]

    def _mlstm(self, p: str, m: Dict[str, Any], h: Tensor) -> Tensor:
        w, T, H, d, dv = self.w, h.shape[0], m["heads"], m["dim"], m["vdim"]
        q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
        k = (h @ w[p + "k"].T).view(T, H, d)
        v = (h @ w[p + "v"].T).view(T, H, dv)
        o = ops.mlstm(q, k, v, h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"])
        return ops.mlstm_output(o, w[p + "norm"], h @ w[p + "g"].T, self.eps) @ w[p + "o"].T

    def _attention(self, p: str, l: Dict[str, Any], h: Tensor) -> Tensor:
        w, T = self.w, h.shape[0]
        pos = torch.arange(T)
        q = (h @ w[p + "q"].T).view(T, l["heads"], l["dim"])
        v = (h @ w[p + "k"].T).view(T, l["kv_heads"], l["dim"])           # the keys as projected are the values
        turn = lambda x: ops.rms_unit(ops.rotate_half_split(x, pos, l["rot"]["base"], l["rot"]["dims"]), self.eps)
        o = ops.attention(turn(q), turn(v), v, l["scale"], l["softcap"], sink=True)
        return o.reshape(T, -1) @ w[p + "o"].T

    def _rglru(self, p: str, r: Dict[str, Any], h: Tensor) -> Tensor:
        w = self.w
        y = ops.gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
        u = ops.short_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
        S = ops.rglru(u, w[p + "ra"], w[p + "ra.b"], w[p + "ri"], w[p + "ri.b"], w[p + "lam"])
        return (S * y) @ w[p + "o"].T

    def hidden(self, tokens: Sequence[int]) -> Tensor:
        w = self.w
        norm = lambda x, name: ops.rms_norm_around_zero(x, w[name], self.eps)
        x = w["embed"][torch.tensor(list(tokens))]
        for n, layer in enumerate(self.c["layers"]):
            p, m = f"l{n}.", layer["mixer"]
            h = norm(x, p + "norm1")
            if layer["type"] == "mlstm":
                y = self._mlstm(p + "mix.", m, h)
            else:
                y = m["left_scale"] * self._attention(p + "mix.left.", m["left"], h) + \
                    m["right_scale"] * self._rglru(p + "mix.right.", m["right"], h)
            x = x + norm(y, p + "norm1b")
            if layer["mlp"]:
                y = ops.squared_relu(norm(x, p + "norm2") @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
                x = x + norm(y, p + "norm2b")
        return x

    def logits(self, tokens: Sequence[int]) -> Tensor:
        """[tokens, vocab]"""
        return ops.rms_norm_around_zero(self.hidden(tokens), self.w["final.norm"], self.eps) @ self.w["embed"].T

    def greedy(self, prompt: Sequence[int], new_tokens: int) -> List[int]:
        out = list(prompt)
        for _ in range(new_tokens):
            out.append(int(self.logits(out)[-1].argmax()))
        return out
