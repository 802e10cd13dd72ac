"""CPU oracle of the mechanisms hybrid graphs are made of: one plain, slow function each.

TEST INFRASTRUCTURE ONLY.  Whole sequences in, token loops for the recurrences, in the dtype of the inputs (the tests use
float64).  Shares nothing with the product path.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Sequence, Tuple

import torch

Tensor = torch.Tensor


def rms_unit(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm_around_zero(x: Tensor, w: Tensor, eps: float) -> Tensor:
    return rms_unit(x, eps) * (1 + w)


def residual_norm(x: Tensor, y: Optional[Tensor], w_post: Optional[Tensor], w_next: Tensor, eps: float,
                  around_zero: bool = True) -> Tuple[Tensor, Tensor]:
    """(new stream, normed stream)."""
    one = 1.0 if around_zero else 0.0
    if y is not None:
        x = x + (y if w_post is None else rms_unit(y, eps) * (one + w_post))
    return x, rms_unit(x, eps) * (one + w_next)


def rotate_half_split(x: Tensor, pos: Tensor, base: float, dims: int) -> Tensor:
    """x [tokens, heads, size]; component i < dims / 2 turns with component i + dims / 2 by pos * base^(-2 i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * c - v * s
        out[..., i + dims // 2] = v * c + u * s
    return out


def attention(q: Tensor, k: Tensor, v: Tensor, scale: float, softcap: float = 0.0, sink: bool = False) -> Tensor:
    """q [tokens, H, d], k [tokens, G, d], v [tokens, G, dv]: causal, grouped heads -> [tokens, H, dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            s = (k[:t + 1, g] @ q[t, h]) * scale
            if softcap:
                s = softcap * torch.tanh(s / softcap)
            top = torch.clamp(s.max(), min=0.0) if sink else s.max()
            e = torch.exp(s - top)
            total = e.sum() + (torch.exp(-top) if sink else 0.0)
            out[t, h] = (e / total) @ v[:t + 1, g]
    return out


def short_conv(x: Tensor, taps: Tensor, bias: Optional[Tensor]) -> Tensor:
    """x [tokens, C], taps [C, n] (last column: the current token)."""
    T, C = x.shape
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = torch.zeros(C, dtype=x.dtype) if bias is None else bias.clone()
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                acc = acc + taps[:, j] * x[src]
        out[t] = acc
    return out


def gelu_tanh(z: Tensor) -> Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rglru(u: Tensor, ra: Tensor, ra_b: Tensor, ri: Tensor, ri_b: Tensor, lam: Tensor, decay: float = 8.0) -> Tensor:
    """u [tokens, width], gate matrices [blocks, size, size] -> the recurrence's state after every token."""
    T, width = u.shape
    nb, size = ra.shape[:2]
    S = torch.zeros(width, dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(T):
        r, i = torch.zeros_like(S), torch.zeros_like(S)
        for b in range(nb):
            sl = slice(b * size, (b + 1) * size)
            r[sl] = torch.sigmoid(ra[b] @ u[t, sl] + ra_b[b])
            i[sl] = torch.sigmoid(ri[b] @ u[t, sl] + ri_b[b])
        log_a = -decay * r * torch.nn.functional.softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i * u[t]
        out[t] = S
    return out


def mlstm(q: Tensor, k: Tensor, v: Tensor, i_pre: Tensor, f_pre: Tensor, cap: float) -> Tensor:
    """q (already scaled), k [tokens, H, d], v [tokens, H, dv], gate pre-activations [tokens, H] -> read-outs
    [tokens, H, dv], with the running maximum that keeps the exponentials bounded."""
    T, H, d = q.shape
    i_log = cap * torch.tanh(i_pre / cap)
    f_log = torch.nn.functional.logsigmoid(cap * torch.tanh(f_pre / cap))
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        n = torch.zeros(d, dtype=q.dtype)
        m = torch.zeros((), dtype=q.dtype)
        for t in range(T):
            m_new = torch.maximum(f_log[t, h] + m, i_log[t, h])
            keep, add = torch.exp(f_log[t, h] + m - m_new), torch.exp(i_log[t, h] - m_new)
            m = m_new
            S = keep * S + add * torch.outer(k[t, h], v[t, h])
            n = keep * n + add * k[t, h]
            out[t, h] = (q[t, h] @ S) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm_output(o: Tensor, norm: Tensor, gate: Tensor, eps: float) -> Tensor:
    """Read-outs [tokens, H, dv] -> per-head unit norm, times the weight, times sigmoid(gate) [tokens, H * dv]."""
    return rms_unit(o, eps).reshape(o.shape[0], -1) * norm * torch.sigmoid(gate)


def squared_relu(x: Tensor) -> Tensor:
    return torch.relu(x) ** 2


def layer_norm(x: Tensor, w: Tensor, b: Tensor, eps: float) -> Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def attention_sinks(q: Tensor, k: Tensor, v: Tensor, scale: float, sinks: Tensor) -> Tensor:
    """Causal attention as above, one key/value head per query head; exp(sinks[h]) joins head h's denominator."""
    T, H = q.shape[:2]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        for t in range(T):
            s = (k[:t + 1, h] @ q[t, h]) * scale
            top = torch.maximum(s.max(), sinks[h])
            e = torch.exp(s - top)
            out[t, h] = (e / (e.sum() + torch.exp(sinks[h] - top))) @ v[:t + 1, h]
    return out


def latent_attention(h: Tensor, w_q: Tensor, w_dkv: Tensor, latent_norm: Tensor, w_uk: Tensor, w_uv: Tensor, sinks: Tensor, *,
                     heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, base: float, scale: float,
                     eps: float) -> Tensor:
    """Keys and values expanded from the latents, per head; h [tokens, width] -> [tokens, heads * vdim]."""
    T = h.shape[0]
    pos = torch.arange(T)
    q = (h @ w_q.T).view(T, heads, dim + rot_dim)
    q_rot = rotate_half_split(q[..., dim:], pos, base, rot_dim)
    down = h @ w_dkv.T
    c = rms_unit(down[:, :kv_rank], eps) * latent_norm
    k_rot = rotate_half_split(down[:, None, kv_rank:], pos, base, rot_dim).expand(T, heads, rot_dim)
    k = torch.cat([(c @ w_uk.T).view(T, heads, dim), k_rot], -1)
    v = (c @ w_uv.T).view(T, heads, vdim)
    return attention_sinks(torch.cat([q[..., :dim], q_rot], -1), k, v, scale, sinks).reshape(T, heads * vdim)


def gla(q: Tensor, k: Tensor, v: Tensor, z: Tensor, tau: float) -> Tensor:
    """Gated linear attention: q (already scaled), k, gate pre-activations z [tokens, H, d], v [tokens, H, dv]."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = (torch.sigmoid(z[t, h]) ** (1.0 / tau))[:, None] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = q[t, h] @ S
    return out


def silu(z: Tensor) -> Tensor:
    return z * torch.sigmoid(z)


def gated_ff(h: Tensor, gate: Tensor, up: Tensor, down: Tensor, act) -> Tensor:
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def grouped_choice(scores: Tensor, correction: Tensor, groups: int, keep: int, top: int) -> list:
    """Experts of one token: `scores` [experts]; groups of neighbours compete with the sum of their two best choice scores."""
    choice = scores + correction
    size = choice.shape[0] // groups
    totals = [float(sum(sorted(choice[g * size:(g + 1) * size].tolist(), reverse=True)[:2])) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -totals[g])[:keep]
    allowed = [e for e in range(choice.shape[0]) if e // size in kept]
    return sorted(allowed, key=lambda e: -float(choice[e]))[:top]


def softcap(z: Tensor, cap: float) -> Tensor:
    return cap * torch.tanh(z / cap)


def rms_norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
    return rms_unit(x, eps) * w


def rotary_frequencies(base: float, dims: int, scaling: Optional[Dict[str, float]] = None) -> list:
    """Angle per position of every pair.  `scaling`: long wavelengths are stretched by `factor`, short ones kept, those between
    original / high and original / low blended."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            waves = scaling["original"] * f / (2 * math.pi)        # turns within the original length
            if waves < scaling["low"]:
                f = f / scaling["factor"]
            elif waves <= scaling["high"]:
                s = (waves - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(x: Tensor, pos: Tensor, freqs: Sequence[float], interleaved: bool) -> Tensor:
    """x [tokens, heads, size]; pair i is (i, i + n) of the first 2 n components, or (2 i, 2 i + 1), n = len(freqs)."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + len(freqs))
        c, s = torch.cos(pos.to(x.dtype) * f)[:, None], torch.sin(pos.to(x.dtype) * f)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def visible(i: int, window: int = 0, keep_first: int = 0) -> list:
    """Keys position i sees: itself and the window - 1 before it (all before it without a window), and the first `keep_first`."""
    return [j for j in range(i + 1) if not window or i - j < window or j < keep_first]


def window_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, window: int = 0, keep_first: int = 0, sink: bool = False) -> Tensor:
    """Grouped heads over the visible keys; `sink` adds one to the softmax denominator."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        at = torch.tensor(visible(t, window, keep_first))
        for h in range(H):
            g = h // (H // G)
            s = (k[at, g] @ q[t, h]) * scale
            top = torch.clamp(s.max(), min=0.0) if sink else s.max()
            e = torch.exp(s - top)
            out[t, h] = (e / (e.sum() + (torch.exp(-top) if sink else 0.0))) @ v[at, g]
    return out


def diff_lambda(lq1: Tensor, lk1: Tensor, lq2: Tensor, lk2: Tensor, diff: float) -> Tensor:
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def diff_combine(a1: Tensor, a2: Tensor, lam: Tensor, diff: float, eps: float) -> Tensor:
    """The two maps' outputs [.., vdim] -> unit norm of their difference, times 1 - diff."""
    return rms_unit(a1 - lam * a2, eps) * (1 - diff)


def diff_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, lam: Tensor, diff: float, eps: float, window: int = 0) -> Tensor:
    """q [tokens, H, 2, d], k [tokens, G, 2, d], v [tokens, G, dv]: one attention per map over the same values."""
    a1, a2 = (window_attention(q[:, :, m], k[:, :, m], v, scale, window) for m in range(2))
    return diff_combine(a1, a2, lam, diff, eps)


def selective_scan(x: Tensor, dt: Tensor, A: Tensor, B: Tensor, C: Tensor, D: Tensor) -> Tensor:
    """x, dt [tokens, channels], A [channels, n], B, C [tokens, n] -> read-outs [tokens, channels]."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def softmax_choice(logits: Tensor, top: int) -> Tuple[list, Tensor]:
    """Experts of one token with their weights: the largest probabilities, as they are."""
    p = torch.softmax(logits, -1)
    chosen = sorted(range(p.shape[0]), key=lambda e: -float(p[e]))[:top]
    return chosen, p[torch.tensor(chosen)]


def bigram_rows(tokens: Sequence[int], buckets: int, mul_prev: int, mul_cur: int) -> list:
    """Row of the bigram table for every token of a sequence; the first token has the row behind the buckets."""
    return [buckets] + [(a * mul_prev + b * mul_cur) % buckets for a, b in zip(tokens, tokens[1:])]


def sinusoids(tokens: int, width: int, dtype: torch.dtype) -> Tensor:
    """[tokens, width]: sine and cosine, in turn, of position * 10000^(-2 i / width)."""
    out = torch.zeros(tokens, width, dtype=dtype)
    for p in range(tokens):
        for j in range(width):
            a = p * 10000.0 ** (-2.0 * (j // 2) / width)
            out[p, j] = math.cos(a) if j % 2 else math.sin(a)
    return out


def depth_average(history: Sequence[Tensor], weights: Tensor) -> Tensor:
    """Weighted sum of the embedding output and all layers' results so far."""
    assert len(history) == weights.shape[0]
    out = torch.zeros_like(history[0])
    for x, w in zip(history, weights):
        out = out + w * x
    return out


def query_temperature(position: int, coef: float, every: int) -> float:
    return 1.0 + coef * math.log((position + 1) // every + 1)


def biased_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, window: int, r1: Tensor, r2: Tensor) -> Tensor:
    """Grouped heads over the visible keys; a key d positions back has r1[h] * ln(1 + r2[h] * d) taken off its score."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        at = torch.tensor(visible(t, window))
        for h in range(H):
            g = h // (H // G)
            s = (k[at, g] @ q[t, h]) * scale - r1[h] * torch.log(1 + r2[h] * (t - at).to(q.dtype))
            out[t, h] = torch.softmax(s, 0) @ v[at, g]
    return out


def latent_window_attention(q: Tensor, c: Tensor, w_uk: Tensor, w_uv: Tensor, scale: float, window: int) -> Tensor:
    """q [tokens, H, d], latents c [tokens, rank]: keys and values expanded per head -> [tokens, H, dv]."""
    T, H, d = q.shape
    k = (c @ w_uk.T).view(T, H, d)
    v = (c @ w_uv.T).view(T, H, -1)
    return window_attention(q, k, v, scale, window)


def poly_norm(z: Tensor, coef: Tensor, eps: float) -> Tensor:
    """Weighted sum of the first three powers of z, each divided by its root mean square, and a constant (four numbers)."""
    return coef[0] * rms_unit(z, eps) + coef[1] * rms_unit(z ** 2, eps) + coef[2] * rms_unit(z ** 3, eps) + coef[3]
