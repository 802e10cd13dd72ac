"""Shared helpers of the Palarax tests: small configurations and a runner over them."""
import json
import os

import torch

from oracle import palarax as P


def mixed_config(vocab=96, width=64, eps=1e-5):
    """Both mixers, in an order of its own, sizes that differ between layers, one layer without feed-forward."""
    return P.config(vocab, width, [
        P.mlstm_layer(heads=2, dim=16, vdim=24, cap=9.0, ff=80),
        P.parallel_layer(heads=4, kv_heads=2, dim=16, rot=8, width=48, blocks=3, taps=3, ff=None),
        P.mlstm_layer(heads=1, dim=20, vdim=8, ff=48),
        P.parallel_layer(heads=2, kv_heads=2, dim=32, rot=32, width=64, blocks=1, taps=4, ff=96),
    ], eps)


def runner(c, w, dtype=torch.float32, *, mode="online", requests=8, slots=4, tokens=64, pages=40, page=16, max_seq=400, **kw):
    from mirage_b200.builders.palarax import PalaraxConfig
    from mirage_b200.builders.runner import PalaraxRunner
    return PalaraxRunner(PalaraxConfig.from_dict(c), w, mode=mode, dtype=dtype, total_num_requests=requests,
                         max_seq_length=max_seq, max_num_batched_requests=slots, max_num_batched_tokens=tokens,
                         max_num_pages=pages, page_size=page, **kw)


def run_portions(session, rid, tokens, cuts):
    """One request in portions of the given sizes; logits of all its tokens."""
    out, at = [], 0
    for n in cuts:
        part = tokens[at:at + n]
        out += session.step([(rid, part, list(range(len(part))))])
        at += n
    assert at == len(tokens)
    session.step([], [rid])
    return torch.cat(out)


def cuts_of(n, sizes):
    """`n` cut into portions that cycle through `sizes`."""
    out, i = [], 0
    while n > 0:
        out.append(min(n, sizes[i % len(sizes)]))
        n -= out[-1]
        i += 1
    return out


def rel(got, ref):
    """Largest row error: RMS of the difference over the RMS of all reference logits."""
    got, ref = got.double().cpu(), ref.double()
    return float((got - ref).pow(2).mean(-1).sqrt().max() / ref.pow(2).mean().sqrt())


def save_checkpoint(path, c, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(c, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
