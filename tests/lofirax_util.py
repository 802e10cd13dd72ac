"""Shared helpers of the Lofirax tests: small configurations and a runner over them."""
from oracle import lofirax as P


def mixed_config(vocab=96, width=64, eps=1e-5):
    """Every mixer and feed-forward, a loop in the middle with a layer before and after it, sizes that differ between layers."""
    return P.config(vocab, width, [
        P.gla_layer(heads=2, dim=16, vdim=24, tau=4.0, mlp=P.moe(6, 2, 40, groups=2, keep=1, shared=None)),
        P.latent_layer(heads=3, dim=12, rot=8, vdim=20, rank=40, mlp=P.dense(80)),
        P.gla_layer(heads=1, dim=20, vdim=8, tau=16.0, mlp=P.moe(10, 3, 24, groups=5, keep=3, shared=56)),
        P.latent_layer(heads=2, dim=16, rot=4, vdim=8, rank=24, mlp=None),
    ], loop=(1, 3, 3), eps=eps)


def runner(c, w, dtype, *, mode="online", requests=8, slots=4, tokens=64, pages=40, page=16, max_seq=400, **kw):
    from mirage_b200.builders.lofirax import LofiraxConfig
    from mirage_b200.builders.runner import LofiraxRunner
    return LofiraxRunner(LofiraxConfig.from_dict(c), w, mode=mode, dtype=dtype, total_num_requests=requests,
                         max_seq_length=max_seq, max_num_batched_requests=slots, max_num_batched_tokens=tokens,
                         max_num_pages=pages, page_size=page, **kw)
