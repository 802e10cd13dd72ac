"""Shared helpers of the Ruludra tests: small configurations and a runner over them."""
from oracle import ruludra as P


def mixed_config(vocab=96, width=64, eps=1e-5, **kw):
    """Every mixer, latents shared over two layers that are not neighbours (with other heads and windows), sizes that differ between
    layers, layers without feed-forward."""
    return P.config(vocab, width, [
        P.latent_layer(heads=3, dim=12, vdim=20, q_rank=24, kv_rank=40, window=21, ff=80),
        P.attention_layer(heads=6, kv_heads=2, dim=20, window=30, ff=None),
        P.mlstm_layer(heads=2, dim=16, vdim=24, ff=48),
        P.latent_layer(heads=5, dim=16, vdim=8, q_rank=36, kv_rank=40, window=50, ff=None, kv_from=0, scale=0.2),
        P.attention_layer(heads=3, kv_heads=3, dim=8, window=9, ff=72, coef=0.7, every=16),
        P.mlstm_layer(heads=1, dim=20, vdim=8, ff=None),
    ], eps=eps, **kw)


def runner(c, w, dtype, *, mode="online", requests=8, slots=4, tokens=64, pages=40, page=16, max_seq=400, **kw):
    from mirage_b200.builders.ruludra import RuludraConfig
    from mirage_b200.builders.runner import RuludraRunner
    return RuludraRunner(RuludraConfig.from_dict(c), w, mode=mode, dtype=dtype, total_num_requests=requests,
                         max_seq_length=max_seq, max_num_batched_requests=slots, max_num_batched_tokens=tokens,
                         max_num_pages=pages, page_size=page, **kw)
