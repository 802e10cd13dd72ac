"""Shared helpers of the Bebuzen tests: small configurations and a runner over them."""
from oracle import bebuzen as P


def mixed_config(vocab=96, width=64, eps=1e-5):
    """Every mixer and feed-forward, keys and values shared over two layers that are not neighbours, sizes that differ between layers."""
    return P.config(vocab, width, [
        P.diff_layer(heads=4, kv_heads=2, dim=12, vdim=20, rot=8, window=21, taps=3, mlp=P.moe(6, 2, 40, 1.3, None)),
        P.mamba_layer(inner=72, state=10, dt_rank=5, taps=4, mlp=P.moe(9, 3, 24, 0.7, 56)),
        P.sink_layer(heads=3, kv_heads=1, dim=20, vdim=12, rot=12, window=30, keep=5, mlp=None),
        P.diff_layer(heads=6, kv_heads=2, dim=12, vdim=20, rot=8, window=50, taps=2, mlp=P.dense(80), diff=0.7, kv_from=0),
        P.mamba_layer(inner=40, state=16, dt_rank=8, taps=2, mlp=None),
    ], eps=eps)


def runner(c, w, dtype, *, mode="online", requests=8, slots=4, tokens=64, pages=40, page=16, max_seq=400, **kw):
    from mirage_b200.builders.bebuzen import BebuzenConfig
    from mirage_b200.builders.runner import BebuzenRunner
    return BebuzenRunner(BebuzenConfig.from_dict(c), w, mode=mode, dtype=dtype, total_num_requests=requests,
                         max_seq_length=max_seq, max_num_batched_requests=slots, max_num_batched_tokens=tokens,
                         max_num_pages=pages, page_size=page, **kw)
