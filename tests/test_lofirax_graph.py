"""CPU checks of the Lofirax graph (dry run, no CUDA call) -- layer sequence, dependencies, folding, refused shapes -- of its
configuration reader and of its oracle against independent formulations."""
import json

import pytest
import torch

import mirage_b200 as mi
from lofirax_util import mixed_config
from mirage_b200.builders import registry
from mirage_b200.builders.lofirax import LofiraxBuilder, LofiraxConfig, LofiraxModelConfig, allocate_state
from oracle import hybrid_ops as ops
from oracle import lofirax as P
from palarax_util import save_checkpoint

D = torch.float64


def dry(c, *, mbr=2, mbt=16, S=64, page=16, dtype=torch.bfloat16, mode="offline"):
    z = lambda *s, dt=torch.int32: torch.zeros(*s, dtype=dt)
    pages, i64 = mbr * S // page, torch.int64
    meta = {"step": z(mbr), "tokens": z(mbr, S, dt=i64), "input_tokens": z(mbt, 1, dt=i64), "output_tokens": z(mbt, 1, dt=i64),
            "num_new_tokens": z(mbr), "prompt_lengths": z(mbr), "qo_indptr_buffer": z(mbr + 1), "paged_kv_indptr_buffer": z(mbr + 1),
            "paged_kv_indices_buffer": z(pages), "paged_kv_last_page_len_buffer": z(mbr), "request_ctl": z(2, mbr), "request_ids": z(mbr)}
    pk = mi.PersistentKernel(mode=mode, max_seq_length=S, max_num_batched_requests=mbr, max_num_batched_tokens=mbt,
                             max_num_pages=pages, page_size=page, meta_tensors=meta, dry_run=True)
    cfg = LofiraxConfig.from_dict(c)
    LofiraxBuilder(pk).build_from_config(LofiraxModelConfig(cfg, P.make_weights(c, 1), allocate_state(
        cfg, slots=mbr, max_num_pages=pages, page_size=page, dtype=dtype, device="cpu", num_workers=pk.num_workers), dtype))
    return pk


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_layer_sequence_and_side_by_side_branches(dtype):
    pk = dry(mixed_config(), dtype=dtype)
    pk.compile()
    ev = json.loads(pk.dump_task_graph())["events"]
    types = [e["type"] for e in ev]
    lin, moe = ("linear", "moe_gemm") if dtype == torch.bfloat16 else ("linear_f32", "moe_gemm_f32")
    gla = ["residual_norm", lin, "gla", lin]
    lat = ["residual_norm", lin, lin, lin, "latent_append", "ext_attention", "attn_merge", lin, lin]
    dense = ["residual_norm", lin, lin]
    routed = ["residual_norm", lin, "moe_routing", moe, moe]
    shared = ["residual_norm", lin, "moe_routing", lin, lin, moe, moe]
    loop = lat + dense + gla + shared
    assert types == ["batch", "embed_f32"] + gla + routed + 3 * loop + lat + ["residual_norm", lin, "argmax_partial", "argmax_reduce"]
    deps = lambda i: sorted(d[0] for d in ev[i]["deps"])
    i = types.index("latent_append")
    norm, q_un, proj, uk, attn, merge, uv = i - 4, i - 3, i - 2, i - 1, i + 1, i + 2, i + 3
    # the queries' way into the latent space and the cache rows do not wait for one another
    assert deps(q_un) == deps(proj) == [norm] and deps(uk) == [q_un] and deps(i) == [proj] and deps(attn) == [uk, i]
    assert deps(merge) == [attn] and deps(uv) == [merge]
    j = len(types) - 1 - types[::-1].index("moe_routing")          # an expert layer with a shared expert
    assert deps(j) == [j - 1] and deps(j + 1) == [j - 2] and deps(j + 3) == [j] and deps(j + 5) == [j + 2, j + 4]


def test_norms_fold_into_the_linears_of_single_token_graphs():
    c = P.config(64, 64, [P.gla_layer(2, 16, 16, 4.0, P.dense(64)), P.gla_layer(2, 16, 16, 4.0, P.moe(4, 2, 32, 2, 1, 32))], loop=(0, 2, 2))
    pk = dry(c, mbt=1)
    pk.compile()
    ev = json.loads(pk.dump_task_graph())["events"]
    # of each pass: the mixers' norms and the dense feed-forward's, not the expert layer's (two linears read it) nor the norm that
    # sums the experts in front of the second pass and of the head
    assert sum(e.get("prologue") == "residual_norm" for e in ev) == pk.graph_info()["num_folded"] == 5
    assert sum(e["type"] == "residual_norm" for e in ev) == 4
    pk = dry(c, mbt=3)
    pk.compile()
    assert pk.graph_info()["num_folded"] == 0


def test_wide_rows_and_many_experts_compile_in_every_batch_size():
    c = P.config(64, 256, [P.latent_layer(33, 128, 64, 128, 512, P.moe(64, 8, 96, 8, 4, 200)), P.gla_layer(3, 130, 70, 8.0, P.dense(130))],
                 loop=(0, 1, 2))
    for mbt in (1, 2, 8, 9, 64):
        dry(c, mbt=mbt).compile()
    dry(c, mbt=64, dtype=torch.float32).compile()


def test_refused_graphs_say_why():
    with pytest.raises(mi.MpkError, match="64 tokens"):
        dry(mixed_config(), mbt=65).compile()
    with pytest.raises(mi.MpkError, match="key sizes"):
        dry(P.config(32, 64, [P.gla_layer(1, 1032, 8, 4.0, None)])).compile()
    with pytest.raises(mi.MpkError, match="head sizes"):
        dry(P.config(32, 64, [P.latent_layer(1, 8, 8, 8, 1200, None)])).compile()


def test_configuration_reader_takes_every_value_and_refuses_the_unknown():
    c = mixed_config(eps=3e-4)
    cfg = LofiraxConfig.from_dict(json.loads(json.dumps(c)))
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.embed_scale, cfg.logit_softcap, cfg.loop) == (96, 64, 3e-4, 3.0, 20.0, (1, 3, 3))
    g, a, m = cfg.layers[0].mixer, cfg.layers[1].mixer, cfg.layers[2].ff
    assert (g.heads, g.dim, g.vdim, g.tau) == (2, 16, 24, 4.0)
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.rot_base, a.scale) == (3, 12, 8, 20, 40, 5000.0, 0.2)
    assert (m.experts, m.top, m.ff, m.groups, m.keep, m.shared_ff) == (10, 3, 24, 5, 3, 56)
    assert cfg.layers[0].ff.shared_ff is None and cfg.layers[1].ff == 80 and cfg.layers[3].ff is None
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 1, "mlp", "kind"), "sparse"), (("layers", 1, "mixer", "rot", "dims"), 4),
                        (("layers", 2, "mlp", "router", "groups", "count"), 4), (("layers", 2, "mlp", "router", "top"), 7),
                        (("loop", "stop"), 5), (("loop", "times"), 0)):
        bad = json.loads(json.dumps(c))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            LofiraxConfig.from_dict(bad)


def test_loop_order_is_the_oracles():
    for loop in (None, (0, 4, 1), (0, 1, 3), (1, 3, 2), (3, 4, 2)):
        c = dict(mixed_config(), loop=None if loop is None else dict(zip(("start", "stop", "times"), loop)))
        assert LofiraxConfig.from_dict(c).runs() == P.LofiraxOracle(c, {}).order()


def test_registry_picks_runner_and_kernel_family_by_config(tmp_path):
    c = mixed_config()
    save_checkpoint(str(tmp_path / "p"), c, P.make_weights(c, 1))
    cls, dtypes = mi.runner_class(str(tmp_path / "p"))
    assert cls.__name__ == "LofiraxRunner" and torch.float32 in dtypes and registry.kernel_family(str(tmp_path / "p")) == "hybrid"
    assert mi.get_builder("Lofirax") is LofiraxBuilder


def test_gated_rows_interleave_in_pairs():
    g, u = torch.arange(6.).view(6, 1), 10 + torch.arange(6.).view(6, 1)
    assert mi.PersistentKernel.interleave_gated(g, u)[:, 0].tolist() == [0, 1, 10, 11, 2, 3, 12, 13, 4, 5, 14, 15]


# ---- the oracle's mechanisms against independent formulations
def test_gla_recurrence_equals_the_quadratic_form():
    g = torch.Generator().manual_seed(1)
    T, H, d, dv, tau = 17, 2, 5, 7, 3.0
    q, k, z = (torch.randn(T, H, d, generator=g, dtype=D) for _ in range(3))
    v = torch.randn(T, H, dv, generator=g, dtype=D)
    log = torch.nn.functional.logsigmoid(z) / tau
    F = log.cumsum(0)
    out = torch.zeros(T, H, dv, dtype=D)
    for t in range(T):
        w = torch.exp(F[t] - F[:t + 1])                            # [s, H, d]: the decays after step s
        out[t] = torch.einsum("hd,shd,shd,shv->hv", q[t], w, k[:t + 1], v[:t + 1])
    torch.testing.assert_close(ops.gla(q, k, v, z, tau), out, rtol=1e-9, atol=1e-11)


def test_latent_attention_equals_the_absorbed_form():
    """Attention in the latent space -- queries through W_uk^T, outputs through W_uv -- is the expanded one."""
    g = torch.Generator().manual_seed(2)
    T, W, H, dim, rot, vdim, rank = 13, 11, 3, 6, 4, 5, 8
    r = lambda *s: torch.randn(*s, generator=g, dtype=D)
    h, wq, wd, nw, uk, uv, sinks = r(T, W), r(H * (dim + rot), W), r(rank + rot, W), r(rank), r(H * dim, rank), r(H * vdim, rank), r(H)
    kw = dict(heads=H, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, base=50.0, scale=0.3, eps=1e-4)
    q = (h @ wq.T).view(T, H, dim + rot)
    c = ops.rms_unit(h @ wd[:rank].T, 1e-4) * nw
    ang = torch.arange(T, dtype=D)[:, None] * 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=D) / rot)
    turn = lambda x: torch.cat([x[..., :rot // 2] * torch.cos(ang)[:, None] - x[..., rot // 2:] * torch.sin(ang)[:, None],
                                x[..., rot // 2:] * torch.cos(ang)[:, None] + x[..., :rot // 2] * torch.sin(ang)[:, None]], -1)
    q_lat = torch.einsum("thd,hdr->thr", q[..., :dim], uk.view(H, dim, rank))
    s = torch.einsum("thr,sr->hts", q_lat, c) + torch.einsum("thd,sd->hts", turn(q[..., dim:]), turn((h @ wd[rank:].T)[:, None])[:, 0])
    s = (0.3 * s).masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    p = torch.cat([s, sinks.view(H, 1, 1).expand(H, T, 1)], -1).softmax(-1)[..., :-1]     # the sink takes weight and gives nothing
    out = torch.einsum("hts,sr,hvr->thv", p, c, uv.view(H, vdim, rank)).reshape(T, -1)
    torch.testing.assert_close(ops.latent_attention(h, wq, wd, nw, uk, uv, sinks, **kw), out, rtol=1e-9, atol=1e-11)


def test_layer_norm_and_grouped_choice():
    g = torch.Generator().manual_seed(3)
    x, w, b = (torch.randn(*s, generator=g, dtype=D) for s in ((5, 9), (9,), (9,)))
    torch.testing.assert_close(ops.layer_norm(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (9,), w, b, 1e-3))
    s = torch.tensor([0.9, 0.1, 0.5, 0.6, 0.2, 0.3])
    c = torch.tensor([-2.0, 0.0, -0.2, -0.1, 0.0, 0.0])             # the best score has the worst choice score
    assert ops.grouped_choice(s, c, 3, 1, 2) == [3, 2]               # groups: -1.0, 0.8, 0.5
    assert ops.grouped_choice(s, c, 3, 2, 3) == [3, 2, 5]
    assert ops.grouped_choice(s, c - 5.0, 3, 2, 3) == [3, 2, 5]      # all choice scores negative: what is not kept stays out
    assert ops.grouped_choice(s, c, 1, 1, 6) == [3, 2, 5, 4, 1, 0]
