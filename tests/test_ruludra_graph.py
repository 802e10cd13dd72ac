"""CPU checks of the Ruludra graph (dry run, no CUDA call) -- layer sequence, dependencies, folding, refused shapes -- of its
configuration reader and of its oracle against independent formulations."""
import json
import math

import pytest
import torch

import mirage_b200 as mi
from mirage_b200.builders import registry
from mirage_b200.builders.hybrid import MlstmSpec
from mirage_b200.builders.ruludra import RuludraBuilder, RuludraConfig, RuludraModelConfig, allocate_state
from oracle import hybrid_ops as ops
from oracle import ruludra as P
from palarax_util import save_checkpoint
from ruludra_util import mixed_config

D = torch.float64


def dry(c, *, mbr=2, mbt=16, S=64, page=16, dtype=torch.bfloat16, mode="offline"):
    z = lambda *s, dt=torch.int32: torch.zeros(*s, dtype=dt)
    pages, i64 = mbr * S // page, torch.int64
    meta = {"step": z(mbr), "tokens": z(mbr, S, dt=i64), "input_tokens": z(mbt, 1, dt=i64), "output_tokens": z(mbt, 1, dt=i64),
            "num_new_tokens": z(mbr), "prompt_lengths": z(mbr), "qo_indptr_buffer": z(mbr + 1), "paged_kv_indptr_buffer": z(mbr + 1),
            "paged_kv_indices_buffer": z(pages), "paged_kv_last_page_len_buffer": z(mbr), "request_ctl": z(2, mbr), "request_ids": z(mbr)}
    pk = mi.PersistentKernel(mode=mode, max_seq_length=S, max_num_batched_requests=mbr, max_num_batched_tokens=mbt,
                             max_num_pages=pages, page_size=page, meta_tensors=meta, dry_run=True)
    cfg = RuludraConfig.from_dict(c)
    RuludraBuilder(pk).build_from_config(RuludraModelConfig(cfg, P.make_weights(c, 1), allocate_state(
        cfg, slots=mbr, max_num_pages=pages, page_size=page, dtype=dtype, device="cpu", num_workers=pk.num_workers), dtype))
    return pk


def events(pk):
    pk.compile()
    return json.loads(pk.dump_task_graph())["events"]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_layer_sequence_and_dependencies(dtype):
    ev = events(dry(mixed_config(), dtype=dtype))
    types = [e["type"] for e in ev]
    lin = "linear" if dtype == torch.bfloat16 else "linear_f32"
    attention = [lin, "qkv_append", "ext_attention", lin, "residual_norm"]
    latent = lambda own: [lin, "residual_norm"] + ["latent_append"] * own + [lin, lin, "ext_attention", "attn_merge", lin, lin, "residual_norm"]
    mlstm, ff = [lin, "mlstm", lin, "residual_norm"], [lin, "poly_norm", lin, "residual_norm"]
    assert types == ["batch", "embed_f32", "residual_norm"] + latent(1) + ff + attention + mlstm + ff + latent(0) + attention + ff + mlstm + \
        [lin, "argmax_partial", "argmax_reduce"]
    deps = lambda i: sorted(d[0] for d in ev[i]["deps"])
    j = types.index("latent_append")                               # beside the norm of the query latent
    assert deps(j) == deps(j - 1) == [j - 2] and deps(j + 1) == [j - 1] and deps(j + 3) == [j, j + 2]


def test_norms_fold_into_the_linears_of_single_token_graphs():
    c = mixed_config()
    pk = dry(c, mbt=1)
    ev = events(pk)
    # the first norm, two query latents, three in front of a feed-forward, one with an average per layer; and three activations
    kinds = [e.get("prologue") for e in ev]
    assert (kinds.count("residual_norm"), kinds.count("poly_norm")) == (6 + len(c["layers"]), 3) and pk.graph_info()["num_folded"] == 15
    assert not {"residual_norm", "poly_norm"} & {e["type"] for e in ev}
    # an average over many results is formed once, not by every task of the linear behind it
    deep = dry(P.config(32, 64, [P.mlstm_layer(1, 8, 8, ff=None)] * 17), mbt=1)
    assert [e["type"] for e in events(deep)].count("residual_norm") == 2
    pk = dry(c, mbt=3)
    pk.compile()
    assert pk.graph_info()["num_folded"] == 0


def test_a_layer_without_latents_of_its_own_waits_for_the_cache_it_reads():
    c = P.config(32, 64, [P.latent_layer(2, 16, 16, 24, 32, 5, None), P.latent_layer(3, 8, 16, 24, 32, 9, None, kv_from=0)])
    pk = dry(c)
    ev = events(pk)
    att = [i for i, e in enumerate(ev) if e["type"] == "ext_attention"]
    assert sum(e["type"] == "latent_append" for e in ev) == 1
    assert [d[0] for d in ev[att[1]]["deps"]] == [att[1] - 1]      # its queries, which lie behind the first layer


def test_real_sizes_compile_in_every_batch_size():
    c = P.config(512, 1024, [P.latent_layer(16, 128, 128, 384, 512, 300, 4096), P.attention_layer(16, 4, 128, 1024, 130),
                             P.mlstm_layer(4, 256, 512, ff=4096), P.latent_layer(40, 24, 200, 70, 512, 7, None, kv_from=0)])
    for mbt in (1, 2, 8, 9, 64):
        dry(c, mbt=mbt).compile()
    dry(c, mbt=64, dtype=torch.float32).compile()


def test_refused_graphs_say_why():
    with pytest.raises(mi.MpkError, match="64 tokens"):
        dry(mixed_config(), mbt=65).compile()
    with pytest.raises(mi.MpkError, match="head sizes"):
        dry(P.config(32, 64, [P.attention_layer(1, 1, 264, 8)])).compile()
    with pytest.raises(mi.MpkError, match="head sizes"):
        dry(P.config(32, 64, [P.latent_layer(1, 16, 16, 16, 520, 8)])).compile()
    pk = mi.PersistentKernel(**{**mi.PersistentKernel.get_default_init_parameters(), "test_mode": True, "dry_run": True, "max_num_batched_tokens": 4})
    x, w = pk.new_tensor((4, 64), dtype=mi.float32, name="x"), pk.new_tensor((32,), name="w")
    with pytest.raises(ValueError, match="temperature"):
        pk.qkv_append_layer(x, x, None, None, None, None, heads=1, kv_heads=1, dim=8, vdim=8, q_col=0, rot_dims=0, eps=1e-5, whole_norm=True,
                            temperature=(0.1, 0))
    pk.residual_norm_layer(x, norm_weight=w, added_row=w, output=pk.new_tensor((4, 64), name="o"), columns=32)
    with pytest.raises(mi.MpkError, match="leading columns"):
        pk.compile()


def test_configuration_reader_takes_every_value_and_refuses_the_unknown():
    c = mixed_config(eps=3e-4, logit_scale=0.3, buckets=11, mul_prev=5, mul_cur=3)
    cfg = RuludraConfig.from_dict(json.loads(json.dumps(c)))
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.logit_scale, cfg.bigram) == (96, 64, 3e-4, 0.3, (11, 5, 3))
    l, a, m, k = (cfg.layers[n].mixer for n in range(4))
    assert (l.heads, l.dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.window, l.kv_from) == (3, 12, 20, 24, 40, 0.25, 21, None)
    assert (k.heads, k.dim, k.vdim, k.q_rank, k.scale, k.window, k.kv_from) == (5, 16, 8, 36, 0.2, 50, 0)
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.window, a.temperature) == (6, 2, 20, 0.2, 30, (0.4, 50))
    assert m == MlstmSpec(2, 16, 24, 9.0) and cfg.layers[4].mixer.temperature == (0.7, 16)
    assert [x.ff for x in cfg.layers] == [80, None, 48, None, 72, None]
    plain = json.loads(json.dumps(c))
    del plain["layers"][1]["mixer"]["q_temp"], plain["layers"][1]["mixer"]["mask"]
    a = RuludraConfig.from_dict(plain).layers[1].mixer
    assert (a.temperature, a.window) == (None, 0)
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mlp", "kind"), "sparse"), (("layers", 1, "mixer", "kv_heads"), 4),
                        (("layers", 1, "mixer", "vdim"), 16), (("layers", 3, "mixer", "kv_from"), 1), (("layers", 3, "mixer", "kv_from"), 3),
                        (("layers", 3, "mixer", "kv_rank"), 24)):
        bad = json.loads(json.dumps(c))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            RuludraConfig.from_dict(bad)


def test_registry_picks_runner_and_kernel_family_by_config(tmp_path):
    c = mixed_config()
    save_checkpoint(str(tmp_path / "p"), c, P.make_weights(c, 1))
    cls, dtypes = mi.runner_class(str(tmp_path / "p"))
    assert cls.__name__ == "RuludraRunner" and torch.float32 in dtypes and registry.kernel_family(str(tmp_path / "p")) == "hybrid"
    assert mi.get_builder("Ruludra") is RuludraBuilder


def test_position_frequencies_are_exact_turns():
    """position * frequency modulo 2^64 is the angle's fraction of a turn, far beyond what a float32 angle keeps."""
    for width in (1, 7, 64):
        f = mi.PersistentKernel.position_frequencies(width)
        assert f.shape == ((width + 1) // 2,)
        ref = ops.sinusoids(3, width, D)
        for pos in (0, 1, 2, 999, 123457):
            turns = [(pos * int(v)) % 2 ** 64 / 2 ** 64 for v in f]
            for j in range(width):
                a = pos * 10000.0 ** (-2.0 * (j // 2) / width)
                want = math.cos(a) if j % 2 else math.sin(a)
                got = (math.cos if j % 2 else math.sin)(2 * math.pi * turns[j // 2])
                assert abs(got - want) < 1e-9
                assert pos > 2 or abs(float(ref[pos, j]) - want) < 1e-12


# ---- the oracle's mechanisms against independent formulations
def test_bigram_rows_use_the_last_row_for_the_first_token():
    assert ops.bigram_rows([4], 10, 3, 5) == [10]
    assert ops.bigram_rows([4, 0, 7], 10, 3, 5) == [10, (4 * 3) % 10, 35 % 10]


@pytest.mark.parametrize("window", [1, 4, 0, 50])
def test_biased_attention_equals_masked_softmax(window):
    g = torch.Generator().manual_seed(2)
    T, H, G = 13, 4, 2
    q, k, v = torch.randn(T, H, 6, generator=g, dtype=D), torch.randn(T, G, 6, generator=g, dtype=D), torch.randn(T, G, 3, generator=g, dtype=D)
    r1, r2 = torch.rand(H, generator=g, dtype=D) * 2, torch.rand(H, generator=g, dtype=D)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = (j <= i) & (i - j < (window or T))
    kk, vv = (t.repeat_interleave(H // G, 1) for t in (k, v))
    s = torch.einsum("ihd,jhd->hij", q, kk) * 0.3 - r1[:, None, None] * torch.log1p(r2[:, None, None] * (i - j).clamp(min=0))
    ref = torch.einsum("hij,jhd->ihd", s.masked_fill(~seen, float("-inf")).softmax(-1), vv)
    torch.testing.assert_close(ops.biased_attention(q, k, v, 0.3, window, r1, r2), ref)


def test_latent_attention_equals_its_absorbed_form():
    g = torch.Generator().manual_seed(3)
    T, H, d, dv, r = 11, 3, 5, 4, 7
    q, c = torch.randn(T, H, d, generator=g, dtype=D), torch.randn(T, r, generator=g, dtype=D)
    uk, uv = torch.randn(H * d, r, generator=g, dtype=D), torch.randn(H * dv, r, generator=g, dtype=D)
    qa = torch.einsum("thd,hdr->thr", q, uk.view(H, d, r))
    mid = ops.window_attention(qa, c[:, None], c[:, None], 0.4, 4)
    torch.testing.assert_close(ops.latent_window_attention(q, c, uk, uv, 0.4, 4), torch.einsum("thr,hvr->thv", mid, uv.view(H, dv, r)))


def test_poly_norm_depth_average_and_temperature():
    g = torch.Generator().manual_seed(4)
    z, co = torch.randn(3, 9, generator=g, dtype=D), torch.tensor([0.3, -0.7, 1.1, 0.2], dtype=D)
    ms = lambda p: (z ** (2 * p)).mean(-1, keepdim=True)
    want = co[3] + sum(co[p - 1] * z ** p / (ms(p) + 1e-3).sqrt() for p in (1, 2, 3))
    torch.testing.assert_close(ops.poly_norm(z, co, 1e-3), want)
    h = [torch.randn(4, 5, generator=g, dtype=D) for _ in range(3)]
    torch.testing.assert_close(ops.depth_average(h, co[:3]), torch.einsum("j,jtd->td", co[:3], torch.stack(h)))
    assert [ops.query_temperature(p, 0.5, 4) for p in (0, 2, 3, 7)] == [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)]
