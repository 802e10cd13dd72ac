"""CPU checks of the Bebuzen graph (dry run, no CUDA call) -- layer sequence, dependencies, folding, refused shapes -- of its
configuration reader and of its oracle against independent formulations."""
import json
import math

import pytest
import torch

import mirage_b200 as mi
from bebuzen_util import mixed_config
from mirage_b200.builders import registry
from mirage_b200.builders.bebuzen import BebuzenBuilder, BebuzenConfig, BebuzenModelConfig, allocate_state
from mirage_b200.builders.hybrid import RotaryScaling, rotary_tables
from oracle import bebuzen as P
from oracle import hybrid_ops as ops
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
    cfg = BebuzenConfig.from_dict(c)
    BebuzenBuilder(pk).build_from_config(BebuzenModelConfig(cfg, P.make_weights(c, 1), allocate_state(
        cfg, slots=mbr, max_num_pages=pages, page_size=page, dtype=dtype, device="cpu", num_workers=pk.num_workers), dtype))
    return pk


def events(pk):
    pk.compile()
    return json.loads(pk.dump_task_graph())["events"]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_layer_sequence_and_dependencies(dtype):
    ev = events(dry(mixed_config(), dtype=dtype))
    types = [e["type"] for e in ev]
    lin, moe = ("linear", "moe_gemm") if dtype == torch.bfloat16 else ("linear_f32", "moe_gemm_f32")
    diff = [lin, "short_conv", "qkv_append", "ext_attention", "diff_combine", lin, "residual_norm"]
    sink = [lin, "qkv_append", "ext_attention", lin, "residual_norm"]
    mamba = [lin, "short_conv", lin, "selective_scan", lin, "residual_norm"]
    routed = [lin, "moe_routing", moe, moe, "residual_norm"]
    shared = [lin, "moe_routing", lin, lin, moe, moe, "residual_norm"]
    dense = [lin, lin, "residual_norm"]
    assert types == ["batch", "embed_f32", "residual_norm"] + diff + routed + mamba + shared + sink + diff + dense + mamba + \
        [lin, "argmax_partial", "argmax_reduce"]
    deps = lambda i: sorted(d[0] for d in ev[i]["deps"])
    j = len(types) - 1 - types[::-1].index("moe_routing")          # an expert layer with a shared expert: the two run side by side
    assert deps(j) == [j - 1] and deps(j + 1) == [j - 2] and deps(j + 3) == [j] and deps(j + 5) == [j + 2, j + 4]


def test_norms_fold_into_the_linears_of_single_token_graphs():
    c = mixed_config()
    pk = dry(c, mbt=1)
    ev = events(pk)
    # the norms in front of a single linear: five mixers, of which the first reads the embedding, the dense feed-forward, the head; not
    # those in front of the experts nor the one that sums the experts up (two expert layers, each followed by a mixer)
    assert sum(e.get("prologue") == "residual_norm" for e in ev) == pk.graph_info()["num_folded"] == 5
    assert sum(e["type"] == "residual_norm" for e in ev) == 4
    pk = dry(c, mbt=3)
    pk.compile()
    assert pk.graph_info()["num_folded"] == 0


def test_a_layer_without_keys_of_its_own_waits_for_the_cache_it_reads():
    """Two layers in a row over one cache: the second one's attention depends on its queries only, which lie behind the first layer."""
    c = P.config(32, 64, [P.diff_layer(2, 1, 16, 16, 8, 5, 2, None), P.diff_layer(2, 1, 16, 16, 8, 5, 2, None, kv_from=0)])
    pk = dry(c)
    ev = events(pk)
    att = [i for i, e in enumerate(ev) if e["type"] == "ext_attention"]
    app = [i for i, e in enumerate(ev) if e["type"] == "qkv_append"]
    assert [d[0] for d in ev[att[1]]["deps"]] == [app[1]] and app[0] < att[0] < app[1]


def test_wide_layers_and_many_experts_compile_in_every_batch_size():
    c = P.config(64, 256, [P.diff_layer(16, 4, 64, 128, 64, 1024, 4, P.moe(64, 8, 96, 2.0, 200)), P.mamba_layer(1024, 16, 32, 4, P.dense(130)),
                           P.sink_layer(16, 2, 128, 128, 128, 512, 4, P.moe(128, 4, 64, 1.0, None)), P.mamba_layer(40, 128, 700, 4, None)])
    for mbt in (1, 2, 8, 9, 64):
        dry(c, mbt=mbt).compile()
    dry(c, mbt=64, dtype=torch.float32).compile()


def test_refused_graphs_say_why():
    with pytest.raises(mi.MpkError, match="64 tokens"):
        dry(mixed_config(), mbt=65).compile()
    with pytest.raises(mi.MpkError, match="state sizes"):
        dry(P.config(32, 64, [P.mamba_layer(64, 129, 4, 4, None)])).compile()
    with pytest.raises(mi.MpkError, match="head sizes"):
        dry(P.config(32, 64, [P.diff_layer(1, 1, 136, 8, 8, 5, 2, None)])).compile()


def test_configuration_reader_takes_every_value_and_refuses_the_unknown():
    c = mixed_config(eps=3e-4)
    cfg = BebuzenConfig.from_dict(json.loads(json.dumps(c)))
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.residual_mult) == (96, 64, 3e-4, 0.8)
    d, m, s, k = (cfg.layers[n].mixer for n in range(4))
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.taps, d.diff, d.scale, d.window, d.keep_first, d.kv_from) == (4, 2, 12, 20, 3, 0.4, 0.15, 21, 0, None)
    assert (d.rot_base, d.rot_dims, d.scaling, d.MAPS, d.q_rows, d.k_rows, d.v_rows) == (20000.0, 8, RotaryScaling(3.0, 1.0, 5.0, 300.0), 2, 96, 48, 40)
    assert (m.inner, m.state, m.dt_rank, m.taps) == (72, 10, 5, 4)
    assert (s.heads, s.kv_heads, s.dim, s.vdim, s.window, s.keep_first, s.rot_base, s.rot_dims, s.scaling, s.scale, s.MAPS) == \
        (3, 1, 20, 12, 30, 5, 3000.0, 12, None, 0.2, 1)
    assert (k.kv_from, k.window, k.diff, k.heads) == (0, 50, 0.7, 6)
    e = cfg.layers[1].ff
    assert (e.experts, e.top, e.ff, e.scale, e.shared_ff) == (9, 3, 24, 0.7, 56)
    assert cfg.layers[0].ff.shared_ff is None and cfg.layers[3].ff == 80 and cfg.layers[4].ff is None
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 3, "mlp", "kind"), "sparse"), (("layers", 0, "mixer", "rot", "dims"), 14),
                        (("layers", 0, "mixer", "rot", "dims"), 5), (("layers", 2, "mixer", "kv_heads"), 2), (("layers", 1, "mlp", "router", "top"), 10),
                        (("layers", 3, "mixer", "kv_from"), 1), (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "dim"), 16)):
        bad = json.loads(json.dumps(c))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            BebuzenConfig.from_dict(bad)


def test_registry_picks_runner_and_kernel_family_by_config(tmp_path):
    c = mixed_config()
    save_checkpoint(str(tmp_path / "p"), c, P.make_weights(c, 1))
    cls, dtypes = mi.runner_class(str(tmp_path / "p"))
    assert cls.__name__ == "BebuzenRunner" and torch.float32 in dtypes and registry.kernel_family(str(tmp_path / "p")) == "hybrid"
    assert mi.get_builder("Bebuzen") is BebuzenBuilder


@pytest.mark.parametrize("scaling", [None, (5.0, 1.0, 6.0, 640), (8.0, 2.0, 3.0, 100), (2.0, 0.5, 32.0, 8192)])
def test_rotary_tables_equal_the_oracles_frequencies(scaling):
    kw = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    for base, dims in ((20000.0, 40), (300000.0, 8), (50.0, 2)):
        cos, sin = rotary_tables(base, dims, 300, "cpu", RotaryScaling(**{k: float(v) for k, v in kw.items()}) if kw else None)
        f = torch.tensor(ops.rotary_frequencies(base, dims, kw), dtype=D)
        a = torch.arange(300, dtype=D)[:, None] * f
        torch.testing.assert_close(cos, a.cos().float(), rtol=0, atol=2e-7)
        torch.testing.assert_close(sin, a.sin().float(), rtol=0, atol=2e-7)
        # the definition by wavelengths
        for i in range(dims // 2):
            g = base ** (-2.0 * i / dims)
            if kw:
                wave = 2 * math.pi / g
                if wave > kw["original"] / kw["low"]:
                    g /= kw["factor"]
                elif wave >= kw["original"] / kw["high"]:
                    s = (kw["original"] / wave - kw["low"]) / (kw["high"] - kw["low"])
                    g = (1 - s) * g / kw["factor"] + s * g
            assert abs(float(f[i]) - g) < 1e-12


# ---- the oracle's mechanisms against independent formulations
def test_rotation_layouts():
    g = torch.Generator().manual_seed(1)
    x, pos, freqs = torch.randn(5, 2, 8, generator=g, dtype=D), torch.arange(5), [0.7, 0.2, 0.05]
    z = torch.polar(torch.ones(5, 1, 3, dtype=D), pos[:, None, None].to(D) * torch.tensor(freqs, dtype=D))
    halves = torch.complex(x[..., :3], x[..., 3:6]) * z
    pairs = torch.view_as_complex(x[..., :6].reshape(5, 2, 3, 2).contiguous()) * z
    torch.testing.assert_close(ops.rotate_pairs(x, pos, freqs, False), torch.cat([halves.real, halves.imag, x[..., 6:]], -1))
    torch.testing.assert_close(ops.rotate_pairs(x, pos, freqs, True), torch.cat([torch.view_as_real(pairs).flatten(-2), x[..., 6:]], -1))


@pytest.mark.parametrize("window,keep", [(4, 0), (4, 2), (1, 3), (0, 0), (50, 5)])
def test_windowed_attention_equals_masked_softmax(window, keep):
    g = torch.Generator().manual_seed(2)
    T, H, G = 13, 4, 2
    q, k, v = torch.randn(T, H, 6, generator=g, dtype=D), torch.randn(T, G, 6, generator=g, dtype=D), torch.randn(T, G, 3, generator=g, dtype=D)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = (j <= i) & ((i - j < (window or T)) | (j < keep))
    kk, vv = (t.repeat_interleave(H // G, 1) for t in (k, v))
    s = (torch.einsum("ihd,jhd->hij", q, kk) * 0.3).masked_fill(~seen, float("-inf"))
    for sink in (False, True):
        full = torch.cat([s, torch.zeros(H, T, 1, dtype=D)], -1).softmax(-1)[..., :-1] if sink else s.softmax(-1)
        torch.testing.assert_close(ops.window_attention(q, k, v, 0.3, window, keep, sink), torch.einsum("hij,jhd->ihd", full, vv))


def test_selective_scan_equals_the_quadratic_form():
    g = torch.Generator().manual_seed(3)
    T, C, n = 11, 5, 3
    x, dt = torch.randn(T, C, generator=g, dtype=D), torch.rand(T, C, generator=g, dtype=D)
    A, Bm, Cm, skip = -torch.rand(C, n, generator=g, dtype=D), *(torch.randn(T, n, generator=g, dtype=D) for _ in range(2)), torch.randn(C, generator=g, dtype=D)
    F = dt.cumsum(0)
    out = skip * x
    for t in range(T):
        for s in range(t + 1):
            out[t] += (torch.exp((F[t] - F[s])[:, None] * A) * Bm[s] * Cm[t]).sum(-1) * dt[s] * x[s]
    torch.testing.assert_close(ops.selective_scan(x, dt, A, Bm, Cm, skip), out)


def test_differential_attention_with_equal_maps_is_plain_attention_up_to_its_norm():
    g = torch.Generator().manual_seed(4)
    T, H, d, dv = 9, 2, 4, 6
    q, k, v = (torch.randn(T, H, w, generator=g, dtype=D) for w in (d, d, dv))
    o = ops.diff_attention(torch.stack([q, q], 2), torch.stack([k, k], 2), v, 0.4, torch.tensor(0.25, dtype=D), 0.6, 0.0)
    torch.testing.assert_close(o, 0.4 * ops.rms_unit(ops.window_attention(q, k, v, 0.4), 0.0))
    l = [torch.randn(d, generator=g, dtype=D) for _ in range(4)]
    assert float(ops.diff_lambda(*l, 0.3)) == pytest.approx(math.exp(float(l[0] @ l[1])) - math.exp(float(l[2] @ l[3])) + 0.3)


def test_softmax_choice_keeps_probabilities():
    z = torch.tensor([0.1, 2.0, -1.0, 1.5], dtype=D)
    chosen, p = ops.softmax_choice(z, 2)
    assert chosen == [1, 3] and float(p.sum()) < 1.0
    torch.testing.assert_close(p, torch.softmax(z, -1)[[1, 3]])
