"""CPU checks (dry run, no CUDA call) of hybrid graphs: layer sequence and dependencies, kernel family, refused shapes and
mixtures; the configuration reader; the registry."""
import json

import pytest
import torch

import mirage_b200 as mi
from mirage_b200.builders import registry
from mirage_b200.builders.palarax import PalaraxBuilder, PalaraxConfig, PalaraxModelConfig, allocate_state
from oracle import palarax as P
from palarax_util import mixed_config, save_checkpoint


def dry(c, *, mbr=2, mbt=16, S=64, page=16, dtype=torch.bfloat16, mode="offline", **kw):
    z = lambda *s, dt=torch.int32: torch.zeros(*s, dtype=dt)
    pages, i64 = mbr * S // page, torch.int64
    meta = {"step": z(mbr), "tokens": z(mbr, S, dt=i64), "input_tokens": z(mbt, 1, dt=i64), "output_tokens": z(mbt, 1, dt=i64),
            "num_new_tokens": z(mbr), "prompt_lengths": z(mbr), "qo_indptr_buffer": z(mbr + 1), "paged_kv_indptr_buffer": z(mbr + 1),
            "paged_kv_indices_buffer": z(pages), "paged_kv_last_page_len_buffer": z(mbr), "request_ctl": z(2, mbr), "request_ids": z(mbr)}
    pk = mi.PersistentKernel(mode=mode, max_seq_length=S, max_num_batched_requests=mbr, max_num_batched_tokens=mbt,
                             max_num_pages=pages, page_size=page, meta_tensors=meta, dry_run=True, **kw)
    cfg = PalaraxConfig.from_dict(c)
    b = PalaraxBuilder(pk)
    b.build_from_config(PalaraxModelConfig(cfg, P.make_weights(c, 1), allocate_state(
        cfg, slots=mbr, max_num_pages=pages, page_size=page, dtype=dtype, device="cpu", num_workers=pk.num_workers), dtype))
    return pk


@pytest.mark.parametrize("dtype,linear", [(torch.bfloat16, "linear"), (torch.float32, "linear_f32")])
def test_layer_sequence_and_parallel_branches(dtype, linear):
    pk = dry(mixed_config(), dtype=dtype)
    pk.compile()
    ev = json.loads(pk.dump_task_graph())["events"]
    types = [e["type"] for e in ev]
    mlstm = ["residual_norm", linear, "mlstm", linear]
    ff = ["residual_norm", linear, linear]
    par = ["residual_norm", linear, "short_conv", "qkv_append", "ext_attention", "rglru", linear]
    assert types == ["batch", "embed_f32"] + mlstm + ff + par + mlstm + ff + par + ff + \
        ["residual_norm", linear, "argmax_partial", "argmax_reduce"]
    deps = lambda i: sorted(d[0] for d in ev[i]["deps"])
    i = types.index("qkv_append")
    proj, attn, conv, rg, out = i - 2, i + 1, i - 1, i + 2, i + 3
    # the branches run side by side: both hang on the projections, only the output linear waits for both
    assert deps(i) == [proj] and deps(attn) == [i] and deps(conv) == [proj] and deps(rg) == [conv] and deps(out) == [attn, rg]


def test_online_mode_and_state_slots_are_part_of_the_graph_api():
    pk = dry(mixed_config(), mode="online")
    pk.compile()
    assert pk.graph_info()["num_tasks"] > 0
    with pytest.raises(ValueError, match="request_ctl"):
        mi.PersistentKernel(mode="online", max_seq_length=8, meta_tensors={k: v for k, v in dry(mixed_config()).meta_tensors.items()
                                                                          if k not in ("request_ctl", "request_ids")} | {
            "tokens": torch.zeros(2, 8, dtype=torch.int64)}, max_num_batched_requests=2, max_num_pages=4, page_size=16, dry_run=True)


def test_refused_graphs_say_why():
    with pytest.raises(mi.MpkError, match="64 tokens"):
        dry(mixed_config(), mbt=65).compile()
    with pytest.raises(mi.MpkError, match="head sizes"):
        dry(P.config(32, 64, [P.parallel_layer(1, 1, 264, 8, 16, 1, 2)])).compile()
    with pytest.raises(mi.MpkError, match="key sizes"):
        dry(P.config(32, 64, [P.mlstm_layer(1, 1032, 8)])).compile()
    pk = dry(mixed_config())
    a = pk.new_tensor(dims=(16, 64), name="a")
    pk.rmsnorm_layer(input=a, weight=pk.attach_input(torch.ones(64, dtype=torch.bfloat16), "g"), output=pk.new_tensor(dims=(16, 64), name="b"),
                     grid_dim=(16, 1, 1), block_dim=(128, 1, 1))
    with pytest.raises(mi.MpkError, match="not available in a hybrid graph"):
        pk.compile()


def test_configuration_reader_takes_every_value_and_refuses_the_unknown():
    c = mixed_config(eps=3e-4)
    cfg = PalaraxConfig.from_dict(json.loads(json.dumps(c)))
    assert (cfg.vocab, cfg.width, cfg.eps) == (96, 64, 3e-4) and [l.ff for l in cfg.layers] == [80, None, 48, 96]
    m = cfg.layers[1].mixer
    assert (m.left.heads, m.left.kv_heads, m.left.dim, m.left.rot_dims, m.left.rot_base, m.left.scale, m.left.softcap) == \
        (4, 2, 16, 8, 7000.0, 0.3, 20.0)
    assert (m.right.width, m.right.blocks, m.right.taps, m.left_scale, m.right_scale) == (48, 3, 3, 0.7, 0.9)
    assert cfg.layers[0].mixer.gate_cap == 9.0
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mlp", "kind"), "gated"), (("layers", 1, "mixer", "left", "vdim"), 8),
                        (("layers", 1, "mixer", "left", "kv_heads"), 3), (("layers", 1, "mixer", "right", "blocks"), 5)):
        bad = json.loads(json.dumps(c))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            PalaraxConfig.from_dict(bad)


def test_registry_picks_runner_and_kernel_family_by_config(tmp_path):
    c = mixed_config()
    save_checkpoint(str(tmp_path / "p"), c, P.make_weights(c, 1))
    cls, dtypes = mi.runner_class(str(tmp_path / "p"))
    assert cls.__name__ == "PalaraxRunner" and torch.float32 in dtypes and registry.kernel_family(str(tmp_path / "p")) == "hybrid"
    (tmp_path / "q").mkdir()
    (tmp_path / "q" / "config.json").write_text(json.dumps({"architectures": ["Qwen3ForCausalLM"]}))
    assert mi.runner_class(str(tmp_path / "q"))[0].__name__ == "Qwen3Runner" and registry.kernel_family(str(tmp_path / "q")) == "decoder"
    with pytest.raises(registry.UnsupportedDtype):
        mi.load_runner(str(tmp_path / "q"), torch.float32)
    (tmp_path / "u").mkdir()
    (tmp_path / "u" / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(KeyError):
        mi.runner_class(str(tmp_path / "u"))
    assert mi.get_builder("Palarax") is PalaraxBuilder


def test_norms_fold_into_the_linears_of_single_token_graphs():
    c = mixed_config()
    pk = dry(c, mbt=1)
    pk.compile()
    ev = json.loads(pk.dump_task_graph())["events"]
    assert "residual_norm" not in [e["type"] for e in ev]
    assert sum(e.get("prologue") == "residual_norm" for e in ev) == pk.graph_info()["num_folded"] == 8     # 4 mixers, 3 feed-forwards, head
    for kw in (dict(mbt=3), dict(mbt=1, dtype=torch.float32)):
        pk = dry(c, **kw)
        pk.compile()
        assert pk.graph_info()["num_folded"] == 0
