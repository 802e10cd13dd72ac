"""Palarax end to end on the GPU against oracle/palarax.py: prompts, decoding, portions, mixed batches, reused pages and
slots, long decoding, other sizes, generation through the scheduler, the trace runner."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import palarax as P
from oracle.batching import REQ_CLOSE, REQ_HOLD, REQ_RUN, BatchState
from palarax_util import cuts_of, mixed_config, rel, run_portions, runner, save_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 4e-2}


@pytest.fixture(scope="module")
def model():
    c = mixed_config()
    w = P.make_weights(c, 3)
    orc = P.PalaraxOracle(c, w)
    toks = {r: random.Random(r).choices(range(c["vocab"]), k=n) for r, n in (("a", 150), ("b", 61), ("c", 17), ("d", 1), ("e", 40))}
    return c, w, toks, {r: orc.logits(t) for r, t in toks.items()}


@pytest.fixture(scope="module", params=[torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def session(request, model):
    from mirage_b200 import OnlineSession
    c, w, _, _ = model
    r = runner(c, w, request.param)
    return OnlineSession(r), request.param


@pytest.mark.parametrize("cuts", [[10 ** 6], [1], [2], [64, 1, 1, 1], [37, 2, 5], [16], [15, 17], [3]], ids=str)
def test_portions_agree_with_the_whole_sequence(session, model, cuts):
    s, dt = session
    _, _, toks, ref = model
    got = run_portions(s, "a", toks["a"], cuts_of(len(toks["a"]), cuts))
    assert rel(got, ref["a"]) < TOL[dt], rel(got, ref["a"])


def test_mixed_batches_and_reused_pages_and_slots(session, model):
    """Requests of unequal length come and go beside one another, paused now and then; more of them, over time, than slots."""
    s, dt = session
    c, _, toks, ref = model
    rng = random.Random(7)
    waiting = [(f"{r}{k}", r) for k in range(3) for r in ("a", "b", "c", "d", "e")]
    rng.shuffle(waiting)
    live, got = {}, {}
    while waiting or live:
        while waiting and len(live) < 4:
            rid, r = waiting.pop()
            live[rid], got[rid] = [r, 0], []
        entries, end = [], []
        for rid, st in live.items():
            if rng.random() < 0.2:
                continue                                              # left out of this step
            r, at = st
            n = min(rng.choice([1, 1, 2, 5, 16, 33, 70]), len(toks[r]) - at)
            entries.append((rid, toks[r][at:at + n], list(range(n))))
            st[1] += n
            if st[1] == len(toks[r]):
                end.append(rid)
        for (rid, _, _), l in zip(entries, s.step(entries, end)):
            got[rid].append(l)
        for rid in end:
            r = live.pop(rid)[0]
            assert rel(torch.cat(got[rid]), ref[r]) < TOL[dt], (rid, rel(torch.cat(got[rid]), ref[r]))


def test_only_the_wanted_places_come_back_in_their_order(session, model):
    s, dt = session
    _, _, toks, ref = model
    out = s.step([("p", toks["b"], [60, 3, 3]), ("q", toks["c"], []), ("r", toks["e"][:5], [4])], ["p", "q", "r"])
    assert [tuple(o.shape) for o in out] == [(3, 96), (0, 96), (1, 96)]
    assert rel(out[0], ref["b"][[60, 3, 3]]) < TOL[dt] and rel(out[2], ref["e"][4:5]) < TOL[dt]


def test_errors_leave_the_session_usable(session, model):
    s, dt = session
    _, _, toks, ref = model
    for bad in ([("x", [1] * 500, [])], [("x", [1], []), ("x", [2], [])]):
        with pytest.raises(ValueError):
            s.step(bad)
    with pytest.raises(RuntimeError):
        s.step([(f"x{i}", [1], []) for i in range(9)])
    assert not s._live and len(s._free) + len(s._closing) == 8
    assert rel(s.step([("y", toks["c"], list(range(17)))], ["y"])[0], ref["c"]) < TOL[dt]


@pytest.mark.parametrize("tokens", [1, 4, 8, 20])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_batch_sizes_select_other_linear_bodies(model, dtype, tokens):
    from mirage_b200 import OnlineSession
    c, w, toks, ref = model
    s = OnlineSession(runner(c, w, dtype, tokens=tokens))
    for rid in ("b", "c"):
        assert rel(run_portions(s, rid, toks[rid], cuts_of(len(toks[rid]), [23, 1, 1])), ref[rid]) < TOL[dtype]


SHAPES = {
    "every size odd": P.config(51, 36, [P.parallel_layer(3, 1, 12, 6, 15, 5, 2, ff=21), P.mlstm_layer(3, 9, 11, ff=17)], 1e-4),
    "ones": P.config(33, 32, [P.parallel_layer(1, 1, 16, 2, 16, 16, 1, ff=32), P.mlstm_layer(1, 1, 4, ff=None)], 1e-6),
    "attention only, wide heads": P.config(64, 64, [P.parallel_layer(2, 1, 136, 96, 32, 2, 5, softcap=3.0, ff=64)] * 2, 1e-5),
    "recurrent only": P.config(200, 128, [P.mlstm_layer(4, 40, 72, cap=3.0, ff=128)] * 3, 1e-3),
    "grouped heads, one block": P.config(70, 96, [P.parallel_layer(8, 1, 24, 24, 80, 1, 4, scale=1.0, left_scale=1.5,
                                                                    right_scale=0.25)], 1e-5),
    "large head sizes": P.config(40, 64, [P.mlstm_layer(1, 264, 130, ff=64), P.parallel_layer(4, 4, 80, 40, 96, 2, 3)], 1e-5),
}


@pytest.mark.parametrize("name", list(SHAPES))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_other_sizes(dtype, name):
    from mirage_b200 import OnlineSession
    c = SHAPES[name]
    w = P.make_weights(c, 5)
    toks = random.Random(1).choices(range(c["vocab"]), k=75)
    ref = P.PalaraxOracle(c, w).logits(toks)
    s = OnlineSession(runner(c, w, dtype, page=8, pages=40))
    for cuts in ([75], [64, 1], [9, 2, 1]):
        got = run_portions(s, "r", toks, cuts_of(75, cuts))
        assert rel(got, ref) < TOL[dtype], (cuts, rel(got, ref))


def test_long_decoding_does_not_drift(model):
    """700 single-token steps in 32-bit: the carried state stays the sequence's, far past every portion and page."""
    from mirage_b200 import OnlineSession
    c, w, _, _ = model
    toks = random.Random(9).choices(range(c["vocab"]), k=720)
    ref = P.PalaraxOracle(c, w).logits(toks)
    s = OnlineSession(runner(c, w, torch.float32, slots=2, requests=4, pages=46, max_seq=730))
    got = run_portions(s, "r", toks, [20] + [1] * 700)
    assert rel(got, ref) < TOL[torch.float32]
    assert rel(got[-50:], ref[-50:]) < TOL[torch.float32]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_greedy_generation_through_the_scheduler(model, dtype):
    """More requests than slots, prompts longer than a batch, retirement and admission on the device."""
    c, w, toks, _ = model
    prompts = [toks["a"][:70], toks["b"][:9], toks["c"][:3], toks["e"][:30], toks["d"]]
    S = 84
    r = runner(c, w, dtype, mode="offline", requests=5, slots=2, tokens=24, pages=14, page=16, max_seq=S)
    got = r.generate(prompts)
    orc = P.PalaraxOracle(c, w)
    for p, g in zip(prompts, got):
        assert g[:len(p)] == p and len(g) == S
        # every chosen id is the oracle's choice for the same prefix, unless its two best are too close to call
        lg = orc.logits(g[:-1])[len(p) - 1:]
        top = lg.topk(2, -1)
        gap = (top.values[:, 0] - top.values[:, 1]) / lg.pow(2).mean().sqrt()
        same = top.indices[:, 0] == torch.tensor(g[len(p):])
        assert bool((same | (gap < (1e-4 if dtype == torch.float32 else 0.15))).all())
        assert float(same.double().mean()) > 0.8
    assert r.generate(prompts) == got                               # a second run starts from clean state


def test_generation_through_the_model_wrapper(model):
    import mirage_b200 as mi
    from mirage_b200.builders.palarax import PalaraxConfig, PalaraxModelConfig, allocate_state
    c, w, toks, _ = model
    cfg = PalaraxConfig.from_dict(c)
    prompts = [toks["c"][:6], toks["b"][:10]]
    sizes = dict(max_num_batched_requests=2, max_num_batched_tokens=8, max_num_pages=8, page_size=16)
    state = allocate_state(cfg, slots=2, max_num_pages=8, page_size=16, dtype=torch.float32, device="cuda",
                           num_workers=mi.get_configurations_from_gpu(0)[0])
    m = mi.MPK(mi.MPKMetadata(mode="offline", total_num_requests=2, max_seq_length=40, model_name="Palarax",
                              model_config=PalaraxModelConfig(cfg, {k: v.cuda() for k, v in w.items()}, state, torch.float32), **sizes))
    m.build()
    m.compile()
    out = m.run_ids(prompts)
    orc = P.PalaraxOracle(c, w)
    assert [o[:len(p) + 5] for o, p in zip(out, prompts)] == [orc.greedy(p, 5) for p in prompts]
    assert m.run_ids(prompts) == out


def test_sampled_ids_are_the_largest_keys_of_the_logits(model):
    from oracle import sampling_ops as so
    c, w, toks, _ = model
    flat = dict(w)
    flat["final.norm"] = (w["final.norm"].float() * 0.05 - 0.95).to(torch.bfloat16)   # logits small enough for the noise to decide
    seed = 4242
    r = runner(c, flat, torch.bfloat16, mode="offline", requests=3, slots=3, tokens=12, pages=12, max_seq=40, sampling_seed=seed)
    r.load_prompts([toks["c"], toks["b"][:5], toks["d"]])
    differs = 0
    for _ in range(12):
        r.step(1)
        n = r.mpk.status().active_tokens
        logits, ids = r.logits[:n].cpu(), r.meta["output_tokens"][:n, 0].cpu()
        keys = so.sampling_keys(logits.to(torch.bfloat16), seed, 1).float()
        top = keys.max(-1).values
        step = 2.0 ** (torch.floor(torch.log2(top.abs().clamp_min(1e-20))) - 7)       # one bf16 step at the top key
        assert bool((keys.gather(1, ids[:, None])[:, 0] >= top - 2 * step).all())
        differs += int((ids != logits.argmax(-1)).sum())
    assert differs > 0


def test_online_scheduler_matches_its_oracle_bit_for_bit(model):
    """Random posts, extensions and closes; after every launch the batch description, state slots and control words equal
    oracle/batching.py's.  One request decodes on its own (REQ_RUN)."""
    c, w, _, _ = model
    R, S, mbr, mbt, pages, page = 6, 60, 3, 12, 14, 4
    r = runner(c, w, torch.float32, requests=R, slots=mbr, tokens=mbt, pages=pages, page=page, max_seq=S)
    r.mpk.reset()
    st = BatchState(np.zeros((R, S), np.int64), np.zeros(R), max_num_batched_requests=mbr, max_num_batched_tokens=mbt,
                    max_num_pages=pages, page_size=page, online=True)
    m, rng = r.meta, random.Random(3)
    slots = torch.zeros(mbr, dtype=torch.int32, device="cuda")
    for it in range(120):
        row = rng.randrange(R)
        ctl = int(st.request_ctl[row])
        if ctl == 0:
            n = rng.randint(1, 20)
            st.tokens[row, :n] = [rng.randrange(c["vocab"]) for _ in range(n)]
            st.prompt_lengths[row], st.request_ctl[row] = n, REQ_RUN if rng.random() < 0.2 else REQ_HOLD
        elif ctl == REQ_HOLD and rng.random() < 0.5:
            n0 = int(st.prompt_lengths[row])
            n = min(S - 2, n0 + rng.randint(1, 9))
            st.tokens[row, n0:n] = [rng.randrange(c["vocab"]) for _ in range(n - n0)]
            st.prompt_lengths[row] = n
        elif ctl == REQ_HOLD:
            st.request_ctl[row] = REQ_CLOSE
        m["tokens"].copy_(torch.from_numpy(st.tokens))
        m["prompt_lengths"].copy_(torch.from_numpy(st.prompt_lengths))
        m["request_ctl"][0].copy_(torch.from_numpy(st.request_ctl))
        more = st.prepare_next_batch()
        r.step(1)
        status = r.mpk.status()
        assert bool(status.all_done) == (not more) and status.active_tokens == st.num_active_tokens
        eq = lambda key, ref: m[key].cpu().numpy().reshape(-1)[:len(ref)].tolist() == list(ref)
        npg, nreq = int(st.paged_kv_indptr[mbr]), int((st.request_ids >= 0).sum())
        assert eq("qo_indptr_buffer", st.qo_indptr) and eq("paged_kv_indptr_buffer", st.paged_kv_indptr), it
        assert eq("paged_kv_indices_buffer", st.paged_kv_indices[:npg]) and eq("request_ids", st.request_ids), it
        assert eq("paged_kv_last_page_len_buffer", st.paged_kv_last_page_len[:nreq]) and eq("step", st.step), it
        assert eq("request_ctl", st.request_ctl) and eq("input_tokens", st.input_tokens[:st.num_active_tokens]), it
        st.output_tokens[:st.num_active_tokens] = m["output_tokens"].cpu().numpy().reshape(-1)[:st.num_active_tokens]
        assert eq("tokens", st.tokens.reshape(-1)), it


def test_online_session_over_another_model():
    """Qwen3 behind the same session: two requests in portions, one left out of a step, rows used again."""
    from gpu_util import shape_of
    from mirage_b200 import OnlineSession
    from mirage_b200.builders.runner import Qwen3Runner
    from oracle.qwen3_decoder import Qwen3Config, greedy_generate, make_weights
    cfg = Qwen3Config.tiny()
    w = make_weights(cfg, seed=9)
    rng = random.Random(2)
    prompts = [rng.choices(range(cfg.vocab_size), k=n) for n in (21, 14)]
    ref = []
    for p in prompts:
        _, _, lg = greedy_generate(cfg, w, [p], 40, max_num_batched_requests=1, max_num_batched_tokens=1, max_num_pages=3, page_size=16,
                                   max_iterations=len(p), keep_logits=True)
        ref.append(torch.cat([l[:1] for l in lg]).float())
    r = Qwen3Runner(shape_of(cfg), w, total_num_requests=4, max_seq_length=40, max_num_batched_requests=2, max_num_batched_tokens=16,
                    max_num_pages=4, page_size=16, mode="online")
    s = OnlineSession(r)
    for turn in range(3):
        a, b = f"a{turn}", f"b{turn}"
        out = {0: [], 1: []}
        for cut in ([(0, 0, 5)], [(0, 5, 6), (1, 0, 9)], [(1, 9, 10)], [(0, 6, 21), (1, 10, 14)]):
            entries = [((a, b)[k], prompts[k][lo:hi], list(range(hi - lo))) for k, lo, hi in cut]
            for (k, _, _), l in zip(cut, s.step(entries, [a, b] if cut[-1][2] == 14 else [])):
                out[k].append(l)
        for k in (0, 1):
            assert float((torch.cat(out[k]) - ref[k]).abs().max()) <= 5e-2, (turn, k)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_and_command_line(model, tmp_path, dtype):
    c, w, toks, ref = model
    save_checkpoint(str(tmp_path / "m"), c, w)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks["b"][:40], "want": [0, 39]}, {"id": "y", "tokens": toks["c"], "want": []}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "y2", "tokens": toks["e"][:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y2", "tokens": toks["e"][3:], "want": [36]}, {"id": "x", "tokens": toks["b"][40:41], "want": [0]}], "end": ["x", "y2"]}]
    out = tmp_path / "out"
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", "<f4")).view(-1, c["vocab"])
    assert not (out / "1.f32").exists()
    tol = TOL[getattr(torch, dtype)]
    assert rel(read(0), ref["b"][[0, 39]]) < tol
    assert rel(read(2), torch.stack([ref["e"][39], ref["b"][40]])) < tol
    if dtype == "float32":
        g = subprocess.run([sys.executable, "-m", "mirage_b200", "generate", "--model", str(tmp_path / "m"), "--dtype", dtype,
                            "--prompt", ",".join(map(str, toks["c"][:6])), "--prompt", "5", "--max-new-tokens", "4"], cwd=ROOT,
                           text=True, capture_output=True, timeout=300)
        assert g.returncode == 0, g.stderr[-2000:]
        orc = P.PalaraxOracle(c, w)
        assert [json.loads(l) for l in g.stdout.splitlines()] == [orc.greedy(toks["c"][:6], 4), orc.greedy([5], 4)]
