"""Ruludra end to end on the GPU against oracle/ruludra.py: prompts, decoding, portions, mixed batches, reused pages and slots,
long decoding, other sizes, shared keys and values, generation through the scheduler, the trace runner."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from ruludra_util import mixed_config, runner
from oracle import ruludra as P
from palarax_util import cuts_of, rel, run_portions, save_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 5e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


@pytest.fixture(scope="module")
def model():
    c = mixed_config()
    w = P.make_weights(c, 3)
    orc = P.RuludraOracle(c, w)
    toks = {r: random.Random(r).choices(range(c["vocab"]), k=n) for r, n in (("a", 150), ("b", 61), ("c", 17), ("d", 1), ("e", 40))}
    return c, w, toks, {r: orc.logits(t) for r, t in toks.items()}


@pytest.fixture(scope="module", params=[torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def session(request, model):
    from mirage_b200 import OnlineSession
    c, w, _, _ = model
    return OnlineSession(runner(c, w, request.param)), request.param


def close(got, ref, dt):
    rows = (got.double() - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(rows.max()) < TOL[dt], (int(rows.argmax()), float(rows.max()))


@pytest.mark.parametrize("cuts", [[10 ** 6], [1], [2], [64, 1, 1, 1], [37, 2, 5], [16], [15, 17], [3]], ids=str)
def test_portions_agree_with_the_whole_sequence(session, model, cuts):
    s, dt = session
    _, _, toks, ref = model
    close(run_portions(s, "a", toks["a"], cuts_of(len(toks["a"]), cuts)), ref["a"], dt)


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
            close(torch.cat(got[rid]), ref[live.pop(rid)[0]], dt)


@BOTH
@pytest.mark.parametrize("tokens", [1, 2, 4, 8, 20])
def test_batch_sizes_select_other_bodies(model, dtype, tokens):
    from mirage_b200 import OnlineSession
    c, w, toks, ref = model
    s = OnlineSession(runner(c, w, dtype, tokens=tokens))
    for rid in ("b", "c"):
        close(run_portions(s, rid, toks[rid], cuts_of(len(toks[rid]), [23, 1, 1])), ref[rid], dtype)


SHAPES = {
    "every size odd": P.config(51, 37, [P.mlstm_layer(3, 5, 7, ff=17), P.latent_layer(3, 7, 9, 11, 13, 7, 19), P.attention_layer(3, 3, 9, 5, 7),
                                        P.latent_layer(1, 5, 3, 7, 13, 11, None, kv_from=1)], eps=1e-4, logit_scale=1.0, buckets=7, mul_prev=3, mul_cur=1),
    "ones": P.config(33, 32, [P.latent_layer(1, 1, 1, 1, 1, 1, 1), P.attention_layer(1, 1, 1, 1, 1, every=1), P.mlstm_layer(1, 1, 1, ff=1)],
                     buckets=1, mul_prev=1, mul_cur=1),
    "attention only, wide heads": P.config(64, 64, [P.attention_layer(4, 2, 136, 33, 100, scale=0.08, every=3), P.attention_layer(8, 1, 72, 64, None, coef=0.0),
                                                    P.attention_layer(2, 2, 200, 500, 64)], logit_scale=3.0, buckets=5000, mul_prev=99991, mul_cur=70001),
    "recurrent only": P.config(200, 128, [P.mlstm_layer(2, 130, 40, ff=130), P.mlstm_layer(3, 40, 136, cap=4.0, ff=None)], eps=1e-3),
    "shared twice, other masks": P.config(70, 96, [P.latent_layer(2, 24, 40, 56, 72, 64, None), P.mlstm_layer(2, 24, 40, ff=None),
                                                   P.latent_layer(6, 40, 8, 24, 72, 9, 40, kv_from=0, scale=0.4), P.attention_layer(6, 3, 24, 30, None),
                                                   P.latent_layer(17, 8, 24, 130, 72, 70, None, kv_from=0)], logit_scale=0.1),
    "windows beyond the sequence": P.config(40, 64, [P.latent_layer(4, 16, 16, 16, 192, 500, 90, scale=0.1), P.attention_layer(4, 4, 16, 400, None),
                                                     P.latent_layer(20, 32, 16, 48, 320, 200, None)]),
}


@pytest.mark.parametrize("name", list(SHAPES))
@BOTH
def test_other_sizes(dtype, name):
    from mirage_b200 import OnlineSession
    c = SHAPES[name]
    w = P.make_weights(c, 8)
    toks = random.Random(1).choices(range(c["vocab"]), k=75)
    ref = P.RuludraOracle(c, w).logits(toks)
    s = OnlineSession(runner(c, w, dtype, page=8, pages=40))
    for cuts in ([75], [64, 1], [9, 2, 1]):
        close(run_portions(s, "r", toks, cuts_of(75, cuts)), ref, dtype)


def test_shared_layers_have_no_cache_of_their_own(model):
    c, w, _, _ = model
    r = runner(c, w, torch.float32)
    assert [sorted(st) for st in r.state] == [["latent"], ["k", "v"], ["memory", "normaliser"], [], ["k", "v"], ["memory", "normaliser"]]
    assert not {"l3.mix.dkv", "l3.mix.dkv.norm"} & set(w)


@BOTH
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_a_key_counts_up_to_the_windows_edge(dtype, kind):
    """One token's value stands out among equal scores: logits tell whether it is in the window, from prompt rows and decoded tokens."""
    from mirage_b200 import OnlineSession
    window, T, loud = 24, 90, 41
    layer = P.attention_layer(2, 1, 16, window, None, scale=1.0) if kind == "attention" else P.latent_layer(2, 16, 16, 16, 24, window, None, scale=1.0)
    c = P.config(40, 64, [layer], buckets=1)
    w = P.make_weights(c, 6)
    w["l0.mix.q" if kind == "attention" else "l0.mix.uq"][:] = 0.0      # equal scores, up to the distance
    w["bigram"][:] = 0.0
    w["l0.norm1b"] *= 4.0
    toks = random.Random(4).choices(range(39), k=T)
    toks[loud] = 39
    quiet = toks[:loud] + [3] + toks[loud + 1:]
    orc = P.RuludraOracle(c, w)
    ref = orc.logits(toks)
    moved = (ref - orc.logits(quiet)).abs().amax(-1)
    assert float(moved[loud + 1:loud + window].min()) > 0.05 and float(moved[loud + window:].max()) < 1e-9
    for cuts in ([T], [64] + [1] * 26, [50] + [1] * 40, [40, 2, 20, 28]):
        close(run_portions(OnlineSession(runner(c, w, dtype)), "r", toks, cuts_of(T, cuts)), ref, dtype)


@BOTH
def test_the_first_tokens_of_a_sequence(dtype):
    """The previous token, also across portions and beside other requests; a sequence's first token has a row of its own."""
    from mirage_b200 import OnlineSession
    c = P.config(50, 48, [P.mlstm_layer(1, 8, 8, ff=None)], buckets=997, mul_prev=131, mul_cur=17)
    w = P.make_weights(c, 8)
    w["bigram"] *= 6.0
    toks = {r: random.Random(r).choices(range(50), k=n) for r, n in (("p", 9), ("q", 7), ("r", 2))}
    ref = {r: P.RuludraOracle(c, w).logits(t) for r, t in toks.items()}
    s = OnlineSession(runner(c, w, dtype))
    at, got = dict.fromkeys(toks, 0), {r: [] for r in toks}
    for step in ([("p", 1), ("q", 2)], [("q", 1), ("p", 1)], [("r", 1)], [("p", 3), ("r", 1), ("q", 1)], [("q", 3), ("p", 4)]):
        entries = [(r, toks[r][at[r]:at[r] + n], list(range(n))) for r, n in step]
        for (r, n), l in zip(step, s.step(entries, [])):
            got[r].append(l)
            at[r] += n
    for r in toks:
        close(torch.cat(got[r]), ref[r], dtype)


def test_long_decoding_does_not_drift(model):
    """700 single-token steps in 32-bit: the carried state stays the sequence's, far past every portion and page."""
    from mirage_b200 import OnlineSession
    c, w, _, _ = model
    toks = random.Random(9).choices(range(c["vocab"]), k=720)
    ref = P.RuludraOracle(c, w).logits(toks)
    s = OnlineSession(runner(c, w, torch.float32, slots=2, requests=4, pages=46, max_seq=730))
    got = run_portions(s, "r", toks, [20] + [1] * 700)
    close(got, ref, torch.float32)


@BOTH
def test_greedy_generation_through_the_scheduler(model, dtype):
    """More requests than slots, prompts longer than a batch, retirement and admission on the device."""
    c, w, toks, _ = model
    prompts = [toks["a"][:70], toks["b"][:9], toks["c"][:3], toks["e"][:30], toks["d"]]
    S = 84
    r = runner(c, w, dtype, mode="offline", requests=5, slots=2, tokens=24, pages=14, page=16, max_seq=S)
    got = r.generate(prompts)
    orc = P.RuludraOracle(c, w)
    for p, g in zip(prompts, got):
        assert g[:len(p)] == p and len(g) == S
        # every chosen id is the oracle's choice for the same prefix, unless its two best are too close to call
        lg = orc.logits(g[:-1])[len(p) - 1:]
        top = lg.topk(2, -1)
        gap = (top.values[:, 0] - top.values[:, 1]) / lg.pow(2).mean().sqrt()
        same = top.indices[:, 0] == torch.tensor(g[len(p):])
        ok = same | (gap < (1e-4 if dtype == torch.float32 else 0.2))
        assert float(ok.double().mean()) >= (1.0 if dtype == torch.float32 else 0.97)
        assert float(same.double().mean()) > 0.8
    assert r.generate(prompts) == got                               # a second run starts from clean state


def test_generation_through_the_model_wrapper(model):
    import mirage_b200 as mi
    from mirage_b200.builders.ruludra import RuludraConfig, RuludraModelConfig, allocate_state
    c, w, toks, _ = model
    cfg = RuludraConfig.from_dict(c)
    prompts = [toks["c"][:6], toks["b"][:10]]
    sizes = dict(max_num_batched_requests=2, max_num_batched_tokens=8, max_num_pages=8, page_size=16)
    state = allocate_state(cfg, slots=2, max_num_pages=8, page_size=16, dtype=torch.float32, device="cuda",
                           num_workers=mi.get_configurations_from_gpu(0)[0])
    m = mi.MPK(mi.MPKMetadata(mode="offline", total_num_requests=2, max_seq_length=40, model_name="Ruludra",
                              model_config=RuludraModelConfig(cfg, {k: v.cuda() for k, v in w.items()}, state, torch.float32), **sizes))
    m.build()
    m.compile()
    out = m.run_ids(prompts)
    orc = P.RuludraOracle(c, w)
    assert [o[:len(p) + 5] for o, p in zip(out, prompts)] == [orc.greedy(p, 5) for p in prompts]


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
    tol = 4 * TOL[getattr(torch, dtype)]
    assert rel(read(0), ref["b"][[0, 39]]) < tol
    assert rel(read(2), torch.stack([ref["e"][39], ref["b"][40]])) < tol
    if dtype == "float32":
        g = subprocess.run([sys.executable, "-m", "mirage_b200", "generate", "--model", str(tmp_path / "m"), "--dtype", dtype,
                            "--prompt", ",".join(map(str, toks["c"][:6])), "--prompt", "5", "--max-new-tokens", "4"], cwd=ROOT,
                           text=True, capture_output=True, timeout=300)
        assert g.returncode == 0, g.stderr[-2000:]
        orc = P.RuludraOracle(c, w)
        assert [json.loads(l) for l in g.stdout.splitlines()] == [orc.greedy(toks["c"][:6], 4), orc.greedy([5], 4)]
