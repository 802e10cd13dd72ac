"""CPU checks of the oracle of hybrid graphs against independent formulations, and of the scheduler oracle's additions."""
import numpy as np
import torch

from oracle import hybrid_ops as ops
from oracle.batching import REQ_CLOSE, REQ_FREE, REQ_HOLD, REQ_RUN, BatchState

D = torch.float64


def test_mlstm_recurrence_equals_the_quadratic_form():
    g = torch.Generator().manual_seed(1)
    T, H, d, dv, cap = 19, 2, 5, 7, 6.0
    q, k = torch.randn(T, H, d, generator=g, dtype=D), torch.randn(T, H, d, generator=g, dtype=D)
    v = torch.randn(T, H, dv, generator=g, dtype=D)
    ip, fp = 3 * torch.randn(T, H, generator=g, dtype=D), 3 * torch.randn(T, H, generator=g, dtype=D) + 2
    i, f = cap * torch.tanh(ip / cap), torch.nn.functional.logsigmoid(cap * torch.tanh(fp / cap))
    F = f.cumsum(0)
    out = torch.zeros(T, H, dv, dtype=D)
    for t in range(T):
        w = torch.exp(F[t] - F[:t + 1] + i[:t + 1])                     # [s, H] unstabilised weights
        sc = torch.einsum("hd,shd->sh", q[t], k[:t + 1]) * w
        # the stabiliser m cancels except in the floor exp(-m) and the 1e-6, both relative to exp(-m)
        m = torch.maximum(F[t], (F[t] - F[:t + 1] + i[:t + 1]).max(0).values)   # running maximum that starts at 0
        den = torch.maximum(sc.sum(0).abs(), torch.ones(H, dtype=D)) + 1e-6 * torch.exp(m)
        out[t] = torch.einsum("sh,shv->hv", sc, v[:t + 1]) / den[:, None]
    torch.testing.assert_close(ops.mlstm(q, k, v, ip, fp, cap), out, rtol=1e-9, atol=1e-11)


def test_short_conv_and_gelu_match_torch():
    g = torch.Generator().manual_seed(2)
    x, w, b = (torch.randn(*s, generator=g, dtype=D) for s in ((11, 6), (6, 4), (6,)))
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (3, 0)), w[:, None], b, groups=6)[0].T
    torch.testing.assert_close(ops.short_conv(x, w, b), ref)
    torch.testing.assert_close(ops.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))


def test_rglru_equals_the_closed_form():
    g = torch.Generator().manual_seed(3)
    T, nb, s = 9, 2, 3
    u = torch.randn(T, nb * s, generator=g, dtype=D)
    ra, ri = torch.randn(nb, s, s, generator=g, dtype=D), torch.randn(nb, s, s, generator=g, dtype=D)
    rb, ib = torch.randn(nb, s, generator=g, dtype=D), torch.randn(nb, s, generator=g, dtype=D)
    lam = torch.randn(nb * s, generator=g, dtype=D)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", u.view(T, nb, s), ra) + rb).reshape(T, -1)
    i = torch.sigmoid(torch.einsum("tbi,boi->tbo", u.view(T, nb, s), ri) + ib).reshape(T, -1)
    la = -8.0 * r * torch.nn.functional.softplus(lam)
    x = torch.sqrt(1 - torch.exp(la) ** 2) * i * u
    L = la.cumsum(0)
    ref = torch.stack([sum(torch.exp(L[t] - L[j]) * x[j] for j in range(t + 1)) for t in range(T)])
    torch.testing.assert_close(ops.rglru(u, ra, rb, ri, ib, lam), ref)


def test_attention_rotation_sink_and_cap():
    g = torch.Generator().manual_seed(4)
    q, k = torch.randn(6, 4, 8, generator=g, dtype=D), torch.randn(6, 2, 8, generator=g, dtype=D)
    kk = k.repeat_interleave(2, 1)
    s = 5 * torch.tanh(torch.einsum("ihd,jhd->hij", q, kk) * 0.7 / 5)
    e = torch.exp(s) * torch.tril(torch.ones(6, 6, dtype=D))
    ref = torch.einsum("hij,jhd->ihd", e / (1 + e.sum(-1, keepdim=True)), kk)
    torch.testing.assert_close(ops.attention(q, k, k, 0.7, 5.0, True), ref)
    # a rotation keeps pair norms and turns with the position difference only
    a = ops.rotate_half_split(q, torch.arange(6) + 3, 100.0, 6)
    b = ops.rotate_half_split(q, torch.arange(6) + 10, 100.0, 6)
    torch.testing.assert_close(torch.einsum("ihd,jhd->hij", a, a), torch.einsum("ihd,jhd->hij", b, b))
    torch.testing.assert_close(a[..., 6:], q[..., 6:])


def test_scheduler_keeps_state_slots_through_compaction_and_reuses_them():
    tok = np.ones((5, 12), np.int64)
    st = BatchState(tok, np.array([2, 9, 3, 4, 2]), max_num_batched_requests=2, max_num_batched_tokens=8, max_num_pages=16,
                    page_size=4)
    held = {}
    for _ in range(60):
        if not st.prepare_next_batch():
            break
        live = {int(r): int(s) for r, s in zip(st.request_ids, st.state_slots) if r >= 0}
        assert len(set(live.values())) == len(live) and all(0 <= s < 2 for s in live.values())
        for r, s in live.items():
            assert held.setdefault(r, s) == s
    assert set(held) == set(range(5))


def test_scheduler_online_hold_close_and_page_limit():
    st = BatchState(np.ones((4, 40), np.int64), np.zeros(4), max_num_batched_requests=2, max_num_batched_tokens=16,
                    max_num_pages=3, page_size=4, online=True)
    assert not st.prepare_next_batch()
    st.prompt_lengths[1], st.request_ctl[1] = 6, REQ_HOLD
    assert st.prepare_next_batch() and st.num_active_tokens == 6
    assert not st.prepare_next_batch() and st.step[1] == 6 and st.request_ids[0] == 1     # held: pages stay
    st.prompt_lengths[1] = 30
    assert st.prepare_next_batch() and st.num_active_tokens == 6                          # three pages hold 12
    assert not st.prepare_next_batch()
    st.prompt_lengths[1], st.request_ctl[1] = 12, REQ_CLOSE
    st.prompt_lengths[3], st.request_ctl[3] = 5, REQ_RUN
    assert st.prepare_next_batch() and st.request_ids.tolist() == [3, -1]
    assert st.request_ctl.tolist() == [REQ_FREE, REQ_FREE, REQ_FREE, REQ_RUN] and st.num_active_tokens == 5
    assert st.prepare_next_batch() and st.num_active_tokens == 1                          # decodes on its own
