"""Every mechanism of hybrid graphs alone, as a one-mechanism graph on the GPU against oracle/hybrid_ops.py: sizes that
divide nothing, several requests of unequal length in one batch, portions down to one token, state slots and pages that are
not the identity."""
import pytest
import torch

from oracle import hybrid_ops as ops

pytestmark = pytest.mark.gpu
D = torch.float64
TOL = {torch.float32: 3e-6, torch.bfloat16: 8e-3}
DTYPES = [torch.float32, torch.bfloat16]


class Bench:
    """A batch description of its own (online_notoken): `run` feeds each request its next tokens."""

    def __init__(self, requests, tokens=32, page=8, pages=64, max_seq=256):
        self.R, self.B, self.page = requests, tokens, page
        i32 = dict(dtype=torch.int32, device="cuda")
        self.meta = {"input_tokens": torch.zeros(tokens, 1, dtype=torch.int64, device="cuda"),
                     "qo_indptr_buffer": torch.zeros(requests + 1, **i32),
                     "paged_kv_indptr_buffer": torch.zeros(requests + 1, **i32),
                     "paged_kv_indices_buffer": torch.zeros(pages, **i32),
                     "paged_kv_last_page_len_buffer": torch.zeros(requests, **i32),
                     "state_slots": torch.arange(requests - 1, -1, -1, **i32)}
        self.free = torch.randperm(pages, generator=torch.Generator().manual_seed(5)).tolist()
        self.pages = [[] for _ in range(requests)]
        self.len = [0] * requests
        import mirage_b200 as mi
        self.mi = mi
        self.pk = mi.PersistentKernel(mode="online_notoken", max_seq_length=max_seq, max_num_batched_requests=requests,
                                      max_num_batched_tokens=tokens, max_num_pages=pages, page_size=page, meta_tensors=self.meta)

    def inp(self, t, name):
        return self.pk.attach_input(t.cuda().contiguous(), name=name)

    def zeros(self, *shape, dtype=torch.float32):
        return torch.zeros(*shape, dtype=dtype, device="cuda")

    def restart(self, r):
        self.free += self.pages[r]
        self.pages[r], self.len[r] = [], 0

    def describe(self, counts):
        """Batch of counts[r] tokens per request; returns [(request, first position, batch row)] of the tokens."""
        qo, kv, idx, last, where = [0], [0], [], [], []
        for r, n in enumerate(counts):
            where += [(r, self.len[r] + j, qo[-1] + j) for j in range(n)]
            self.len[r] += n
            while len(self.pages[r]) * self.page < self.len[r]:
                self.pages[r].append(self.free.pop(0))
            qo.append(qo[-1] + n)
            idx += self.pages[r]
            kv.append(len(idx))
            last.append((self.len[r] - 1) % self.page + 1 if self.len[r] else 0)
        put = lambda k, v: self.meta[k][:len(v)].copy_(torch.tensor(v, dtype=torch.int32))
        put("qo_indptr_buffer", qo), put("paged_kv_indptr_buffer", kv), put("paged_kv_last_page_len_buffer", last)
        if idx:
            put("paged_kv_indices_buffer", idx)
        return where


def feed(b, src, dst, out, schedule, restarts=()):
    """Runs the schedule (lists of token counts per request): row src[request][position] goes to dst[batch row].  Returns
    per request the collected output rows."""
    got = [[] for _ in src]
    for n, counts in enumerate(schedule):
        for step, r in restarts:
            if step == n:
                b.restart(r)
                got[r].clear()
        where = b.describe(counts)
        for r, pos, row in where:
            dst[row] = src[r][pos]
        b.pk.step(1)
        b.pk.status()
        for r, pos, row in where:
            got[r].append(out[row].clone())
    return [torch.stack(g).double().cpu() for g in got]


def err(got, ref):
    return float((got - ref).abs().max() / ref.abs().max())


# three requests: one long in uneven portions, one that starts late, one token by token; the late one restarts in a used slot
SCHEDULE = [[7, 0, 1], [2, 5, 1], [1, 1, 1], [11, 2, 1], [3, 9, 1], [2, 1, 2], [1, 0, 1], [20, 6, 3]]
RESTART = [(4, 1)]
LENGTHS = [sum(s[0] for s in SCHEDULE), sum(s[1] for s in SCHEDULE[4:]), sum(s[2] for s in SCHEDULE)]


def sources(width, seed):
    g = torch.Generator().manual_seed(seed)
    # the second request's first life (before its restart) reads other rows than its second
    n = [LENGTHS[0], max(LENGTHS[1], 16), LENGTHS[2]]
    return [torch.randn(k, width, generator=g).float() for k in n]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 24), (1, 20, 7), (3, 130, 66), (1, 300, 40), (2, 64, 200), (1, 600, 530), (2, 256, 96)])
def test_mlstm(dtype, heads, dim, vdim):
    qk, v = heads * dim, heads * vdim
    src = sources(2 * qk + 2 * v + 2 * heads, 11)
    for s in src:
        s[:, -heads:] += 3.0                                      # forget gates near one
    g = torch.Generator().manual_seed(1)
    ib, fb, norm = (torch.randn(n, generator=g).to(torch.bfloat16) for n in (heads, heads, v))
    b = Bench(3)
    proj, out = b.zeros(b.B, src[0].shape[1]), b.zeros(b.B, v, dtype=dtype)
    chunks = b.pk.mlstm_chunks(b.pk.num_workers, 3, heads, dim, vdim)
    b.pk.mlstm_layer(b.pk.attach_input(proj, name="proj"), b.inp(ib, "ib"), b.inp(fb, "fb"),
                     b.inp(norm, "norm"), b.pk.attach_input(b.zeros(3, heads, dim, (vdim + 3) // 4 * 4), name="S"),
                     b.pk.attach_input(b.zeros(3, heads, chunks, dim + 1), name="nm"),
                     b.pk.attach_input(b.zeros(b.B, v), name="raw"), b.pk.attach_input(out, name="out"), heads=heads, dim=dim,
                     vdim=vdim, q_col=0, k_col=qk, v_col=2 * qk, gate_col=2 * qk + v, i_col=2 * qk + 2 * v,
                     f_col=2 * qk + 2 * v + heads, gate_cap=7.0, eps=1e-4, q_scale=dim ** -0.5)
    b.pk.compile()
    got = feed(b, src, proj, out, SCHEDULE, RESTART)
    for r in range(3):
        s = src[r][:LENGTHS[r]].to(D)
        cut = lambda a, n, w: s[:, a:a + n * w].view(-1, n, w)
        o = ops.mlstm(cut(0, heads, dim) * dim ** -0.5, cut(qk, heads, dim), cut(2 * qk, heads, vdim),
                      s[:, 2 * qk + 2 * v:][:, :heads] + ib.to(D), s[:, 2 * qk + 2 * v + heads:] + fb.to(D), 7.0)
        ref = ops.mlstm_output(o, norm.to(D), s[:, 2 * qk + v:2 * qk + 2 * v], 1e-4)
        assert got[r].shape == ref.shape and err(got[r], ref) < TOL[dtype], (r, err(got[r], ref))


@pytest.mark.parametrize("channels,taps", [(40, 4), (33, 1), (96, 2), (64, 7)])
def test_short_conv(channels, taps):
    src = sources(channels + 5, 12)
    g = torch.Generator().manual_seed(2)
    w, ib, cb = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((channels, taps), (channels,), (channels,)))
    b = Bench(3)
    x, out = b.zeros(b.B, channels + 5), b.zeros(b.B, channels)
    b.pk.short_conv_layer(b.pk.attach_input(x, name="x"), b.inp(w, "w"),
                          b.pk.attach_input(b.zeros(3, max(taps - 1, 1), channels), name="st"), b.pk.attach_input(out, name="o"),
                          input_bias=b.inp(ib, "ib"), bias=b.inp(cb, "cb"), in_col=5)
    b.pk.compile()
    got = feed(b, src, x, out, SCHEDULE, RESTART)
    for r in range(3):
        ref = ops.short_conv(src[r][:LENGTHS[r], 5:].to(D) + ib.to(D), w.to(D), cb.to(D))
        assert err(got[r], ref) < TOL[torch.float32], r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("blocks,size", [(3, 16), (1, 70), (2, 15), (1, 1), (2, 160)])
def test_rglru(dtype, blocks, size):
    width = blocks * size
    src = sources(2 * width, 13)
    g = torch.Generator().manual_seed(3)
    bf = lambda *s, std=1.0, mean=0.0: (mean + std * torch.randn(*s, generator=g)).to(torch.bfloat16)
    ra, ri = bf(blocks, size, size, std=size ** -0.5), bf(blocks, size, size, std=size ** -0.5)
    rab, rib, yb, lam = bf(blocks, size), bf(blocks, size), bf(width), bf(width, mean=-4.0)
    b = Bench(3)
    both, u, out = b.zeros(b.B, 2 * width), b.zeros(b.B, width), b.zeros(b.B, width + 3, dtype=dtype)

    class Split:                                                   # one source row fills u and the y projections
        def __setitem__(self, row, v):
            u[row], both[row] = v[:width].cuda(), v.cuda()
    b.pk.rglru_layer(b.pk.attach_input(u, name="u"), b.pk.attach_input(both, name="proj"), b.inp(yb, "yb"), b.inp(ra, "ra"),
                     b.inp(rab, "rab"), b.inp(ri, "ri"), b.inp(rib, "rib"), b.inp(lam, "lam"),
                     b.pk.attach_input(b.zeros(3, width), name="st"), b.pk.attach_input(out, name="o"), y_col=width, out_col=3,
                     out_scale=0.6, decay=5.0)
    b.pk.compile()
    got = feed(b, src, Split(), out[:, 3:], SCHEDULE, RESTART)
    for r in range(3):
        s = src[r][:LENGTHS[r]].to(D)
        S = ops.rglru(s[:, :width], ra.to(D), rab.to(D), ri.to(D), rib.to(D), lam.to(D), 5.0)
        assert err(got[r], 0.6 * S * ops.gelu_tanh(s[:, width:] + yb.to(D))) < TOL[dtype], r
    assert float(out[:, :3].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_rglru_of_a_full_batch_in_several_token_groups(dtype):
    """64 tokens of four requests against gates so wide that the task takes them in groups that cut through requests."""
    size = width = 300
    counts = [[29, 1, 20, 14], [3, 40, 1, 20]]
    g = torch.Generator().manual_seed(8)
    bf = lambda *s, std=1.0, mean=0.0: (mean + std * torch.randn(*s, generator=g)).to(torch.bfloat16)
    ra, ri = bf(1, size, size, std=size ** -0.5), bf(1, size, size, std=size ** -0.5)
    rab, rib, yb, lam = bf(1, size), bf(1, size), bf(width), bf(width, mean=-4.0)
    src = [torch.randn(sum(c[r] for c in counts), 2 * width, generator=g).float() for r in range(4)]
    b = Bench(4, tokens=64)
    both, u, out = b.zeros(64, 2 * width), b.zeros(64, width), b.zeros(64, width, dtype=dtype)

    class Split:
        def __setitem__(self, row, v):
            u[row], both[row] = v[:width].cuda(), v.cuda()
    b.pk.rglru_layer(b.pk.attach_input(u, name="u"), b.pk.attach_input(both, name="proj"), b.inp(yb, "yb"), b.inp(ra, "ra"),
                     b.inp(rab, "rab"), b.inp(ri, "ri"), b.inp(rib, "rib"), b.inp(lam, "lam"),
                     b.pk.attach_input(b.zeros(4, width), name="st"), b.pk.attach_input(out, name="o"), y_col=width)
    b.pk.compile()
    got = feed(b, src, Split(), out, counts)
    for r in range(4):
        s = src[r].to(D)
        S = ops.rglru(s[:, :width], ra.to(D), rab.to(D), ri.to(D), rib.to(D), lam.to(D))
        assert err(got[r], S * ops.gelu_tanh(s[:, width:] + yb.to(D))) < TOL[dtype], r


def attention_graph(b, dtype, H, G, dim, rot, base, scale, cap, sink, unit, eps, separate_v=False):
    vdim = dim
    width = (H + G) * dim + (G * vdim if separate_v else 0)
    proj, out = b.zeros(b.B, width), b.zeros(b.B, H * vdim + 2, dtype=dtype)
    dp = (dim + 7) // 8 * 8
    from mirage_b200.builders.hybrid import rotary_tables
    cos, sin = rotary_tables(base, rot, b.pk.max_seq_length, "cuda")
    kc, vc = b.zeros(b.pk.max_num_pages, b.page, G, dp, dtype=dtype), b.zeros(b.pk.max_num_pages, b.page, G, dp, dtype=dtype)
    kct, vct = b.pk.attach_input(kc, name="kc"), b.pk.attach_input(vc, name="vc")
    q = b.pk.attach_input(b.zeros(b.B, H * dp, dtype=dtype), name="q")
    b.pk.qkv_append_layer(b.pk.attach_input(proj, name="proj"), q, kct, vct, b.pk.attach_input(cos, name="cos"),
                          b.pk.attach_input(sin, name="sin"), heads=H, kv_heads=G, dim=dim, vdim=vdim, q_col=0, k_col=H * dim,
                          v_col=(H + G) * dim if separate_v else H * dim, rot_dims=rot, unit_norm=unit, eps=eps)
    b.pk.ext_attention_layer(q, kct, vct, b.pk.attach_input(out, name="o"), heads=H, kv_heads=G, vdim=vdim, scale=scale, softcap=cap,
                             sink=sink, out_col=2, out_scale=0.8)
    b.pk.compile()
    return proj, out


def attention_reference(s, H, G, dim, rot, base, scale, cap, sink, unit, eps, separate_v=False):
    s = s.to(D)
    T = s.shape[0]
    q, k = s[:, :H * dim].view(T, H, dim), s[:, H * dim:(H + G) * dim].view(T, G, dim)
    v = s[:, (H + G) * dim:].view(T, G, dim) if separate_v else k
    turn = lambda x: ops.rotate_half_split(x, torch.arange(T), base, rot)
    n = (lambda x: ops.rms_unit(turn(x), eps)) if unit else turn
    return 0.8 * ops.attention(n(q), n(k), v, scale, cap, sink).reshape(T, -1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,rot,cap,sink,unit,sv", [
    (4, 2, 16, 8, 20.0, True, True, False), (3, 3, 20, 20, 0.0, False, True, True), (6, 1, 72, 0, 5.0, True, False, False),
    (5, 1, 128, 64, 30.0, True, True, False), (2, 1, 168, 40, 50.0, True, True, False), (16, 2, 64, 64, 50.0, False, True, True)])
def test_attention(dtype, H, G, dim, rot, cap, sink, unit, sv):
    args = (H, G, dim, rot, 900.0, 0.25 if unit else 0.02, cap, sink, unit, 1e-5, sv)
    src = sources((H + G) * dim + (G * dim if sv else 0), 14)
    b = Bench(3)
    proj, out = attention_graph(b, dtype, *args)
    got = feed(b, src, proj, out[:, 2:], SCHEDULE, RESTART)
    for r in range(3):
        # bf16: q, k, v and the result are each rounded once
        assert err(got[r], attention_reference(src[r][:LENGTHS[r]], *args)) < (TOL[dtype] if dtype == torch.float32 else 1.5e-2), r
    assert float(out[:, :2].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim", [(8, 2, 128), (16, 1, 128), (4, 4, 96)])
def test_attention_in_graphs_of_few_tokens(dtype, H, G, dim):
    """At most eight batched tokens: the streams of one 16-row tile, with the upper rows in use (16 heads) and not."""
    args = (H, G, dim, dim // 2, 900.0, 0.25, 30.0, True, True, 1e-5)
    g = torch.Generator().manual_seed(15)
    src = [torch.randn(n, (H + G) * dim, generator=g).float() for n in (150, 9)]
    b = Bench(2, tokens=8, page=16, pages=32)
    proj, out = attention_graph(b, dtype, *args)
    got = feed(b, src, proj, out[:, 2:], [[8, 0]] * 17 + [[3, 2], [1, 1], [2, 1], [1, 1], [5, 3], [2, 1]])
    for r in range(2):
        assert err(got[r], attention_reference(src[r], *args)) < (TOL[dtype] if dtype == torch.float32 else 1.5e-2), r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 7, 8, 63, 64, 127, 128, 383, 384, 700, 895])
def test_attention_far_key_at_page_and_chunk_borders(dtype, key):
    """One key that stands out (same direction as the last queries, its value scaled up) at places around page, tile and
    chunk borders of a sequence split into several chunks; asked for by a prompt portion and by a decoded token."""
    H, G, dim = 2, 1, 32
    args = (H, G, dim, 16, 500.0, 1.0, 30.0, True, True, 1e-6)
    T = 900
    g = torch.Generator().manual_seed(key)
    s = torch.randn(T, (H + G) * dim, generator=g).float()
    s[:, H * dim:] *= 0.3
    d = torch.zeros(dim)
    d[20] = 8.0                                                     # outside the rotated part: no decay with distance
    s[key, H * dim:] = d
    for t in (T - 3, T - 1):
        s[t, :H * dim] = d.repeat(H) * 0.5
    b = Bench(2, page=8, pages=256, max_seq=1024)
    proj, out = attention_graph(b, dtype, *args)
    sched = [[0, 32]] * 28 + [[0, 3], [0, 1]]
    rows = []
    for counts in sched:
        where = b.describe(counts)
        for _, pos, row in where:
            proj[row] = s[pos].cuda()
        b.pk.step(1)
        b.pk.status()
        rows += [out[row, 2:].clone() for _, _, row in where]
    got = torch.stack(rows).double().cpu()
    ref = attention_reference(s, *args)
    # the value itself is what the asking tokens must return, in magnitude far above the rest
    for t in (T - 3, T - 1):
        assert ref[t].abs().max() > 2.0
        assert float((got[t] - ref[t]).abs().max() / ref[t].abs().max()) < (2e-6 if dtype == torch.float32 else 1.5e-2), t
    assert err(got, ref) < (3e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,post", [(64, True), (37, True), (1030, True), (96, False), (640, None)])
def test_residual_norm(dtype, width, post):
    g = torch.Generator().manual_seed(6)
    b = Bench(2)
    x0, y0 = torch.randn(b.B, width, generator=g), 3 * torch.randn(b.B, width, generator=g)
    wp, wn = (0.3 * torch.randn(width, generator=g)).to(torch.bfloat16), (0.3 * torch.randn(width, generator=g)).to(torch.bfloat16)
    x, out = x0.cuda(), b.zeros(b.B, width, dtype=dtype)
    b.pk.residual_norm_layer(b.pk.attach_input(x, name="x"), None if post is None else b.inp(y0, "y"), b.inp(wp, "wp") if post else None,
                             b.inp(wn, "wn"), b.pk.attach_input(out, name="o"), eps=1e-3, zero_centered=bool(post))
    b.pk.compile()
    b.describe([20, 12])
    b.pk.step(1)
    b.pk.status()
    rx, ro = ops.residual_norm(x0.to(D), None if post is None else y0.to(D), wp.to(D) if post else None, wn.to(D), 1e-3, bool(post))
    assert err(x.double().cpu(), rx) < 1e-6
    assert err(out.double().cpu(), ro) < TOL[dtype]


@pytest.mark.parametrize("tokens", [1, 5, 8, 30, 64])
@pytest.mark.parametrize("dtype", DTYPES)
def test_linear_float32_output_and_squared_relu(dtype, tokens):
    """Linears of a hybrid graph: K a multiple of 64 only in bf16 graphs, few and many rows, both epilogues."""
    K, N1, N2 = (320, 200, 77) if dtype == torch.bfloat16 else (173, 200, 77)
    g = torch.Generator().manual_seed(7)
    b = Bench(1, tokens=tokens)
    x0 = torch.randn(tokens, K, generator=g)
    w1, w2 = ((K ** -0.5) * torch.randn(n, K, generator=g) for n in (N1, N2))
    w1, w2 = w1.to(torch.bfloat16), w2.to(torch.bfloat16)
    x = x0.cuda()
    h, y1, y2 = b.zeros(tokens, K, dtype=dtype), b.zeros(tokens, N1, dtype=dtype), b.zeros(tokens, N2)
    ht = b.pk.attach_input(h, name="h")
    b.pk.residual_norm_layer(b.pk.attach_input(x, name="x"), norm_weight=b.inp(torch.ones(K, dtype=torch.bfloat16), "ones"), output=ht)
    b.pk.linear_layer(input=ht, weight=b.inp(w1, "w1"), output=b.pk.attach_input(y1, name="y1"), grid_dim=(1, 1, 1),
                      block_dim=(128, 1, 1), activation="relu2")
    b.pk.linear_layer(input=ht, weight=b.inp(w2, "w2"), output=b.pk.attach_input(y2, name="y2"), grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    hd = h.double().cpu()
    assert err(hd, ops.rms_unit(x0.to(D), 1e-6)) < TOL[dtype]
    assert err(y2.double().cpu(), hd @ w2.to(D).T) < 3e-6             # float32 accumulation and output in both
    assert err(y1.double().cpu(), ops.squared_relu(hd @ w1.to(D).T)) < TOL[dtype]
