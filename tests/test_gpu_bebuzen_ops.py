"""The mechanisms Bebuzen adds to hybrid graphs, each alone on the GPU against oracle/hybrid_ops.py: sizes that divide nothing,
requests of unequal length in one batch, portions down to one token, state slots and pages that are not the identity, keys that
stand out at the edges of windows and of the kept first tokens."""
import pytest
import torch

from oracle import hybrid_ops as ops
from test_gpu_hybrid_ops import D, DTYPES, LENGTHS, RESTART, SCHEDULE, TOL, Bench, err, feed, sources
from test_gpu_lofirax_ops import RAND, mark_type, pad_k

pytestmark = pytest.mark.gpu
# the same requests in batches of at most eight tokens
SMALL = [[5, 0, 1], [2, 3, 1], [1, 1, 1], [6, 1, 1], [2, 4, 1], [1, 5, 2], [3, 0, 1], [1, 0, 1], [4, 2, 2], [8, 0, 0], [7, 1, 0]]
PLANS = {32: (SCHEDULE, RESTART, LENGTHS), 8: (SMALL, [(4, 1)], [sum(s[0] for s in SMALL), sum(s[1] for s in SMALL[4:]), sum(s[2] for s in SMALL)])}
BOTH_SIZES = pytest.mark.parametrize("tokens", [32, 8])
DT = pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])


def rows(width, seed, tokens):
    """One source per request, long enough for its life after the restart."""
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(max(n, 16), width, generator=g).float() for n in PLANS[tokens][2]]


# ---- selective scan
@DT
@BOTH_SIZES
@pytest.mark.parametrize("channels,n,rank", [(40, 16, 8), (33, 5, 3), (300, 24, 20), (8, 1, 1), (70, 128, 130), (1200, 16, 260), (90, 3, 128)])
def test_selective_scan(dtype, tokens, channels, n, rank):
    src = rows(2 * channels + rank + 2 * n, 41, tokens)
    g = torch.Generator().manual_seed(1)
    w = RAND(g, channels, rank, std=rank ** -0.5)
    bias, a_log, skip = RAND(g, channels, std=2.0, mean=-2.0), RAND(g, channels, n), RAND(g, channels)
    b = Bench(3, tokens=tokens)
    u, low, gate, out = b.zeros(b.B, channels), b.zeros(b.B, rank + 2 * n + 2), b.zeros(b.B, channels + 3), b.zeros(b.B, channels + 5, dtype=dtype)
    state = b.zeros(3, channels, (n + 3) // 4 * 4)
    b.pk.selective_scan_layer(b.pk.attach_input(u, name="u"), b.pk.attach_input(low, name="low"), b.pk.attach_input(gate, name="gate"),
                              b.inp(w, "w"), b.inp(bias, "bias"), b.inp(a_log, "a"), b.inp(skip, "d"), b.pk.attach_input(state, name="S"),
                              b.pk.attach_input(out, name="out"), rank=rank, n=n, gate_col=3)
    b.pk.compile()

    class Split:
        def __setitem__(self, r, v):
            v = v.cuda()
            u[r], gate[r, 3:], low[r, :rank + 2 * n] = v[:channels], v[channels:2 * channels], v[2 * channels:]
    schedule, restart, lengths = PLANS[tokens]
    got = feed(b, src, Split(), out[:, :channels], schedule, restart)
    for r in range(3):
        s = src[r][:lengths[r]].to(D)
        x, lo = s[:, :channels], s[:, 2 * channels:]
        dt = torch.nn.functional.softplus(lo[:, :rank] @ w.to(D).T + bias.to(D))
        ref = ops.selective_scan(x, dt, -torch.exp(a_log.to(D)), lo[:, rank:rank + n], lo[:, rank + n:], skip.to(D)) * ops.silu(s[:, channels:2 * channels])
        assert got[r].shape == ref.shape and err(got[r], ref) < TOL[dtype], (r, err(got[r], ref))
    assert float(out[:, channels:].abs().max()) == 0.0 and float(state[..., n:].abs().sum()) == 0.0


@DT
def test_scan_states_of_many_requests_stream_through_the_ring(dtype):
    """More requests in a batch than the ring of states holds, each with a state of its own from an earlier portion."""
    R, channels, n = 20, 24, 16
    g = torch.Generator().manual_seed(2)
    bias, a_log, skip, w = RAND(g, channels, std=1.0, mean=-1.0), RAND(g, channels, n), RAND(g, channels), RAND(g, channels, 4, std=0.5)
    counts = [[2, 1, 3] * 6 + [5, 1], [1] * R, [0, 1] * 10, [3, 0, 1, 1] * 5, [1] * R]
    src = [torch.randn(sum(c[r] for c in counts), 2 * channels + 4 + 2 * n, generator=g) for r in range(R)]
    b = Bench(R, tokens=64, pages=128)
    u, low, gate, out = b.zeros(64, channels), b.zeros(64, 4 + 2 * n), b.zeros(64, channels), b.zeros(64, channels, dtype=dtype)
    b.pk.selective_scan_layer(b.pk.attach_input(u, name="u"), b.pk.attach_input(low, name="low"), b.pk.attach_input(gate, name="gate"), b.inp(w, "w"),
                              b.inp(bias, "bias"), b.inp(a_log, "a"), b.inp(skip, "d"), b.pk.attach_input(b.zeros(R, channels, n), name="S"),
                              b.pk.attach_input(out, name="out"), rank=4, n=n, gate_col=0)
    b.pk.compile()

    class Split:
        def __setitem__(self, r, v):
            v = v.cuda()
            u[r], gate[r], low[r] = v[:channels], v[channels:2 * channels], v[2 * channels:]
    got = feed(b, src, Split(), out, counts)
    for r in range(R):
        s = src[r].to(D)
        dt = torch.nn.functional.softplus(s[:, 2 * channels:2 * channels + 4] @ w.to(D).T + bias.to(D))
        ref = ops.selective_scan(s[:, :channels], dt, -torch.exp(a_log.to(D)), s[:, -2 * n:-n], s[:, -n:], skip.to(D)) * ops.silu(s[:, channels:2 * channels])
        assert err(got[r], ref) < TOL[dtype], (r, err(got[r], ref))


def test_scan_memory_of_a_thousand_tokens():
    """Decays near one: what the first token wrote is read after a thousand steps.  (Steps that vary: a constant one would be rounded
    the same way every time.)"""
    channels, n, T = 8, 4, 1024
    b = Bench(1, tokens=64, page=64, pages=16, max_seq=1024)
    u, low, gate, out = b.zeros(64, channels), b.zeros(64, 1 + 2 * n), b.zeros(64, channels), b.zeros(64, channels)
    bias = torch.linspace(-9.0, -6.0, channels).to(torch.bfloat16)          # steps of 1e-4 .. 2e-3
    w, zero = torch.full((channels, 1), 0.25, dtype=torch.bfloat16), lambda *s: torch.zeros(*s, dtype=torch.bfloat16)
    z = torch.randn(T, generator=torch.Generator().manual_seed(1))
    b.pk.selective_scan_layer(b.pk.attach_input(u, name="u"), b.pk.attach_input(low, name="low"), b.pk.attach_input(gate, name="gate"),
                              b.inp(w, "w"), b.inp(bias, "bias"), b.inp(zero(channels, n), "a"), b.inp(zero(channels), "d"),
                              b.pk.attach_input(b.zeros(1, channels, n), name="S"), b.pk.attach_input(out, name="out"), rank=1, n=n, gate_col=0)
    mark_type(b, torch.float32)
    b.pk.compile()
    gate.fill_(2.0)
    low[:, 1 + n:] = 1.0
    for t in range(T // 64):
        u.zero_(), low[:, 1:1 + n].zero_()
        low[:, 0] = z[64 * t:64 * t + 64].cuda()
        if t == 0:
            u[0], low[0, 1:1 + n] = 1.0, 1.0
        b.describe([64])
        b.pk.step(1)
        b.pk.status()
    dt = torch.nn.functional.softplus(bias.to(D) + 0.25 * z.to(D)[:, None])
    ref = n * dt[0] * torch.exp(-dt[1:].sum(0)) * ops.silu(torch.tensor(2.0, dtype=D))
    assert float(((out[63].double().cpu() - ref) / ref).abs().max()) < 5e-6


@DT
@pytest.mark.parametrize("channels,taps", [(40, 4), (33, 1), (96, 2), (64, 7)])
def test_short_conv_with_silu_and_a_copy_for_the_next_linear(dtype, channels, taps):
    src = rows(channels, 42, 32)
    g = torch.Generator().manual_seed(3)
    w, cb = RAND(g, channels, taps), RAND(g, channels)
    b = Bench(3)
    x, out, copy = b.zeros(b.B, channels), b.zeros(b.B, channels), b.zeros(b.B, channels + 8, dtype=dtype)
    b.pk.short_conv_layer(b.pk.attach_input(x, name="x"), b.inp(w, "w"), b.pk.attach_input(b.zeros(3, max(taps - 1, 1), channels), name="st"),
                          b.pk.attach_input(out, name="o"), bias=b.inp(cb, "cb"), activation="silu", copy=b.pk.attach_input(copy, name="c"))
    mark_type(b, dtype)
    b.pk.compile()

    class Rows:                                                    # output and copy of a batch row side by side
        def __getitem__(self, r):
            return torch.cat([out[r], copy[r, :channels].float()])
    got = feed(b, src, x, Rows(), SCHEDULE, RESTART)
    for r in range(3):
        ref = ops.silu(ops.short_conv(src[r][:LENGTHS[r]].to(D), w.to(D), cb.to(D)))
        assert err(got[r][:, :channels], ref) < TOL[torch.float32] and err(got[r][:, channels:], ref) < TOL[dtype], r
    assert float(copy[:, channels:].abs().max()) == 0.0


# ---- attention: norms in front of the rotation, both pair layouts, windows, kept first tokens, sink
def attention_graph(b, dtype, H, G, dim, vdim, rot, interleaved, scale, window, keep, sink, qn, kn, maps=1, lam=0.0, factor=1.0, second=False):
    """proj [q | k | v] -> attention output (float32 with two maps, then combined).  `second`: the projections' q part once more, as a
    layer that reads the first one's keys and values; returns (proj, out)."""
    from mirage_b200.builders.hybrid import rotary_tables
    r8 = lambda n: (n + 7) // 8 * 8
    nq, nk = H * maps * dim, G * maps * dim
    proj = b.zeros(b.B, nq + nk + G * vdim)
    out = b.zeros(b.B, H * vdim + 2, dtype=dtype)
    cos, sin = rotary_tables(700.0, rot, b.pk.max_seq_length, "cuda")
    cos, sin = b.pk.attach_input(cos, name="cos"), b.pk.attach_input(sin, name="sin")
    kd = r8(maps * dim)
    # (rows nobody wrote hold a value that would show)
    kc = torch.full((b.pk.max_num_pages, b.page, G, kd), 0.0, dtype=dtype, device="cuda")
    vc = b.zeros(b.pk.max_num_pages, b.page, G, r8(vdim), dtype=dtype)
    kct, vct = b.pk.attach_input(kc, name="kc"), b.pk.attach_input(vc, name="vc")
    pt, q = b.pk.attach_input(proj, name="proj"), b.pk.attach_input(b.zeros(b.B, H * maps * kd, dtype=dtype) + 7.0, name="q")
    kw = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, q_col=0, rot_dims=rot, eps=1e-4, interleaved=interleaved, maps=maps)
    b.pk.qkv_append_layer(pt, q, kct, vct, cos, sin, k_col=nq, v_col=nq + nk, q_norm=b.inp(qn, "qn"), k_norm=b.inp(kn, "kn"), **kw)
    if second:
        q = b.pk.attach_input(b.zeros(b.B, H * maps * kd, dtype=dtype) + 7.0, name="q2")
        b.pk.qkv_append_layer(pt, q, None, None, cos, sin, q_norm=b.inp(qn, "qn2"), **kw)
    ot = b.pk.attach_input(out, name="o")
    akw = dict(heads=H * maps, kv_heads=G, vdim=vdim, scale=scale, sink=sink, window=window, keep_first=keep)
    if maps == 1:
        b.pk.ext_attention_layer(q, kct, vct, ot, out_col=2, **akw)
    else:
        m = b.pk.attach_input(b.zeros(b.B, 2 * H * vdim), name="maps")
        b.pk.ext_attention_layer(q, kct, vct, m, **akw)
        b.pk.diff_combine_layer(m, ot, heads=H, vdim=vdim, lam=lam, factor=factor, eps=1e-4)
    b.pk.compile()
    return proj, out[:, 2:] if maps == 1 else out[:, :H * vdim]


def attention_reference(s, H, G, dim, vdim, rot, interleaved, scale, window, keep, sink, qn, kn, maps=1, lam=0.0, factor=1.0, second=False):
    s = s.to(D)
    T, nq, nk = s.shape[0], H * maps * dim, G * maps * dim
    freqs = ops.rotary_frequencies(700.0, rot)
    turn = lambda x, w: ops.rotate_pairs(ops.rms_norm(x, w.to(D), 1e-4), torch.arange(T), freqs, interleaved)
    q, k = turn(s[:, :nq].view(T, -1, dim), qn), turn(s[:, nq:nq + nk].view(T, -1, dim), kn)
    v = s[:, nq + nk:].view(T, G, vdim)
    if maps == 1:
        return ops.window_attention(q, k, v, scale, window, keep, sink).flatten(1)
    a1, a2 = (ops.window_attention(q.view(T, H, 2, dim)[:, :, m], k.view(T, G, 2, dim)[:, :, m], v, scale, window, keep, sink) for m in range(2))
    return (factor * ops.rms_unit(a1 - lam * a2, 1e-4)).flatten(1)


def norms(dim, seed=5):
    g = torch.Generator().manual_seed(seed)
    return RAND(g, dim, std=0.3, mean=1.2), RAND(g, dim, std=0.3, mean=1.2)


ATTENTION = [  # H, G, dim, vdim, rot, interleaved, scale, window, keep, sink
    (4, 2, 16, 24, 8, True, 0.3, 9, 3, True), (3, 3, 20, 12, 20, False, 0.25, 13, 0, False), (6, 1, 72, 40, 36, True, 0.1, 1, 2, True),
    (5, 1, 128, 128, 64, False, 0.1, 16, 16, True), (2, 1, 168, 96, 40, True, 0.08, 20, 1, False), (16, 2, 64, 32, 64, True, 0.12, 0, 0, True),
    (4, 4, 30, 7, 2, False, 0.2, 8, 40, True)]


@DT
@BOTH_SIZES
@pytest.mark.parametrize("case", ATTENTION, ids=str)
def test_windowed_attention(dtype, tokens, case):
    H, G, dim, vdim = case[:4]
    src = [s.to(torch.bfloat16).float() for s in rows((H + G) * dim + G * vdim, 43, tokens)]
    args = case + norms(dim)
    b = Bench(3, tokens=tokens)
    proj, out = attention_graph(b, dtype, *args)
    schedule, restart, lengths = PLANS[tokens]
    got = feed(b, src, proj, out, schedule, restart)
    for r in range(3):
        assert err(got[r], attention_reference(src[r][:lengths[r]], *args)) < (TOL[dtype] if dtype == torch.float32 else 1.5e-2), r


DIFF = [(4, 2, 16, 24, 8, False, 0.3, 9, 0, False), (3, 3, 20, 12, 20, False, 0.25, 13, 0, False), (2, 1, 64, 128, 32, True, 0.1, 17, 0, False),
        (4, 1, 56, 88, 56, False, 0.15, 7, 2, True), (5, 1, 100, 260, 10, False, 0.1, 0, 0, False), (1, 1, 9, 5, 2, False, 0.3, 6, 0, False)]


@DT
@BOTH_SIZES
@pytest.mark.parametrize("second", [False, True], ids=["own", "shared"])
@pytest.mark.parametrize("case", DIFF, ids=str)
def test_differential_attention(dtype, tokens, second, case):
    H, G, dim, vdim = case[:4]
    if dtype == torch.bfloat16 and vdim > 256:
        vdim = 200
    case = (H, G, dim, vdim) + case[4:]
    src = [s.to(torch.bfloat16).float() for s in rows(2 * (H + G) * dim + G * vdim, 44, tokens)]
    args = case + norms(dim) + (2, 0.45, 0.7, second)
    b = Bench(3, tokens=tokens)
    proj, out = attention_graph(b, dtype, *args)
    schedule, restart, lengths = PLANS[tokens]
    got = feed(b, src, proj, out, schedule, restart)
    for r in range(3):
        ref = attention_reference(src[r][:lengths[r]], *args)
        assert err(got[r], ref) < (1e-5 if dtype == torch.float32 else 4e-2), (r, err(got[r], ref))


@DT
@pytest.mark.parametrize("page", [8, 6])
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("window,keep", [(45, 5), (64, 0), (139, 9), (256, 64)])
def test_keys_at_the_edges_of_the_window_and_of_the_kept_tokens(dtype, window, keep, maps, page):
    """Keys that stand out just inside and just outside the window and at the last kept and the next position, asked for from a prompt's
    portion and by decoded tokens, at contexts far beyond the window and before it is full."""
    H, G, dim, vdim, T = 2, 1, 16, 8, 420
    g = torch.Generator().manual_seed(window)
    s = torch.randn(T, maps * (H + G) * dim + G * vdim, generator=g)
    nq, nk = maps * H * dim, maps * dim
    d = torch.zeros(dim)
    d[12] = 6.0                                                    # outside the rotated part: no decay with distance
    s[:, :nq] *= 0.1                                               # (norms: only the direction counts, scores of the rest stay small)
    asked, marked = [window - 1, window, window + 1, 300, 301, T - 70, T - 4, T - 3, T - 2, T - 1], []
    for t in asked:
        s[t, :nq] = d.repeat(maps * H)
        marked += [t - window + 1, t - window]
    marked += [keep - 1, keep]
    noise = torch.randn(T, nk, generator=g).view(T, maps, dim)
    noise[..., 12] = 0.0
    s[:, nq:nq + nk] = noise.flatten(1)
    for j in marked:
        if 0 <= j < T:
            s[j, nq:nq + nk] = d.repeat(maps)
            s[j, nq + nk:] *= 5.0
    one = torch.ones(dim, dtype=torch.bfloat16)
    args = (H, G, dim, vdim, 8, True, 0.6, window, keep, True, one, one) + ((2, 0.5, 0.6) if maps == 2 else ())
    s = s.to(torch.bfloat16).float()
    ref = attention_reference(s, *args)
    for tokens, cuts in ((32, [32] * 9 + [14, 3, 32, 32, 32, 1, 1, 8, 2, 1, 1, 1, 1, 1, 1, 1]), (4, [4] * 105)):
        b = Bench(2, tokens=tokens, page=page, pages=512 // page, max_seq=512)
        proj, out = attention_graph(b, dtype, *args)
        got = run_alone(b, s, proj, out, cuts)
        for t in range(T):
            e = float((got[t] - ref[t]).abs().max() / ref[t].abs().max())
            assert e < ((1e-4 if maps == 2 else 1e-5) if dtype == torch.float32 else 6e-2), (tokens, t, e)


def run_alone(b, s, proj, out, cuts):
    """The second request in portions of the given sizes, to the end of its rows."""
    got, at = [], 0
    for n in cuts:
        n = min(n, s.shape[0] - at)
        if n == 0:
            break
        for _, pos, row in b.describe([0, n]):
            proj[row] = s[pos].cuda()
        b.pk.step(1)
        b.pk.status()
        got.append(out[:n].clone())
        at += n
    return torch.cat(got).double().cpu()


# ---- norms of sublayer outputs, routing, experts, biases
@DT
@pytest.mark.parametrize("tokens", [1, 2, 7, 40])
@pytest.mark.parametrize("width,terms,closing", [(64, "y", False), (50, "y experts", False), (4100, "y", True), (128, "experts", True), (96, "experts", False),
                                                 (37, "y experts", True), (64, "", False)])
def test_norm_of_the_sublayer_output(dtype, tokens, width, terms, closing):
    """x += factor * norm(y + experts) * w, and the stream as it is (or its norm) for the next sublayer."""
    g = torch.Generator().manual_seed(6)
    x, y = torch.randn(tokens, width, generator=g), 3 * torch.randn(tokens, width, generator=g)
    ex, ew = torch.randn(tokens, 5, width, generator=g), torch.rand(tokens, 5, generator=g)
    w, wn = RAND(g, width, std=0.3, mean=1.0), RAND(g, width, std=0.3, mean=1.0)
    b = Bench(1, tokens=tokens)
    kw = {}
    if "y" in terms:
        kw["y"] = b.inp(y, "y")
    if "experts" in terms:
        kw["experts"] = (b.inp(ex, "ex"), b.inp(ew, "ew"))
    xo, out = b.zeros(tokens, width), b.zeros(tokens, width + 5, dtype=dtype)
    b.pk.residual_norm_layer(b.inp(x, "x"), post_weight=b.inp(w, "w") if terms else None, norm_weight=b.inp(wn, "wn") if closing else None,
                             output=b.pk.attach_input(out, name="o"), eps=1e-3, x_out=b.pk.attach_input(xo, name="xo") if terms else None,
                             post_factor=0.7, **kw)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    sub = (y.double() if "y" in terms else 0) + ((ex.double() * ew.double()[..., None]).sum(1) if "experts" in terms else 0)
    new = x.double() + (0.7 * ops.rms_norm(sub, w.double(), 1e-3) if terms else 0)
    if terms:
        assert err(xo.double().cpu(), new) < TOL[torch.float32]
    ref = ops.rms_norm(new, wn.double(), 1e-3) if closing else new
    assert err(out[:, :width].double().cpu(), ref) < TOL[dtype] and float(out[:, width:].abs().max()) == 0.0


@pytest.mark.parametrize("tokens", [1, 2])
@pytest.mark.parametrize("use,closing", [("y", False), ("y", True), ("", False)])
def test_norm_of_the_sublayer_output_folds_into_a_linear(tokens, use, closing):
    g = torch.Generator().manual_seed(7)
    width, N = 100, 70
    x, y = torch.randn(tokens, width, generator=g), 3 * torch.randn(tokens, width, generator=g)
    w, wn, lin, bias = RAND(g, width, std=0.3, mean=1.0), RAND(g, width, std=0.3, mean=1.0), RAND(g, N, width, std=0.1), RAND(g, N)
    b = Bench(1, tokens=tokens)
    xo, out = b.zeros(tokens, width), b.zeros(tokens, N)
    h = b.pk.new_tensor(dims=(tokens, 128), name="h")
    kw = dict(y=b.inp(y, "y"), post_weight=b.inp(w, "w"), x_out=b.pk.attach_input(xo, name="xo"), post_factor=0.6) if use else {}
    b.pk.residual_norm_layer(b.inp(x, "x"), norm_weight=b.inp(wn, "wn") if closing else None, output=h, eps=1e-4, **kw)
    b.pk.linear_layer(input=h, weight=b.inp(pad_k(lin, torch.bfloat16), "lin"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1),
                      block_dim=(128, 1, 1), bias=b.inp(bias, "bias"))
    b.pk.compile()
    assert b.pk.graph_info()["num_folded"] == 1
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    new = x.double() + (0.6 * ops.rms_norm(y.double(), w.double(), 1e-4) if use else 0)
    if use:
        assert err(xo.double().cpu(), new) < TOL[torch.float32]
    ref = (ops.rms_norm(new, wn.double(), 1e-4) if closing else new) @ lin.double().T + bias.double()
    assert err(out.double().cpu(), ref) < TOL[torch.bfloat16]


@DT
@pytest.mark.parametrize("tokens", [1, 8, 30, 64])
def test_linear_bias(dtype, tokens):
    g = torch.Generator().manual_seed(8)
    K, N = 192, 333
    b = Bench(1, tokens=tokens)
    x, w, bias = torch.randn(tokens, K, generator=g).to(dtype), RAND(g, N, K, std=0.1), RAND(g, N, std=2.0)
    out = b.zeros(tokens, N + 3)
    b.pk.linear_layer(input=b.inp(x, "x"), weight=b.inp(w, "w"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1), block_dim=(128, 1, 1),
                      bias=b.inp(bias, "bias"))
    mark_type(b, dtype)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    assert err(out[:, :N].double().cpu(), x.double() @ w.double().T + bias.double()) < 3e-6 and float(out[:, N:].abs().max()) == 0.0


@DT
@pytest.mark.parametrize("tokens", [1, 8, 64])
@pytest.mark.parametrize("E,top,ff,width,scale", [(6, 2, 40, 64, 1.5), (12, 4, 64, 96, 0.3), (5, 5, 24, 64, 1.0), (70, 6, 32, 64, 2.0), (1, 1, 130, 128, 1.0)])
def test_softmax_routed_squared_relu_experts(dtype, tokens, E, top, ff, width, scale):
    """Weights are the probabilities times a scale, not renormalised; their sum over the experts is normed with the shared output."""
    g = torch.Generator().manual_seed(9)
    b = Bench(1, tokens=tokens)
    F = (ff + 63) // 64 * 64 if dtype == torch.bfloat16 else ff
    h, logits = torch.randn(tokens, width, generator=g).to(torch.bfloat16), 2.0 * torch.randn(tokens, E, generator=g)
    up, down = RAND(g, E, ff, width, std=0.2), RAND(g, E, width, ff, std=0.2)
    mi = b.mi
    new = lambda name, dims, dt: b.pk.new_tensor(dims=dims, dtype=dt, name=name)
    wts, idx, act = new("wts", (tokens, top), mi.float32), new("idx", (E, tokens), mi.int32), new("act", (E + 1,), mi.int32)
    grid = dict(grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
    b.pk.moe_topk_softmax_routing_layer(b.inp(logits, "logits"), (wts, idx, act), **grid, renormalize=False, scale=scale)
    mid = new("mid", (tokens, top, F), mi.bfloat16 if dtype == torch.bfloat16 else mi.float32)
    out = new("out", (tokens, top, width), mi.float32)
    b.pk.moe_w13_linear_layer(b.inp(pad_k(h, dtype).to(dtype), "h"), b.inp(pad_k(up, dtype), "up"), idx, act, mid, **grid, activation="relu2")
    b.pk.moe_w2_linear_layer(mid, b.inp(pad_k(down, dtype), "down"), idx, act, out, **grid)
    x, y, xo = torch.randn(tokens, width, generator=g), torch.randn(tokens, width, generator=g), b.zeros(tokens, width)
    w = RAND(g, width, std=0.3, mean=1.0)
    b.pk.residual_norm_layer(b.inp(x, "x"), b.inp(y, "y"), b.inp(w, "w"), output=b.pk.attach_input(b.zeros(tokens, width, dtype=dtype), name="o"),
                             experts=(out, wts), x_out=b.pk.attach_input(xo, name="xo"), eps=1e-4)
    b.pk.compile()
    b.describe([tokens])
    for _ in range(2):
        b.pk.step(1)
        b.pk.status()
    sub = y.double()
    for t in range(tokens):
        for e, p in zip(*ops.softmax_choice(logits[t].double(), top)):
            sub[t] += p * scale * (ops.squared_relu(h[t].double() @ up[e].double().T) @ down[e].double().T)
    assert err(xo.double().cpu(), x.double() + ops.rms_norm(sub, w.double(), 1e-4)) < TOL[dtype]
