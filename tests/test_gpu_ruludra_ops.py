"""The mechanisms Ruludra adds to hybrid graphs, each alone on the GPU against oracle/hybrid_ops.py: sizes that divide nothing, requests
of unequal length in one batch, portions down to one token, state slots and pages that are not the identity, keys that stand out at
the edges of windows."""
import random

import pytest
import torch

from oracle import hybrid_ops as ops
from test_gpu_bebuzen_ops import BOTH_SIZES, DT, PLANS, rows, run_alone
from test_gpu_hybrid_ops import D, TOL, Bench, err, feed
from test_gpu_lofirax_ops import RAND, mark_type, pad_k

pytestmark = pytest.mark.gpu
R8 = lambda n: (n + 7) // 8 * 8


# ---- attention with norms over all heads, query temperature, distance bias
def attention_graph(b, dtype, H, G, dim, scale, window, temperature, qn, kn, r1, r2):
    """[q | k] -> attention whose values are the keys as projected."""
    nq, nk = H * dim, G * dim
    proj, out = b.zeros(b.B, nq + nk), b.zeros(b.B, nq + 2, dtype=dtype)
    kc, vc = (b.pk.attach_input(b.zeros(b.pk.max_num_pages, b.page, G, R8(dim), dtype=dtype), name=n) for n in ("kc", "vc"))
    q = b.pk.attach_input(b.zeros(b.B, H * R8(dim), dtype=dtype) + 7.0, name="q")
    b.pk.qkv_append_layer(b.pk.attach_input(proj, name="proj"), q, kc, vc, None, None, heads=H, kv_heads=G, dim=dim, vdim=dim, q_col=0, k_col=nq,
                          v_col=nq, rot_dims=0, eps=1e-4, q_norm=b.inp(qn, "qn"), k_norm=b.inp(kn, "kn"), whole_norm=True, temperature=temperature)
    b.pk.ext_attention_layer(q, kc, vc, b.pk.attach_input(out, name="o"), heads=H, kv_heads=G, vdim=dim, scale=scale, window=window, out_col=2,
                             distance_bias=(b.inp(r1, "r1"), b.inp(r2, "r2")))
    b.pk.compile()
    return proj, out[:, 2:]


def attention_reference(s, H, G, dim, scale, window, temperature, qn, kn, r1, r2):
    s, T, nq = s.to(D), s.shape[0], H * dim
    heads = lambda y: y.view(T, -1, dim)
    q, k = ops.rms_norm(s[:, :nq], qn.to(D), 1e-4), ops.rms_norm(s[:, nq:], kn.to(D), 1e-4)
    if temperature:
        q = q * torch.tensor([ops.query_temperature(p, *temperature) for p in range(T)], dtype=D)[:, None]
    return ops.biased_attention(heads(q), heads(k), heads(s[:, nq:]), scale, window, r1.to(D), r2.to(D)).flatten(1)


def attention_weights(H, G, dim, seed=5):
    g = torch.Generator().manual_seed(seed)
    uni = lambda top: (top * torch.rand(H, generator=g)).to(torch.bfloat16)
    return RAND(g, H * dim, std=0.3, mean=1.2), RAND(g, G * dim, std=0.3, mean=1.2), uni(2.5), uni(0.8)


ATTENTION = [(4, 2, 16, 0.3, 9, (0.5, 4)), (3, 3, 20, 0.25, 13, (0.3, 1)), (6, 1, 72, 0.1, 1, None), (5, 1, 128, 0.1, 16, (1.5, 7)),
             (2, 1, 168, 0.08, 20, (0.2, 30)), (16, 2, 64, 0.12, 0, (0.0, 3)), (4, 4, 30, 0.2, 8, (-0.3, 5)), (1, 1, 1, 1.0, 3, (0.4, 2)),
             (40, 20, 136, 0.05, 200, (0.7, 3))]


@DT
@BOTH_SIZES
@pytest.mark.parametrize("case", ATTENTION, ids=str)
def test_attention_with_norms_over_all_heads_and_a_distance_bias(dtype, tokens, case):
    H, G, dim = case[:3]
    src = [s.to(torch.bfloat16).float() for s in rows((H + G) * dim, 51, tokens)]
    args = case + attention_weights(H, G, dim)
    b = Bench(3, tokens=tokens)
    proj, out = attention_graph(b, dtype, *args)
    schedule, restart, lengths = PLANS[tokens]
    got = feed(b, src, proj, out, schedule, restart)
    for r in range(3):
        assert err(got[r], attention_reference(src[r][:lengths[r]], *args)) < (TOL[dtype] if dtype == torch.float32 else 1.5e-2), r


def test_norm_over_more_columns_than_registers_hold():
    """Rows of more than 4096 columns, queries only and with caches."""
    H, G, dim, n = 70, 35, 120, 5
    g = torch.Generator().manual_seed(1)
    b = Bench(1, tokens=8)
    x = torch.randn(8, (H + G) * dim, generator=g)
    qn, kn = RAND(g, H * dim, std=0.3, mean=1.0), RAND(g, G * dim, std=0.3, mean=1.0)
    q, only, kc, vc = b.zeros(8, H * dim), b.zeros(8, H * dim), b.zeros(64, b.page, G, dim), b.zeros(64, b.page, G, dim + 8)
    xt, kw = b.inp(x, "x"), dict(heads=H, kv_heads=G, dim=dim, vdim=dim, q_col=0, rot_dims=0, eps=1e-5, whole_norm=True)
    b.pk.qkv_append_layer(xt, b.pk.attach_input(q, name="q"), b.pk.attach_input(kc, name="kc"), b.pk.attach_input(vc, name="vc"), None, None,
                          k_col=H * dim, v_col=0, q_norm=b.inp(qn, "qn"), k_norm=b.inp(kn, "kn"), temperature=(0.5, 2), **kw)
    b.pk.qkv_append_layer(xt, b.pk.attach_input(only, name="only"), None, None, None, None, q_norm=b.inp(qn, "qn2"), **kw)
    mark_type(b, torch.float32)
    b.pk.compile()
    b.describe([n])
    b.pk.step(1)
    b.pk.status()
    s = x[:n].double()
    ref = ops.rms_norm(s[:, :H * dim], qn.double(), 1e-5)
    temp = torch.tensor([ops.query_temperature(p, 0.5, 2) for p in range(n)], dtype=D)[:, None]
    assert err(only[:n].double().cpu(), ref) < 2e-6 and err(q[:n].double().cpu(), ref * temp) < 2e-6
    page = b.pages[0][0]
    assert err(kc[page, :n].flatten(1).double().cpu(), ops.rms_norm(s[:, H * dim:], kn.double(), 1e-5)) < 2e-6
    assert torch.equal(vc[page, :n, :, :dim].flatten(1).cpu(), x[:n, :G * dim]) and float(vc[..., dim:].abs().max()) == 0.0


EDGES = pytest.mark.parametrize("window", [45, 64, 139, 256])


@DT
@pytest.mark.parametrize("page", [8, 6])
@EDGES
def test_keys_at_the_edge_of_the_window(dtype, window, page):
    """Keys that stand out just inside and just outside the window, asked for from prompts and by decoded tokens, under a distance bias."""
    H, G, dim, T = 2, 1, 16, 420
    g = torch.Generator().manual_seed(window)
    s = torch.randn(T, (H + G) * dim, generator=g)
    s[:, :H * dim] *= 0.1
    s[:, 12::dim] = 0.0
    loud, asked = torch.zeros(dim), [window - 1, window, window + 1, 300, 301, T - 70, T - 4, T - 3, T - 2, T - 1]
    loud[12] = 6.0
    for t in asked:
        s[t, :H * dim] = loud.repeat(H)
        for j in (t - window + 1, t - window):
            if 0 <= j < T and j not in asked:
                s[j, H * dim:] = loud * (1.0 + 0.1 * (j % 7))
    one = lambda n: torch.ones(n, dtype=torch.bfloat16)
    bias = torch.tensor([0.3, 1.0]).to(torch.bfloat16), torch.tensor([0.2, 0.05]).to(torch.bfloat16)
    args = (H, G, dim, 0.6, window, (0.2, 100), one(H * dim), one(G * dim), *bias)
    s = s.to(torch.bfloat16).float()
    ref = attention_reference(s, *args)
    for tokens, cuts in ((32, [32] * 9 + [14, 3, 32, 32, 32, 1, 1, 8, 2, 1, 1, 1, 1, 1, 1, 1]), (4, [4] * 105)):
        b = Bench(2, tokens=tokens, page=page, pages=512 // page, max_seq=512)
        proj, out = attention_graph(b, dtype, *args)
        got = run_alone(b, s, proj, out, cuts)
        for t in range(T):
            e = float((got[t] - ref[t]).abs().max() / ref[t].abs().max())
            assert e < (1e-5 if dtype == torch.float32 else 6e-2), (tokens, t, e)


@DT
def test_distance_bias_over_a_long_context(dtype):
    """Equal scores: the weights are the biases' alone, (1 + r2 distance)^-r1 up to their sum."""
    T, H, dim = 900, 4, 8
    g = torch.Generator().manual_seed(3)
    s = torch.randn(T, (H + 1) * dim, generator=g)
    s[:, :H * dim] = 0.0
    s = s.to(torch.bfloat16).float()
    r1, r2 = torch.tensor([0.0, 0.5, 3.0, 1.0]).to(torch.bfloat16), torch.tensor([1.0, 4.0, 0.01, 0.0]).to(torch.bfloat16)
    one = lambda n: torch.ones(n, dtype=torch.bfloat16)
    args = (H, 1, dim, 1.0, 0, None, one(H * dim), one(dim), r1, r2)
    b = Bench(2, tokens=64, page=16, pages=64, max_seq=960)
    proj, out = attention_graph(b, dtype, *args)
    got = run_alone(b, s, proj, out, [64] * 13 + [1] * 68)
    d = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp(min=0).to(D)
    wts = torch.tril(torch.ones(T, T, dtype=D)) * (1 + r2.to(D)[:, None, None] * d) ** (-r1.to(D)[:, None, None])
    ref = torch.einsum("hij,jd->ihd", wts / wts.sum(-1, keepdim=True), s[:, H * dim:].to(D)).flatten(1)
    assert err(got, ref) < (3e-6 if dtype == torch.float32 else 5e-3)


# ---- latent attention with windows, a gate and shared latents
def latent_graph(b, dtype, H, dim, vdim, rank, scale, window, norm, uk, uv, second=None):
    """[queries | latent | gate] -> gated values, as RuludraBuilder wires it.  `second` = (heads, window, uk, uv): a further layer over the
    same latents, whose queries and gate are the leading ones."""
    from mirage_b200.builders.ruludra import LatentSpec
    row = LatentSpec(H, dim, vdim, 1, rank, scale, window, None).row(dtype)
    proj = b.zeros(b.B, rank + H * vdim)
    pt = b.pk.attach_input(proj, name="proj")
    cache = b.pk.attach_input(b.zeros(b.pk.max_num_pages, b.page, 1, row, dtype=dtype), name="cache")
    b.pk.latent_append_layer(pt, b.inp(norm, "norm"), None, cache, None, None, heads=H, rank=rank, rot_dims=0, q_col=0, kv_col=0, eps=1e-4)
    ukp = pad_k(uk.view(H, dim, rank).transpose(1, 2), dtype)
    dim_p = ukp.shape[2]
    q_un = b.zeros(b.B, H, dim_p, dtype=dtype)
    qt = b.pk.attach_input(q_un.view(b.B, -1), name="q_un")

    def layer(tag, heads, win, up, down):
        wk, wv = pad_k(up.view(heads, dim, rank).transpose(1, 2), dtype), pad_k(down.view(heads, vdim, rank), dtype)
        q, mid = (b.pk.attach_input(b.zeros(b.B, heads * n, dtype=dtype), name=tag + nm) for nm, n in (("q", row), ("mid", wv.shape[2])))
        out = b.zeros(b.B, heads * vdim + 4, dtype=dtype)
        b.pk.grouped_linear_layer(qt, b.inp(wk, tag + "uk"), q, in_stride=dim_p, out_stride=row)
        b.pk.ext_attention_layer(q, cache, cache, mid, heads=heads, kv_heads=1, vdim=wv.shape[2], scale=scale, window=win, separate_merge=True)
        b.pk.grouped_linear_layer(mid, b.inp(wv, tag + "uv"), b.pk.attach_input(out, name=tag + "out"), in_stride=wv.shape[2], out_col=4,
                                  out_stride=vdim, gate=pt, gate_col=rank)
        return out[:, 4:]
    outs = [layer("a", H, window, uk, uv)] + ([layer("b", *second)] if second else [])
    b.pk.compile()

    class Split:
        def __setitem__(self, r, v):
            q_un[r, :, :dim] = v[:H * dim].view(H, dim).cuda().to(dtype)
            proj[r] = v[H * dim:].cuda()
    return Split(), outs[-1]


def latent_reference(s, H, dim, vdim, rank, scale, window, norm, uk, uv, second=None):
    s, T = s.to(D), s.shape[0]
    c = ops.rms_norm(s[:, H * dim:H * dim + rank], norm.to(D), 1e-4)
    heads, window, uk, uv = second or (H, window, uk, uv)
    q, gate = s[:, :heads * dim].view(T, heads, dim), s[:, H * dim + rank:][:, :heads * vdim]
    return ops.latent_window_attention(q, c, uk.to(D), uv.to(D), scale, window).flatten(1) * torch.sigmoid(gate)


LATENT = [(2, 16, 24, 40, 9), (3, 12, 10, 24, 1), (1, 64, 16, 72, 0), (6, 20, 32, 128, 17), (5, 24, 16, 200, 30), (17, 16, 8, 64, 8),
          (2, 32, 40, 512, 64), (40, 16, 16, 320, 5), (1, 1, 1, 1, 2)]


@DT
@BOTH_SIZES
@pytest.mark.parametrize("shared", [False, True], ids=["own", "shared"])
@pytest.mark.parametrize("H,dim,vdim,rank,window", LATENT)
def test_windowed_latent_attention(dtype, tokens, shared, H, dim, vdim, rank, window):
    src = [s.to(torch.bfloat16).float() for s in rows(H * (dim + vdim) + rank, 52, tokens)]
    g = torch.Generator().manual_seed(6)
    up = lambda h, n: RAND(g, h * n, rank, std=rank ** -0.5)
    h2 = (H + 1) // 2
    args = (H, dim, vdim, rank, 0.7 * dim ** -0.5, window, RAND(g, rank, std=0.3, mean=1.0), up(H, dim), up(H, vdim),
            (h2, 12 if window != 12 else 3, up(h2, dim), up(h2, vdim)) if shared else None)
    b = Bench(3, tokens=tokens)
    dst, out = latent_graph(b, dtype, *args)
    schedule, restart, lengths = PLANS[tokens]
    got = feed(b, src, dst, out, schedule, restart)
    for r in range(3):
        ref = latent_reference(src[r][:lengths[r]], *args)
        assert err(got[r], ref) < (1e-5 if dtype == torch.float32 else 2.5e-2), (r, err(got[r], ref))


@DT
@pytest.mark.parametrize("page", [8, 6])
@EDGES
def test_latents_at_the_edge_of_the_window(dtype, window, page):
    """Latents that stand out just inside and just outside the window, asked for from prompts and by decoded tokens."""
    H, dim, vdim, rank, T = 3, 16, 8, 64, 420
    g = torch.Generator().manual_seed(window)
    s = 0.3 * torch.randn(T, H * (dim + vdim) + rank, generator=g)
    uk, uv = RAND(g, H * dim, rank, std=rank ** -0.5), RAND(g, H * vdim, rank, std=rank ** -0.5)
    asked = [window - 1, window, window + 1, 300, 301, T - 70, T - 4, T - 3, T - 2, T - 1]
    lat = ops.rms_unit(s[:, H * dim:H * dim + rank].double(), 1e-4)
    for n, t in enumerate(asked):                                   # one asks for the first latent of its window, the next for the one before it
        key = (uk.double() @ lat[max(t - window + 1 - n % 2, 0)]).view(H, dim)
        s[t, :H * dim] = (12.0 * key / (key * key).sum(-1, keepdim=True)).flatten().float()
    s = s.to(torch.bfloat16).float()
    args = (H, dim, vdim, rank, 1.0, window, torch.ones(rank, dtype=torch.bfloat16), uk, uv)
    ref = latent_reference(s, *args)
    for tokens, cuts in ((32, [32] * 9 + [14, 3, 32, 32, 32, 1, 1, 8, 2, 1, 1, 1, 1, 1, 1, 1]), (4, [4] * 105)):
        b = Bench(2, tokens=tokens, page=page, pages=512 // page, max_seq=512)
        dst, out = latent_graph(b, dtype, *args)
        got = run_alone(b, s, dst, out, cuts)
        for t in range(T):
            e = float((got[t] - ref[t]).abs().max() / ref[t].abs().max())
            assert e < (2e-5 if dtype == torch.float32 else 6e-2), (tokens, t, e)


@DT
@pytest.mark.parametrize("tokens", [3, 8, 40])
@pytest.mark.parametrize("groups,N,K", [(3, 20, 64), (1, 200, 128), (17, 8, 64), (4, 130, 192)])
def test_grouped_linear_with_a_gate(dtype, tokens, groups, N, K):
    g = torch.Generator().manual_seed(9)
    b = Bench(1, tokens=tokens)
    stride, ostride, gstride = K + 8, N + 3, N + 1
    w, x = RAND(g, groups, N, K, std=K ** -0.5), torch.randn(tokens, groups * stride, generator=g).to(dtype)
    gate, out = 3 * torch.randn(tokens, 7 + groups * gstride, generator=g), b.zeros(tokens, 5 + groups * ostride, dtype=dtype)
    b.pk.grouped_linear_layer(b.inp(x, "x"), b.inp(w, "w"), b.pk.attach_input(out, name="o"), in_stride=stride, out_col=5, out_stride=ostride,
                              gate=b.inp(gate, "gate"), gate_col=7, gate_stride=gstride)
    mark_type(b, dtype)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    got = out.double().cpu()
    ref = torch.zeros_like(got)
    for i in range(groups):
        ref[:, 5 + i * ostride:][:, :N] = x[:, i * stride:][:, :K].to(D) @ w[i].to(D).T * torch.sigmoid(gate[:, 7 + i * gstride:][:, :N].to(D))
    assert err(got, ref) < TOL[dtype]                             # (columns between the groups stay zero)


# ---- stream, activation, head
@DT
@pytest.mark.parametrize("tokens", [1, 2, 7, 40])
@pytest.mark.parametrize("width,terms,post", [(64, 2, True), (50, 3, True), (4100, 4, True), (128, 9, False), (33, 6, False), (1024, 7, True)])
def test_average_over_the_layers_results(dtype, tokens, width, terms, post):
    g = torch.Generator().manual_seed(10)
    x, y, hist = torch.randn(tokens, width, generator=g), 3 * torch.randn(tokens, width, generator=g), torch.randn(terms + 2, tokens, width, generator=g)
    w, wp, wn = RAND(g, terms), RAND(g, width, std=0.3, mean=1.0), RAND(g, width, std=0.3, mean=1.0)
    b = Bench(1, tokens=tokens)
    results, xo, out = hist.cuda(), b.zeros(tokens, width), b.zeros(tokens, width + 5, dtype=dtype)
    b.pk.residual_norm_layer(b.inp(x, "x"), b.inp(y, "y"), b.inp(wp, "wp") if post else None, b.inp(wn, "wn"), b.pk.attach_input(out, name="o"), eps=1e-3,
                             x_out=b.pk.attach_input(xo, name="xo"), average=(b.pk.attach_input(results, name="results"), b.inp(w, "w")))
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    own = x.double() + (ops.rms_norm(y.double(), wp.double(), 1e-3) if post else y.double())
    new = ops.depth_average([*hist[:terms - 1].double(), own], w.double())
    kept = results.double().cpu()
    assert err(kept[terms - 1], own) < TOL[torch.float32] and torch.equal(kept[:terms - 1], hist[:terms - 1].double()) and torch.equal(kept[terms:], hist[terms:].double())
    assert err(xo.double().cpu(), new) < TOL[torch.float32]
    assert err(out[:, :width].double().cpu(), ops.rms_norm(new, wn.double(), 1e-3)) < TOL[dtype] and float(out[:, width:].abs().max()) == 0.0


@pytest.mark.parametrize("tokens", [1, 2])
@pytest.mark.parametrize("terms", [2, 5, 16, 17])
def test_average_over_the_layers_results_folds_into_a_linear(tokens, terms):
    g = torch.Generator().manual_seed(15)
    width, N = 100, 70
    x, y, hist = torch.randn(tokens, width, generator=g), 3 * torch.randn(tokens, width, generator=g), torch.randn(terms + 1, tokens, width, generator=g)
    w, wp, wn, lin = RAND(g, terms), RAND(g, width, std=0.3, mean=1.0), RAND(g, width, std=0.3, mean=1.0), RAND(g, N, width, std=0.1)
    b = Bench(1, tokens=tokens)
    results, xo, out = hist.cuda(), b.zeros(tokens, width), b.zeros(tokens, N)
    h = b.pk.new_tensor(dims=(tokens, 128), name="h")
    b.pk.residual_norm_layer(b.inp(x, "x"), b.inp(y, "y"), b.inp(wp, "wp"), b.inp(wn, "wn"), h, eps=1e-4, x_out=b.pk.attach_input(xo, name="xo"),
                             average=(b.pk.attach_input(results, name="results"), b.inp(w, "w")))
    b.pk.linear_layer(input=h, weight=b.inp(pad_k(lin, torch.bfloat16), "lin"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1),
                      block_dim=(128, 1, 1))
    b.pk.compile()
    assert b.pk.graph_info()["num_folded"] == int(terms <= 16)
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    own = x.double() + ops.rms_norm(y.double(), wp.double(), 1e-4)
    new = ops.depth_average([*hist[:terms - 1].double(), own], w.double())
    kept = results.double().cpu()
    assert err(kept[terms - 1], own) < TOL[torch.float32] and torch.equal(kept[:terms - 1], hist[:terms - 1].double()) and torch.equal(kept[terms], hist[terms].double())
    assert err(xo.double().cpu(), new) < TOL[torch.float32]
    assert err(out.double().cpu(), ops.rms_norm(new, wn.double(), 1e-4) @ lin.double().T) < TOL[torch.bfloat16]


@pytest.mark.parametrize("tokens", [1, 2])
@pytest.mark.parametrize("n", [1, 37, 64, 1030, 16384])
def test_normed_powers_fold_into_a_linear(tokens, n):
    g = torch.Generator().manual_seed(16)
    z, co, lin = 2.0 * torch.randn(tokens, n, generator=g), torch.tensor([0.6, -0.8, 1.1, 0.3]).to(torch.bfloat16), RAND(g, 70, n, std=n ** -0.5)
    b = Bench(1, tokens=tokens)
    padded, out = pad_k(lin, torch.bfloat16), b.zeros(tokens, 70)
    h = b.pk.new_tensor(dims=(tokens, padded.shape[1]), name="h")
    b.pk.poly_norm_layer(b.inp(z, "z"), b.inp(co, "co"), h, eps=1e-3)
    b.pk.linear_layer(input=h, weight=b.inp(padded, "lin"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
    b.pk.compile()
    assert b.pk.graph_info()["num_folded"] == 1
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    assert err(out.double().cpu(), ops.poly_norm(z.double(), co.double(), 1e-3) @ lin.double().T) < TOL[torch.bfloat16]


@DT
@pytest.mark.parametrize("tokens", [1, 2, 20])
@pytest.mark.parametrize("columns", [72, 33])
def test_norm_of_leading_columns_in_front_of_a_linear(dtype, tokens, columns):
    """One- and two-token bf16 graphs fold the norm into the linear (columns in whole vectors)."""
    g = torch.Generator().manual_seed(11)
    x, w, lin = torch.randn(tokens, 200, generator=g), RAND(g, columns, std=0.3, mean=1.0), RAND(g, 50, columns, std=0.1)
    b = Bench(1, tokens=tokens)
    padded, out = pad_k(lin, dtype), b.zeros(tokens, 50)
    h = b.pk.new_tensor(dims=(tokens, padded.shape[1]), dtype=b.mi.bfloat16 if dtype == torch.bfloat16 else b.mi.float32, name="h")
    b.pk.residual_norm_layer(b.inp(x, "x"), norm_weight=b.inp(w, "w"), output=h, eps=1e-4, columns=columns)
    b.pk.linear_layer(input=h, weight=b.inp(padded, "lin"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
    b.pk.compile()
    assert b.pk.graph_info()["num_folded"] == int(dtype == torch.bfloat16 and tokens <= 2 and columns % 4 == 0)
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    assert err(out.double().cpu(), ops.rms_norm(x[:, :columns].double(), w.double(), 1e-4) @ lin.double().T) < TOL[dtype]


@DT
@pytest.mark.parametrize("tokens", [1, 9, 64])
@pytest.mark.parametrize("n", [1, 37, 64, 1030, 4096, 16384, 20000])
def test_normed_powers(dtype, tokens, n):
    g = torch.Generator().manual_seed(12)
    z, co = 2.5 * torch.randn(tokens, n, generator=g), torch.tensor([0.6, -0.8, 1.1, 0.3]).to(torch.bfloat16)
    b = Bench(1, tokens=tokens)
    out = b.zeros(tokens, n + 4, dtype=dtype)
    b.pk.poly_norm_layer(b.inp(z, "z"), b.inp(co, "co"), b.pk.attach_input(out, name="o"), eps=1e-3)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    ref = ops.poly_norm(z.double(), co.double(), 1e-3)
    rel = (out[:, :n].double().cpu() - ref).abs() / (1.0 + ref.abs())
    assert float(rel.max()) < TOL[dtype] and float(out[:, n:].abs().max()) == 0.0


@DT
@pytest.mark.parametrize("tokens", [1, 8, 30, 64])
def test_linear_times_a_factor(dtype, tokens):
    g = torch.Generator().manual_seed(13)
    x, w = torch.randn(tokens, 192, generator=g).to(dtype), RAND(g, 333, 192, std=0.1)
    b = Bench(1, tokens=tokens)
    out = b.zeros(tokens, 336)
    b.pk.linear_layer(input=b.inp(x, "x"), weight=b.inp(w, "w"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1), block_dim=(128, 1, 1),
                      activation="scale", scale=-0.37)
    mark_type(b, dtype)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    assert err(out[:, :333].double().cpu(), -0.37 * (x.double() @ w.double().T)) < 3e-6 and float(out[:, 333:].abs().max()) == 0.0


# ---- embedding
def embedding(width, V, buckets, bigram, positions, tokens=32, max_seq=256, pages=64, page=8):
    g = torch.Generator().manual_seed(14)
    b = Bench(3, tokens=tokens, max_seq=max_seq, pages=pages, page=page)
    table, ids = b.zeros(3, max_seq, dtype=torch.int64), b.meta["input_tokens"]
    b.pk.finalize()
    b.meta["tokens"] = table
    b.pk = b.mi.PersistentKernel(mode="online_notoken", max_seq_length=max_seq, max_num_batched_requests=3, max_num_batched_tokens=tokens,
                                 max_num_pages=pages, page_size=page, meta_tensors=b.meta)
    e, two = RAND(g, V, width), RAND(g, buckets + 1, width)
    out, copy = b.zeros(tokens, width), b.zeros(2, tokens, width)
    b.pk.embed_layer(input=b.pk.attach_input(ids, name="ids"), weight=b.inp(e, "e"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1),
                     block_dim=(128, 1, 1), input_source=1, factor=0.5, copy=b.pk.attach_input(copy, name="copy"),
                     bigram=(b.inp(two, "two"), 10007, 300) if bigram else None,
                     positions=b.inp(b.pk.position_frequencies(width), "freq") if positions else None)
    mark_type(b, torch.float32)
    b.pk.compile()

    def reference(toks):
        x = 0.5 * e.double()[torch.tensor(toks)]
        if bigram:
            x = x + two.double()[torch.tensor(ops.bigram_rows(toks, buckets, 10007, 300))]
        return x + ops.sinusoids(len(toks), width, D) if positions else x
    return b, table, ids, out, copy, reference


@pytest.mark.parametrize("width,buckets,bigram,positions", [(64, 97, True, True), (37, 1, True, False), (50, 4096, False, True), (1, 5, True, True),
                                                            (1100, 31, True, True)])
def test_embedding_with_bigrams_and_positions(width, buckets, bigram, positions):
    b, table, ids, out, copy, reference = embedding(width, 40, buckets, bigram, positions)
    toks = [random.Random(r).choices(range(40), k=n) for r, n in enumerate((60, 33, 12))]
    for r, t in enumerate(toks):
        table[r, :len(t)] = torch.tensor(t)
    refs, at = [reference(t) for t in toks], [0, 0, 0]
    for counts in ([7, 0, 1], [2, 5, 1], [1, 1, 1], [20, 9, 1], [1, 1, 2], [29, 1, 1], [0, 16, 5]):
        for r, pos, row in b.describe(counts):
            ids[row] = toks[r][pos]
        b.pk.step(1)
        b.pk.status()
        row = 0
        for r, n in enumerate(counts):
            if n:
                assert float((out[row:row + n].double().cpu() - refs[r][at[r]:at[r] + n]).abs().max()) < 2e-6
            at[r] += n
            row += n
        assert torch.equal(copy[0, :row], out[:row]) and float(copy[1].abs().max()) == 0.0
    assert at == [60, 33, 12]


def test_positions_far_into_a_sequence():
    """Angles stay exact where a float32 product of position and frequency would have lost them."""
    width, T = 32, 20000
    b, table, ids, out, _, _ = embedding(width, 4, 3, False, True, tokens=2, max_seq=T, pages=T // 100, page=100)
    b.len[1], b.pages[1] = T - 2, list(range(T // 100))
    b.describe([0, 2, 0])
    ids[:] = 5                                                      # outside the table: a zero row
    b.pk.step(1)
    b.pk.status()
    ref = torch.tensor([[(torch.cos if j % 2 else torch.sin)(torch.tensor(p * 10000.0 ** (-2.0 * (j // 2) / width), dtype=D)) for j in range(width)]
                        for p in (T - 2, T - 1)], dtype=D)
    assert float((out.double().cpu() - ref).abs().max()) < 5e-7
