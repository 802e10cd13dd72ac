"""The mechanisms Lofirax adds to hybrid graphs, each alone on the GPU against oracle/hybrid_ops.py: sizes that divide nothing,
requests of unequal length in one batch, portions down to one token, state slots and pages that are not the identity."""
import pytest
import torch

from oracle import hybrid_ops as ops
from test_gpu_hybrid_ops import D, DTYPES, LENGTHS, RESTART, SCHEDULE, TOL, Bench, err, feed, sources

pytestmark = pytest.mark.gpu
RAND = lambda g, *s, std=1.0, mean=0.0: (mean + std * torch.randn(*s, generator=g)).to(torch.bfloat16)


def pad_k(w, dtype):
    from mirage_b200.builders.hybrid import k_padded
    return torch.nn.functional.pad(w, (0, k_padded(w.shape[-1], dtype) - w.shape[-1]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rank", [(2, 16, 24, 8), (1, 20, 7, 3), (3, 130, 66, 16), (1, 300, 40, 1), (2, 64, 200, 40),
                                                 (1, 600, 530, 5), (2, 256, 96, 16)])
def test_gla(dtype, heads, dim, vdim, rank):
    qk, v = heads * dim, heads * vdim
    src = sources(2 * qk + 2 * v + rank, 21)
    g = torch.Generator().manual_seed(4)
    # decays from a few tokens to far beyond the sequence, per key channel
    a2, bias, norm = RAND(g, qk, rank, std=rank ** -0.5), RAND(g, qk, std=3.0, mean=2.0), RAND(g, vdim, std=0.3, mean=1.0)
    b = Bench(3)
    proj, out = b.zeros(b.B, src[0].shape[1]), b.zeros(b.B, v, dtype=dtype)
    b.pk.gla_layer(b.pk.attach_input(proj, name="proj"), b.inp(a2, "a2"), b.inp(bias, "bias"), b.inp(norm, "norm"),
                   b.pk.attach_input(b.zeros(3, heads, dim, (vdim + 3) // 4 * 4), name="S"), b.pk.attach_input(b.zeros(b.B, v), name="raw"),
                   b.pk.attach_input(out, name="out"), heads=heads, dim=dim, vdim=vdim, q_col=0, k_col=qk, v_col=2 * qk,
                   gate_col=2 * qk + v, a1_col=2 * qk + 2 * v, tau=3.0, eps=1e-4, q_scale=dim ** -0.5,
                   chunks=b.pk.mlstm_chunks(b.pk.num_workers, 3, heads, dim, vdim))
    b.pk.compile()
    got = feed(b, src, proj, out, SCHEDULE, RESTART)
    for r in range(3):
        s = src[r][:LENGTHS[r]].to(D)
        cut = lambda a, n, w: s[:, a:a + n * w].view(-1, n, w)
        z = (s[:, 2 * qk + 2 * v:] @ a2.to(D).T + bias.to(D)).view(-1, heads, dim)
        o = ops.gla(cut(0, heads, dim) * dim ** -0.5, cut(qk, heads, dim), cut(2 * qk, heads, vdim), z, 3.0)
        ref = (ops.rms_unit(o, 1e-4) * norm.to(D)).reshape(-1, v) * ops.silu(s[:, 2 * qk + v:2 * qk + 2 * v])
        assert got[r].shape == ref.shape and err(got[r], ref) < TOL[dtype], (r, err(got[r], ref))


@pytest.mark.parametrize("dtype", DTYPES)
def test_gla_keeps_a_key_for_the_whole_sequence(dtype):
    """One key channel that does not decay holds what the first token wrote; a query far behind asks for it."""
    T, dim, vdim = 150, 16, 8
    src = torch.zeros(T, 2 * dim + 2 * vdim + 1)
    src[0, dim] = 1.0                                             # key of the first token: channel 0
    src[0, 2 * dim:2 * dim + vdim] = torch.arange(1, vdim + 1)
    src[1:, dim + 1] = 1.0                                        # later keys: channel 1, which forgets at once
    src[1:, 2 * dim:2 * dim + vdim] = 50.0
    src[:, 0] = 1.0                                               # queries look at channel 0
    src[:, 2 * dim + vdim:2 * dim + 2 * vdim] = 3.0
    bias = torch.full((dim,), 60.0)
    bias[1] = -60.0
    for cuts in ([[T]], [[1]] * T, [[64], [2]] + [[7]] * 12):
        b = Bench(1, tokens=T if cuts == [[T]] else 64, pages=64)
        if b.B > 64:
            cuts = [[64], [64], [22]]
            b = Bench(1, tokens=64, pages=64)
        proj, out = b.zeros(b.B, src.shape[1]), b.zeros(b.B, vdim, dtype=dtype)
        b.pk.gla_layer(b.pk.attach_input(proj, name="proj"), b.inp(torch.zeros(dim, 1, dtype=torch.bfloat16), "a2"),
                       b.inp(bias.to(torch.bfloat16), "bias"), b.inp(torch.ones(vdim, dtype=torch.bfloat16), "norm"),
                       b.pk.attach_input(b.zeros(1, 1, dim, vdim), name="S"), b.pk.attach_input(b.zeros(b.B, vdim), name="raw"),
                       b.pk.attach_input(out, name="out"), heads=1, dim=dim, vdim=vdim, q_col=0, k_col=dim, v_col=2 * dim,
                       gate_col=2 * dim + vdim, a1_col=2 * dim + 2 * vdim, tau=16.0, eps=1e-5, q_scale=1.0, chunks=1)
        b.pk.compile()
        got = feed(b, [src], proj, out, cuts)[0]
        ref = ops.rms_unit(torch.arange(1, vdim + 1, dtype=D), 1e-5) * ops.silu(torch.tensor(3.0, dtype=D))
        assert err(got, ref.expand_as(got)) < TOL[dtype]


def latent_graph(b, dtype, H, dim, rot, vdim, rank, base, scale, eps, norm, uk, uv, sinks):
    """q_un and proj -> values, as LofiraxBuilder wires it."""
    from mirage_b200.builders.hybrid import rotary_tables
    from mirage_b200.builders.lofirax import LatentSpec
    row = LatentSpec(H, dim, rot, vdim, rank, base, scale).row(dtype)
    uk, uv = pad_k(uk.view(H, dim, rank).transpose(1, 2), dtype), pad_k(uv.view(H, vdim, rank), dtype)
    dim_p, rank_p = uk.shape[2], uv.shape[2]
    q_un, proj = b.zeros(b.B, H, dim_p, dtype=dtype), b.zeros(b.B, (H + 1) * rot + rank)
    out = b.zeros(b.B, H * vdim + 4, dtype=dtype)
    cos, sin = rotary_tables(base, rot, b.pk.max_seq_length, "cuda")
    q = b.pk.attach_input(b.zeros(b.B, H * row, dtype=dtype), name="q")
    cache = b.pk.attach_input(b.zeros(b.pk.max_num_pages, b.page, 1, row, dtype=dtype), name="cache")
    mid = b.pk.attach_input(b.zeros(b.B, H * rank_p, dtype=dtype), name="mid")
    b.pk.grouped_linear_layer(b.pk.attach_input(q_un.view(b.B, -1), name="q_un"), b.inp(uk, "uk"), q, in_stride=dim_p, out_stride=row)
    b.pk.latent_append_layer(b.pk.attach_input(proj, name="proj"), b.inp(norm, "norm"), q, cache, b.inp(cos, "cos"), b.inp(sin, "sin"),
                             heads=H, rank=rank, rot_dims=rot, q_col=0, kv_col=H * rot, eps=eps)
    b.pk.ext_attention_layer(q, cache, cache, mid, heads=H, kv_heads=1, vdim=rank_p, scale=scale, sinks=b.inp(sinks, "sinks"),
                             separate_merge=True)
    b.pk.grouped_linear_layer(mid, b.inp(uv, "uv"), b.pk.attach_input(out, name="out"), in_stride=rank_p, out_col=4, out_stride=vdim)

    class Split:                                                  # source row: [unrotated queries | rotated queries | latent | rotated key]
        def __setitem__(self, r, v):
            q_un[r, :, :dim] = v[:H * dim].view(H, dim).cuda().to(dtype)
            proj[r] = v[H * dim:].cuda()
    return Split(), out[:, 4:]


def latent_reference(s, H, dim, rot, vdim, rank, base, scale, eps, norm, uk, uv, sinks):
    """The mechanism over one sequence of source rows, keys and values expanded."""
    eye = torch.eye(s.shape[1], dtype=D)
    q_un, q_rot = eye[:H * dim].view(H, dim, -1), eye[H * dim:H * (dim + rot)].view(H, rot, -1)
    return ops.latent_attention(s.to(D), torch.cat([q_un, q_rot], 1).flatten(0, 1), eye[H * (dim + rot):], norm.to(D), uk.to(D), uv.to(D),
                                sinks.to(D), heads=H, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, base=base, scale=scale, eps=eps)


LATENT = [(2, 16, 8, 24, 40), (3, 12, 4, 10, 24), (1, 64, 2, 16, 72), (6, 20, 16, 32, 128), (5, 24, 24, 16, 200), (17, 16, 16, 8, 64),
          (2, 32, 64, 40, 512), (40, 16, 32, 16, 320)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [32, 2])
@pytest.mark.parametrize("H,dim,rot,vdim,rank", LATENT)
def test_latent_attention(dtype, tokens, H, dim, rot, vdim, rank):
    src = [s.to(torch.bfloat16).float() for s in sources(H * (dim + rot) + rank + rot, 31)]
    g = torch.Generator().manual_seed(6)
    args = (H, dim, rot, vdim, rank, 900.0, 0.7 * (dim + rot) ** -0.5, 1e-4, RAND(g, rank, std=0.3, mean=1.0),
            RAND(g, H * dim, rank, std=rank ** -0.5), RAND(g, H * vdim, rank, std=rank ** -0.5), RAND(g, H))
    b = Bench(3, tokens=tokens)
    dst, out = latent_graph(b, dtype, *args)
    b.pk.compile()
    schedule, lengths, restart = SCHEDULE, LENGTHS, RESTART
    if tokens == 2:                                               # the small graphs' tiles, with a restart of their own
        schedule, restart = [[1, 1, 0]] * 9 + [[0, 1, 1]] * 7 + [[2, 0, 0]] * 5 + [[1, 0, 1]] * 4, [(9, 1)]
        lengths = [sum(s[0] for s in schedule), 7, sum(s[2] for s in schedule)]
    got = feed(b, src, dst, out, schedule, restart)
    for r in range(3):
        ref = latent_reference(src[r][:lengths[r]], *args)
        assert err(got[r], ref) < (1e-5 if dtype == torch.float32 else 2.5e-2), (r, err(got[r], ref))


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_on_pages_of_odd_size(dtype):
    """Eight consecutive keys may lie in two pages."""
    H, dim, rot, vdim, rank = 3, 16, 8, 8, 48
    src = [s.to(torch.bfloat16).float() for s in sources(H * (dim + rot) + rank + rot, 33)]
    g = torch.Generator().manual_seed(16)
    args = (H, dim, rot, vdim, rank, 900.0, 0.15, 1e-4, RAND(g, rank, std=0.3, mean=1.0), RAND(g, H * dim, rank, std=rank ** -0.5),
            RAND(g, H * vdim, rank, std=rank ** -0.5), RAND(g, H))
    b = Bench(3, page=5)
    dst, out = latent_graph(b, dtype, *args)
    b.pk.compile()
    got = feed(b, src, dst, out, SCHEDULE, RESTART)
    for r in range(3):
        ref = latent_reference(src[r][:LENGTHS[r]], *args)
        assert err(got[r], ref) < (1e-5 if dtype == torch.float32 else 2.5e-2), r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [64, 4])
@pytest.mark.parametrize("H,dim,rot,vdim,rank", [(4, 16, 8, 16, 64), (20, 32, 64, 16, 512)])
def test_far_keys_stand_out(dtype, tokens, H, dim, rot, vdim, rank):
    """One key among hundreds takes nearly all the weight of a query: at page borders, at the borders of the key chunks tasks
    share, the first and the latest key -- from prompt rows and decoded tokens."""
    T = 330 if tokens == 64 else 200
    g = torch.Generator().manual_seed(7)
    src = 0.3 * torch.randn(T, H * (dim + rot) + rank + rot, generator=g)
    norm, uk, uv, sinks = (torch.ones(rank, dtype=torch.bfloat16), RAND(g, H * dim, rank, std=rank ** -0.5),
                           RAND(g, H * vdim, rank, std=rank ** -0.5), RAND(g, H))
    args = (H, dim, rot, vdim, rank, 1e5, 1.0, 1e-5, norm, uk, uv, sinks)
    # query t asks for the latent of key far[t]: its unrotated part is the key's own expansion, scaled up
    far = {t: t - back for t in range(T) for back in [(0, 1, 7, 8, 63, 64, 65, 127, 128, t)[t % 10]] if t - back >= 0}
    lat = ops.rms_unit(src[:, H * (dim + rot):][:, :rank].double(), 1e-5)
    for t, k in far.items():
        key = (uk.double() @ lat[k]).view(H, dim)
        src[t, :H * dim] = (30.0 * key / (key * key).sum(-1, keepdim=True)).flatten().float()
    src = src.to(torch.bfloat16).float()
    ref = latent_reference(src, *args)
    cuts = [[64]] * 4 + [[1]] * 40 + [[2], [32]] if tokens == 64 else [[4]] * 30 + [[1]] * 80
    b = Bench(1, tokens=tokens, pages=64, max_seq=400)
    dst, out = latent_graph(b, dtype, *args)
    b.pk.compile()
    got = feed(b, [src], dst, out, cuts)[0]
    assert got.shape == ref.shape
    rows = (got - ref).abs().amax(-1) / ref.abs().max()
    assert float(rows.max()) < (1e-5 if dtype == torch.float32 else 5e-2), (int(rows.argmax()), float(rows.max()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_are_per_head_and_count_once(dtype):
    """Sinks from negligible to overwhelming over keys that all score alike: the output is the keys' share of the weight."""
    H, dim, rot, vdim, rank, T = 6, 8, 4, 8, 64, 200
    g = torch.Generator().manual_seed(8)
    src = torch.zeros(T, H * (dim + rot) + rank + rot)
    src[:, H * (dim + rot):][:, :rank] = torch.randn(rank, generator=g)
    norm, uk, uv = torch.ones(rank, dtype=torch.bfloat16), RAND(g, H * dim, rank), RAND(g, H * vdim, rank, std=rank ** -0.5)
    sinks = torch.tensor([-30.0, 0.0, 3.0, 5.0, 8.0, 20.0]).to(torch.bfloat16)
    args = (H, dim, rot, vdim, rank, 100.0, 1.0, 1e-5, norm, uk, uv, sinks)
    src = src.to(torch.bfloat16).float()
    ref = latent_reference(src, *args)
    for cuts in ([[64]] * 3 + [[8]], [[1]] * T):
        b = Bench(1, tokens=64, pages=32)
        dst, out = latent_graph(b, dtype, *args)
        b.pk.compile()
        got = feed(b, [src], dst, out, cuts)[0].view(T, H, vdim)
        for h in range(H):
            want = ref.view(T, H, vdim)[:, h]
            assert float((got[:, h] - want).abs().max() / want.abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2), h


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [3, 8, 40])
@pytest.mark.parametrize("groups,N,K", [(3, 20, 64), (1, 200, 128), (17, 8, 64), (4, 130, 192)])
def test_grouped_linear(dtype, tokens, groups, N, K):
    g = torch.Generator().manual_seed(9)
    b = Bench(1, tokens=tokens)
    stride, ostride = K + 8, N + 3
    w, x = RAND(g, groups, N, K, std=K ** -0.5), torch.randn(tokens, groups * stride, generator=g).to(dtype)
    out = b.zeros(tokens, 5 + groups * ostride, dtype=dtype)
    # (a layer of the hybrid family makes the graph one)
    xt = b.inp(x, "x")
    b.pk.grouped_linear_layer(xt, b.inp(w, "w"), b.pk.attach_input(out, name="o"), in_stride=stride, out_col=5, out_stride=ostride)
    mark_type(b, dtype)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    got = out.double().cpu()
    ref = torch.zeros_like(got)
    for i in range(groups):
        ref[:, 5 + i * ostride:][:, :N] = x[:, i * stride:][:, :K].to(D) @ w[i].to(D).T
    assert err(got, ref) < TOL[dtype]                             # (columns between the groups stay zero)


def mark_type(b, dtype):
    """A norm whose output has the graph's activation type."""
    b.pk.residual_norm_layer(b.pk.attach_input(b.zeros(b.B, 8), name="mark_x"), norm_weight=b.inp(torch.ones(8, dtype=torch.bfloat16), "mark_w"),
                             output=b.pk.attach_input(b.zeros(b.B, 8, dtype=dtype), name="mark_o"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 2, 7, 40])
@pytest.mark.parametrize("width,terms", [(64, "y added row experts gate"), (50, "y experts gate bias"), (4100, "y added row bias"), (128, "row bias"),
                                         (96, "experts bias"), (64, "y bias"), (64, "added y row bias"), (33, "")])
def test_layer_norm_and_the_terms_of_the_stream(dtype, tokens, width, terms):
    g = torch.Generator().manual_seed(10)
    n = tokens
    x = 3.0 + torch.randn(n, width, generator=g)                  # a mean of its own, which a norm without it would keep
    y, added, row = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g), RAND(g, width)
    ex, ew, gate = torch.randn(n, 3, width, generator=g), torch.rand(n, 3, generator=g), torch.randn(n, 5, generator=g)
    w, bias = RAND(g, width, std=0.3, mean=1.0), RAND(g, width)
    b = Bench(1, tokens=n)
    t = terms.split()
    kw = {}
    if "y" in t:
        kw["y"] = b.inp(y, "y")
    if "added" in t:
        kw["added"] = b.inp(added, "added")
    if "row" in t:
        kw["added_row"] = b.inp(row, "row")
    if "experts" in t:
        kw["experts"] = (b.inp(ex, "ex"), b.inp(ew, "ew"))
    if "gate" in t:
        kw["y_gate"] = (b.inp(gate, "gate"), 3)
    if "bias" in t:
        kw["norm_bias"] = b.inp(bias, "bias")
    xo, out = b.zeros(n, width), b.zeros(n, width + 5, dtype=dtype)
    b.pk.residual_norm_layer(b.inp(x, "x"), norm_weight=b.inp(w, "w"), output=b.pk.attach_input(out, name="o"), eps=1e-3, layer_norm=True,
                             x_out=b.pk.attach_input(xo, name="xo") if kw and set(kw) != {"norm_bias"} else None, **kw)
    b.pk.compile()
    b.describe([n])
    b.pk.step(1)
    b.pk.status()
    s = x.double()
    if "y" in t:
        s = s + y.double() * (torch.sigmoid(gate[:, 3:4].double()) if "gate" in t else 1.0)
    if "experts" in t:
        s = s + (ex.double() * ew.double()[..., None]).sum(1)
    s = s + (added.double() if "added" in t else 0) + (row.double() if "row" in t else 0)
    ref = ops.layer_norm(s, w.double(), bias.double() if "bias" in t else torch.zeros(width, dtype=D), 1e-3)
    assert err(out[:, :width].double().cpu(), ref) < TOL[dtype] and float(out[:, width:].abs().max()) == 0.0
    if kw and set(kw) != {"norm_bias"}:
        assert err(xo.double().cpu(), s) < TOL[torch.float32]


@pytest.mark.parametrize("tokens", [1, 2])
def test_norms_with_further_terms_fold_into_a_linear(tokens):
    """Graphs of one or two tokens: the stream's sum and the layer norm are the prologue of the linear that reads them."""
    g = torch.Generator().manual_seed(11)
    width, N = 100, 70
    x, y, added, row = (torch.randn(tokens, width, generator=g), torch.randn(tokens, width, generator=g), torch.randn(tokens, width, generator=g),
                        RAND(g, width))
    w, bias, lin = RAND(g, width, std=0.3, mean=1.0), RAND(g, width), RAND(g, N, width, std=0.1)
    for use in (("y",), ("added", "row"), ("y", "added", "row"), ()):
        b = Bench(1, tokens=tokens)
        kw = {}
        if "y" in use:
            kw["y"] = b.inp(y, "y")
        if "added" in use:
            kw["added"] = b.inp(added, "added")
        if "row" in use:
            kw["added_row"] = b.inp(row, "row")
        xo, out = b.zeros(tokens, width), b.zeros(tokens, N)
        h = b.pk.new_tensor(dims=(tokens, 128), name="h")
        b.pk.residual_norm_layer(b.inp(x, "x"), norm_weight=b.inp(w, "w"), norm_bias=b.inp(bias, "bias"), output=h, eps=1e-4, layer_norm=True,
                                 x_out=b.pk.attach_input(xo, name="xo") if use else None, **kw)
        b.pk.linear_layer(input=h, weight=b.inp(pad_k(lin, torch.bfloat16), "lin"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1),
                          block_dim=(128, 1, 1))
        b.pk.compile()
        assert b.pk.graph_info()["num_folded"] == 1
        b.describe([tokens])
        b.pk.step(1)
        b.pk.status()
        s = x.double() + (y.double() if "y" in use else 0) + (added.double() if "added" in use else 0) + (row.double() if "row" in use else 0)
        ref = ops.layer_norm(s, w.double(), bias.double(), 1e-4) @ lin.double().T
        assert err(out.double().cpu(), ref) < TOL[torch.bfloat16], use
        if use:
            assert err(xo.double().cpu(), s) < TOL[torch.float32], use


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 30])
@pytest.mark.parametrize("act", ["gated_silu", "gated_gelu_tanh", "softcap", "relu2"])
def test_linear_activations(dtype, tokens, act):
    g = torch.Generator().manual_seed(12)
    K, N = 96, 74
    b = Bench(1, tokens=tokens)
    x = torch.randn(tokens, K, generator=g).to(dtype)
    gate, up = RAND(g, N, K, std=0.2), RAND(g, N, K, std=0.2)
    gated = act.startswith("gated")
    w = b.pk.interleave_gated(gate, up) if gated else gate
    odt = torch.float32 if act == "softcap" else dtype
    out = b.zeros(tokens, N + 6, dtype=odt)
    xp = pad_k(x, dtype)
    b.pk.linear_layer(input=b.inp(xp, "x"), weight=b.inp(pad_k(w, dtype), "w"), output=b.pk.attach_input(out, name="o"), grid_dim=(1, 1, 1),
                      block_dim=(128, 1, 1), activation=act, **(dict(softcap=1.5) if act == "softcap" else {}))
    mark_type(b, dtype)
    b.pk.compile()
    b.describe([tokens])
    b.pk.step(1)
    b.pk.status()
    z, u = x.double() @ gate.double().T, x.double() @ up.double().T
    ref = {"gated_silu": lambda: ops.silu(z) * u, "gated_gelu_tanh": lambda: ops.gelu_tanh(z) * u, "softcap": lambda: ops.softcap(z, 1.5),
           "relu2": lambda: ops.squared_relu(z)}[act]()
    assert err(out[:, :N].double().cpu(), ref) < TOL[odt] and float(out[:, N:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 8, 64])
@pytest.mark.parametrize("E,top,groups,keep,ff,width", [(6, 2, 2, 1, 40, 64), (12, 4, 4, 3, 64, 96), (8, 8, 1, 1, 24, 64), (5, 1, 5, 2, 130, 128),
                                                        (64, 6, 8, 4, 32, 64)])
def test_expert_layers(dtype, tokens, E, top, groups, keep, ff, width):
    """Routing on negative and positive choice scores, gated experts, and their weighted sum in the norm's task."""
    g = torch.Generator().manual_seed(13)
    b = Bench(1, tokens=tokens)
    F = (ff + 63) // 64 * 64 if dtype == torch.bfloat16 else ff
    h = torch.randn(tokens, width, generator=g).to(torch.bfloat16)
    logits = 2.0 * torch.randn(tokens, E + 2, generator=g)
    corr = 0.8 * torch.randn(E, generator=g) - 0.9                 # many choice scores below zero
    gate, up, down = (RAND(g, E, ff, width, std=0.2), RAND(g, E, ff, width, std=0.2), RAND(g, E, width, ff, std=0.2))
    rows = lambda t: torch.nn.functional.pad(t, (0, 0, 0, F - ff))
    w13 = pad_k(b.pk.interleave_gated(rows(gate), rows(up)), dtype)
    w2 = torch.nn.functional.pad(down, (0, F - ff))
    mi = b.mi
    new = lambda name, dims, dt: b.pk.new_tensor(dims=dims, dtype=dt, name=name)
    wts, idx, act = new("wts", (tokens, top), mi.float32), new("idx", (E, tokens), mi.int32), new("act", (E + 1,), mi.int32)
    grid = dict(grid_dim=(1, 1, 1), block_dim=(128, 1, 1))
    lt = b.inp(logits, "logits")
    b.pk.moe_topk_sigmoid_routing_layer(lt, b.inp(corr, "corr"), (wts, idx, act), **grid, num_groups=groups, topk_group=keep,
                                        routed_scaling_factor=1.0, keep_logits=True)
    mid = new("mid", (tokens, top, F), mi.bfloat16 if dtype == torch.bfloat16 else mi.float32)
    out = new("out", (tokens, top, width), mi.float32)
    b.pk.moe_w13_linear_layer(b.inp(pad_k(h, dtype).to(dtype), "h"), b.inp(w13, "w13"), idx, act, mid, **grid, activation="gated_silu")
    b.pk.moe_w2_linear_layer(mid, b.inp(w2, "w2"), idx, act, out, **grid)
    x, xo = torch.randn(tokens, width, generator=g), b.zeros(tokens, width)
    b.pk.residual_norm_layer(b.inp(x, "x"), norm_weight=b.inp(torch.ones(width, dtype=torch.bfloat16), "w"),
                             output=b.pk.attach_input(b.zeros(tokens, width, dtype=dtype), name="o"), experts=(out, wts),
                             x_out=b.pk.attach_input(xo, name="xo"))
    b.pk.compile()
    b.describe([tokens])
    for _ in range(2):                                             # (the logits are still there the second time)
        b.pk.step(1)
        b.pk.status()
    s = torch.sigmoid(logits[:, :E].double())
    ref = x.double()
    for t in range(tokens):
        chosen = ops.grouped_choice(s[t], corr.double(), groups, keep, top)
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            ref[t] += s[t, e] / total * ops.gated_ff(h[t].double(), gate[e].double(), up[e].double(), down[e].double(), ops.silu)
    assert err(xo.double().cpu(), ref) < TOL[dtype]


def test_embedding_factor():
    b = Bench(1, tokens=5)
    table = RAND(torch.Generator().manual_seed(14), 30, 40)
    ids = torch.tensor([3, 0, 29, 17, 3])
    out = b.zeros(5, 40)
    b.meta["input_tokens"][:, 0] = ids.cuda()
    b.pk.embed_layer(input=b.pk.attach_input(b.meta["input_tokens"], name="ids"), weight=b.inp(table, "t"), output=b.pk.attach_input(out, name="o"),
                     grid_dim=(1, 1, 1), block_dim=(128, 1, 1), input_source=1, factor=2.7)
    mark_type(b, torch.bfloat16)
    b.pk.compile()
    b.describe([5])
    b.pk.step(1)
    b.pk.status()
    assert err(out.double().cpu(), 2.7 * table[ids].double()) < 1e-6
