"""Each kernel of the Delunex path alone, against the plain implementation in float64."""

import math

import pytest
import torch

from oracle import ref_delunex as ref

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *s, dtype=torch.float32, scale=1.0):
    return (torch.randn(*s, generator=g) * scale).to(dtype)


def close(got, want, dtype, f32=2e-5, bf16=1.2e-2):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    assert bool(torch.isfinite(got).all())
    if want.numel() == 0:
        return
    tol = f32 if dtype == torch.float32 else bf16
    err = (got - want).abs().max().item()
    assert err <= tol * max(want.abs().max().item(), 1e-3), err


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C", [5, 52, 320, 1028, 2048, 8200])
def test_embedding_and_norms(dtype, C):
    from diff_gpt_b200 import ops

    g, n, V = gen(C), 7, 19
    table, ids = rnd(g, V, C, dtype=dtype), torch.randint(0, V, (n,), generator=g)
    out = torch.empty(n, C, device="cuda")
    ops.embed_scale(ids.int().cuda(), table.cuda(), out, 3.7)
    close(out, ref.embed(ids, table.double(), 3.7), torch.float32)
    y, w, x = rnd(g, n, C, dtype=dtype, scale=0.01), rnd(g, C), rnd(g, n, C)
    want = x.double() + ref.rms_norm(y.double(), w.double(), 1e-3)
    xd = x.cuda()
    u = torch.empty(n, C, dtype=dtype, device="cuda")
    ops.norm_add(y.cuda(), w.cuda(), 1e-3, xd, xd, rounded=u)  # in place
    close(xd, want, torch.float32)
    close(u, want, dtype, bf16=5e-3)
    slab, a = rnd(g, 5, n, C), rnd(g, 5)
    for rows in (None, torch.tensor([6, 0, 3], dtype=torch.int32)):
        o = torch.empty(n if rows is None else 3, C, dtype=dtype, device="cuda")
        ops.depth_avg_norm(slab.cuda(), 4, a.cuda(), w.cuda(), 1e-2, o, rows=None if rows is None else rows.cuda())
        want = ref.rms_norm(ref.depth_average(list(slab[:4].double()), a.double()), w.double(), 1e-2)
        close(o, want if rows is None else want[rows.long()], dtype, bf16=5e-3)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8, 9, 16])
@pytest.mark.parametrize("C,terms", [(52, 1), (7, 3), (256, 9)])
def test_depth_average_and_convolution_in_portions(taps, C, terms):
    """Whole sequences and the same cut into portions (shorter than the filter too), two sequences at a time; the state
    carried over is the last taps - 1 averages."""
    from diff_gpt_b200 import ops

    g, B, T = gen(100 * taps + C), 2, 150
    slab, a, cw = rnd(g, terms, B, T, C), rnd(g, terms), rnd(g, C, taps)
    avg = ref.depth_average(list(slab.double()), a.double())
    want = torch.stack([avg[b] + ref.causal_conv(avg[b], cw.double()) for b in range(B)])
    wt = cw.t().contiguous().cuda()
    state = [torch.zeros(B, taps - 1, C, device="cuda"), torch.full((B, taps - 1, C), float("nan"), device="cuda")]
    for cuts in ([T], [1] * 6 + [2, 3, 1, 70, 2, 66], [75, 75]):
        state[0].zero_()
        at = 0
        for n in cuts:
            part = slab[:, :, at : at + n].reshape(terms, B * n, C).contiguous().cuda()
            x, h = torch.empty(B * n, C, device="cuda"), torch.empty(B * n, C, device="cuda")
            in_place = n == 1
            ops.depth_avg_conv(part, terms, a.cuda(), wt, h, n_seq=B, T=n, x=x, state_in=state[0],
                               state_out=state[0] if in_place else state[1])
            if not in_place:
                state.reverse()
            close(x.view(B, n, C), avg[:, at : at + n], torch.float32)
            close(h.view(B, n, C), want[:, at : at + n], torch.float32)
            at += n
        assert at == T
        close(state[0], avg[:, T - (taps - 1) :], torch.float32)
    # no state given: zeros before the first token
    h = torch.empty(B * T, C, dtype=torch.bfloat16, device="cuda")
    ops.depth_avg_conv(slab.reshape(terms, B * T, C).cuda(), terms, a.cuda(), wt, h, n_seq=B, T=T)
    close(h.view(B, T, C), want, torch.bfloat16, bf16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,C", [(1, 52), (2, 30), (4, 320), (6, 2048)])
def test_layer_tail_equals_its_parts(dtype, taps, C):
    from diff_gpt_b200 import ops

    g, R, terms = gen(taps), 5, 4
    y, w, x1 = rnd(g, R, C, dtype=dtype), rnd(g, C), rnd(g, R, C)
    slab, a, cw, st = rnd(g, terms + 2, R, C).cuda(), rnd(g, terms).cuda(), rnd(g, taps, C).cuda(), rnd(g, R, taps - 1, C).cuda()
    slab_b, st_b = slab.clone(), st.clone()
    x, h = torch.empty(R, C, device="cuda"), torch.empty(R, C, dtype=dtype, device="cuda")
    ops.layer_tail(y.cuda(), w.cuda(), 1e-4, x1.cuda(), slab, terms, a, cw, st, x, h)
    xb, hb = torch.empty_like(x), torch.empty_like(h)
    ops.norm_add(y.cuda(), w.cuda(), 1e-4, x1.cuda(), slab_b[terms - 1])
    ops.depth_avg_conv(slab_b, terms, a, cw, hb, n_seq=R, T=1, x=xb, state_in=st_b, state_out=st_b)
    for p, q in ((slab, slab_b), (x, xb), (st, st_b)):
        close(p, q.cpu(), torch.float32, f32=1e-6)
    close(h, hb.cpu(), dtype, f32=1e-6, bf16=5e-3)
    # and the plain rule: the new term, the average, the shifted state
    want_new = x1.double() + ref.rms_norm(y.double(), w.double(), 1e-4)
    close(slab[terms - 1], want_new, torch.float32)
    close(x, ref.depth_average(list(slab[:terms].double().cpu()), a.double().cpu()), torch.float32)
    if taps > 1:
        close(st[:, -1], x.double().cpu(), torch.float32, f32=0.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_xielu_values_and_gemm_epilogue(dtype):
    from diff_gpt_b200 import ops
    from diff_gpt_b200.model.delunex import _softplus

    pq = torch.tensor([0.7, -1.3]).double()
    ap, an = _softplus(0.7), 0.5 + _softplus(-1.3)
    z = torch.cat([torch.linspace(-12, 12, 3001), torch.tensor([0.0, -0.0, 1e-6, -1e-6, -80.0])]).to(dtype)
    out = torch.empty_like(z, device="cuda")
    ops.xielu(z.cuda(), out, ap, an)
    want = ref.xielu(z.double(), pq)
    # the two halves of the sum cancel somewhere below zero: the bound follows the terms
    size = want.abs() + z.double().abs() * (dtype == torch.float32)
    assert bool(((out.double().cpu() - want).abs() <= (1e-6 if dtype == torch.float32 else 4e-3) * size + 1e-7).all())
    if dtype == torch.bfloat16:
        g = gen(3)
        for M, N, K in ((300, 272, 136), (129, 16, 64), (2, 512, 512)):
            a, w = rnd(g, M, K, dtype=dtype), rnd(g, N, K, dtype=dtype, scale=0.2)
            o, st = torch.empty(M, N, dtype=dtype, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
            ops.linear(a.cuda(), w.cuda(), o, xielu=(ap, an), status=st)
            want = ref.xielu(a.double() @ w.double().T, pq)
            assert int(st) == 0
            assert bool(((o.double().cpu() - want).abs() <= 6e-3 * want.abs() + 2e-3).all())


def make_latents(dtype, r, lens, pt, seed, paged):
    """Latents of several sequences in a pool with shuffled pages (or dense): (logical latents, layout, slots per sequence)."""
    from diff_gpt_b200 import ops

    g = gen(seed)
    B, cap = len(lens), -(-max(lens) // pt) * pt
    data = rnd(g, B, cap, r, dtype=dtype)
    if not paged:
        c = data.cuda()
        return data, ops.kv_layout(c, c, page_stride=cap * r, head_stride=0, page_tokens=cap)
    per = cap // pt
    perm = torch.randperm(B * per + 3, generator=g)[: B * per].int()
    pool = torch.full((B * per + 3, pt, r), float("nan"), dtype=dtype)
    pool[perm.long()] = data.view(B * per, pt, r)
    p = pool.cuda()
    return data, ops.kv_layout(p, p, page_stride=pt * r, head_stride=0, page_tokens=pt, page_table=perm.view(B, per).contiguous().cuda(),
                               n_pages=p.shape[0])


def plain_latent_attention(q, c, gate, n_keys, window, scale):
    """q [T, H, r], c [slots, r]; query t sees keys n_keys + t - window .. n_keys + t - 1."""
    out = torch.zeros_like(q)
    for t in range(q.shape[0]):
        hi = n_keys + t
        k = c[max(0, hi - window) if window else 0 : hi]
        out[t] = torch.softmax(q[t] @ k.T * scale, dim=-1) @ k * torch.sigmoid(gate[t])[:, None]
    return out


ATTN = [  # r, H, T, window, lens (keys before and including the first new token), pt, splits, paged
    (96, 4, 1, 72, [1, 2, 71, 72, 73, 200], 16, 1, True),
    (8, 1, 1, 1, [1, 64, 65], 64, 1, True),
    (40, 3, 5, 7, [1, 6, 7, 8, 130], 8, 1, True),
    (128, 16, 2, 0, [63, 64, 65, 300], 64, 3, True),
    (256, 17, 1, 129, [128, 129, 130, 700], 32, 2, False),
    (512, 32, 1, 1000, [5, 999, 1000, 1001, 1100], 64, 5, True),
    (136, 5, 31, 40, [1, 39, 40, 41], 4, 2, False),
    (264, 20, 3, 64, [64, 190], 128, 1, True),
    (1024, 4, 2, 33, [40, 100], 16, 2, True),  # larger than the tensor-core form takes
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ATTN, ids=lambda c: f"r{c[0]}H{c[1]}T{c[2]}w{c[3]}")
def test_latent_attention(dtype, case):
    """One key per query scores far above the rest and lies on the window's edge (or just outside it), so a key too many
    or too few, or one page off, shows at full size."""
    from diff_gpt_b200 import ops

    r, H, T, window, lens, pt, splits, paged = case
    g, B = gen(r + H), len(lens)
    data, lay = make_latents(dtype, r, [n + T for n in lens], pt, r, paged)
    q, gate, scale = rnd(g, B, T, H, r, dtype=dtype), rnd(g, B, T, H, dtype=dtype), r**-0.5
    for b, n in enumerate(lens):
        for t in range(T):
            for h in range(H):
                edge = n + t - window if window else 0
                j = edge + (h % 3 - 1) if h % 3 < 2 else n + t - 1  # just outside, just inside, the newest
                if 0 <= j:
                    q[b, t, h] = (q[b, t, h].float() * 0.2 + data[b, j].float() * (12.0 / (r * scale))).to(dtype)
    out = torch.full((B * T, H * r), float("nan"), dtype=dtype, device="cuda")
    ws = torch.empty(ops.latent_attn_workspace_bytes(B * T, H, r, splits) // 4, device="cuda") if splits > 1 else None
    start = torch.zeros(B, dtype=torch.int32, device="cuda")
    n1 = torch.tensor(lens, dtype=torch.int32, device="cuda")
    impls = [0, 1] if dtype == torch.bfloat16 else [0]
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for impl in impls:
        out.fill_(float("nan"))
        ops.latent_attn(q.reshape(B * T, H * r).cuda(), lay, None, start, n1, None, out, n_seq=B, T=T, H=H, r=r, window=window,
                        scale=scale, gate=gate.reshape(B * T, H).cuda(), workspace=ws, n_splits=splits, impl=impl,
                        status=status)
        assert int(status) == 0
        want = torch.stack([plain_latent_attention(q[b].double(), data[b].double(), gate[b].double(), lens[b], window, scale) for b in range(B)])
        close(out.view(B, T, H, r), want, dtype, f32=3e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_over_two_ranges_and_a_device_step(dtype):
    """Prompt slots, a gap, then generated slots; the step counter lives on the device; the window spans the seam."""
    from diff_gpt_b200 import ops

    r, H, pt, window = 64, 6, 16, 50
    len0, start1 = [37, 16, 1, 48], 48
    B = len(len0)
    data, lay = make_latents(dtype, r, [160] * B, pt, 11, True)
    g = gen(12)
    step = torch.zeros(1, dtype=torch.int32, device="cuda")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    for s in (0, 1, 30, 49, 50, 90):
        step.fill_(s)
        q, gate = rnd(g, B, H, r, dtype=dtype, scale=2.0), rnd(g, B, H, dtype=dtype)
        out = torch.empty(B, H * r, dtype=dtype, device="cuda")
        for splits in (1, 2):
            ws = torch.empty(ops.latent_attn_workspace_bytes(B, H, r, splits) // 4, device="cuda") if splits > 1 else None
            ops.latent_attn(q.reshape(B, -1).cuda(), lay, i32(len0), i32([start1] * B), i32([1] * B), step, out, n_seq=B, T=1, H=H, r=r,
                            window=window, scale=0.3, gate=gate.cuda(), workspace=ws, n_splits=splits)
            for b in range(B):
                keys = torch.cat([data[b, : len0[b]], data[b, start1 : start1 + 1 + s]]).double()
                want = plain_latent_attention(q[b : b + 1].double(), keys, gate[b : b + 1].double(), len0[b] + 1 + s, window, 0.3)
                close(out[b].view(1, H, r), want, dtype, f32=3e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,T,pt", [(96, 1, 16), (20, 7, 4), (512, 3, 64), (8, 40, 8)])
def test_latent_append(dtype, rank, T, pt):
    from diff_gpt_b200 import ops

    g, B, r = gen(rank), 3, -(-rank // 8) * 8
    first = [0, 5, pt + 3]
    cap = -(-(max(first) + T + 2) // pt) * pt
    data, lay = make_latents(dtype, r, [cap] * B, pt, 1, True)
    x, w = rnd(g, B * T, rank + 6, dtype=dtype, scale=0.02), rnd(g, rank)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    step = torch.full((1,), 2, dtype=torch.int32, device="cuda")
    flat = torch.full((B * T, r), float("nan"), dtype=dtype, device="cuda")
    ops.latent_append(x.cuda()[:, :rank], w.cuda(), 1e-3, lay, torch.tensor(first, dtype=torch.int32, device="cuda"), step, n_seq=B, T=T,
                      r=r, flat=flat, status=status)
    want = ref.rms_norm(x[:, :rank].double(), w.double(), 1e-3)
    close(flat[:, :rank], want, dtype, bf16=5e-3)
    assert bool((flat[:, rank:] == 0).all()) and int(status) == 0
    pool, table = lay._keep[0].cpu(), lay._keep[2].cpu()
    for b in range(B):
        for s in range(cap):
            row = pool[int(table[b, s // pt]), s % pt]
            t = s - first[b] - 2
            assert torch.equal(row, flat[b * T + t].cpu() if 0 <= t < T else data[b, s])
    step.fill_(cap)  # every slot out of range: reported, nothing written
    before = lay._keep[0].clone()
    ops.latent_append(x.cuda()[:, :rank], w.cuda(), 1e-3, lay, torch.tensor(first, dtype=torch.int32, device="cuda"), step, n_seq=B, T=T,
                      r=r, status=status)
    assert int(status) == 1 and torch.equal(torch.nan_to_num(before), torch.nan_to_num(lay._keep[0]))


WINDOW = [  # D, H, B, Tq, context, window
    (64, 4, 1, 300, 0, 72), (64, 2, 2, 128, 71, 72), (32, 3, 1, 33, 200, 150), (128, 2, 1, 1500, 0, 129), (64, 2, 1, 700, 500, 501),
    (128, 1, 2, 1100, 0, 1), (32, 2, 1, 1030, 64, 128), (64, 1, 1, 1200, 0, 0), (64, 3, 1, 1300, 0, 127), (64, 1, 1, 1290, 0, 128),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", WINDOW, ids=lambda c: f"D{c[0]}T{c[3]}c{c[4]}w{c[5]}")
def test_windowed_attention(dtype, case):
    """Keys and values interleaved per token; every query has one key that stands out, just inside or just outside the
    window or in the middle of it."""
    from diff_gpt_b200 import ops

    D, H, B, Tq, ctx, window = case
    g, n_keys = gen(D + Tq), ctx + Tq
    kv = rnd(g, B, n_keys, 2, H, D, dtype=dtype)
    wide = rnd(g, B, Tq, H * D + 24, dtype=dtype, scale=0.2)
    gate = rnd(g, B * Tq, H + 3, dtype=dtype)
    q = wide[..., : H * D].view(B, Tq, H, D)
    pos = torch.arange(ctx, n_keys)
    span = window if window else n_keys
    for h in range(H):
        for kind in range(3):
            sel = torch.arange(Tq) % 3 == kind
            j = pos - (span, span - 1, span // 2)[kind]
            ok = sel & (j >= 0)
            q[:, ok, h] = (q[:, ok, h].float() + kv[:, j[ok], 0, h].float() * (9.0 / D**0.5)).to(dtype)
    seen = ref.window_mask(n_keys, span)[ctx:]
    s = torch.einsum("bihd,bjhd->bhij", q.double(), kv[:, :, 0].double()) * (0.9 * D**-0.5)
    p = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1)
    want = torch.einsum("bhij,bjhd->bihd", p, kv[:, :, 1].double()) * torch.sigmoid(gate[:, :H].double()).view(B, Tq, H, 1)
    flat = kv.reshape(B * n_keys, 2 * H * D).cuda()
    qd, gd = wide.reshape(B * Tq, -1).cuda()[:, : H * D], gate.cuda()[:, :H]
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    for impl in ([0, 1, 2, 3] if dtype == torch.bfloat16 else [0]):
        o = torch.full((B * Tq, H * D), float("nan"), dtype=dtype, device="cuda")
        ops.fmha_window(qd, flat[:, : H * D], flat[:, H * D :], o, B=B, H=H, D=D, n_keys=n_keys, q_offset=ctx, window=window,
                        scale=0.9 * D**-0.5, gate=gd, impl=impl, status=st)
        assert int(st) == 0
        close(o.view(B, Tq, H, D), want, dtype, f32=3e-5)
    # the one layout rule: strides are multiples of 8 elements
    from diff_gpt_b200._lib import DgptError

    bad = torch.empty(Tq, H * D + 4, dtype=dtype, device="cuda")[:, : H * D]
    with pytest.raises(DgptError, match="multiples of 8"):
        ops.fmha_window(bad, flat[: n_keys, : H * D], flat[: n_keys, H * D :], bad, B=1, H=H, D=D, n_keys=n_keys, q_offset=ctx,
                        window=window, scale=1.0)
