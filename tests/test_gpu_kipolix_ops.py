"""Each kernel of the Kipolix path alone, against the plain implementation in float64."""

import math

import pytest
import torch

from oracle import ref_kipolix as ref

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


def table(base, dims, n):
    from diff_gpt_b200.model.rope import rotation_table

    return rotation_table(base, dims, n, "cuda")


# ---- embedding and streams ---------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,S", [(5, 1), (52, 5), (256, 4), (2048, 2), (4100, 3)])
def test_embedding_with_bigrams_in_portions(dtype, C, S):
    """Two sequences in portions: the token before a portion comes from the state, a first token has a row of its own."""
    from diff_gpt_b200 import ops

    g, B, T, V, buckets, mp, mc = gen(C), 2, 40, 19, 23, 101, 7
    emb, big, a, w = rnd(g, V, C, dtype=dtype), rnd(g, buckets + 1, C, dtype=dtype), rnd(g, S), rnd(g, C)
    ids = torch.randint(0, V, (B, T), generator=g)
    ids[1, :3] = 0  # token 0 is not "none"
    want_e = torch.stack([ref.embed(ids[b], emb.double(), big.double(), mp, mc) for b in range(B)])
    want_h = ref.unit_rms(a.double().sum() * want_e, 1e-3) * w.double()
    for cuts in ([T], [1, 1, 2, 1, 30, 5]):
        prev = [torch.full((1, B), -1, dtype=torch.int32, device="cuda") for _ in range(2)]
        at = 0
        for n in cuts:
            part = ids[:, at : at + n].reshape(-1).int().cuda()
            e, h = torch.empty(B * n, C, device="cuda"), torch.empty(B * n, C, dtype=dtype, device="cuda")
            ops.embed_streams(part, prev[0], prev[0] if n == 1 else prev[1], emb.cuda(), big.cuda(), mp, mc, a.cuda(), w.cuda(), 1e-3, e, h,
                              n_seq=B, T=n)
            if n > 1:
                prev.reverse()
            close(e.view(B, n, C), want_e[:, at : at + n], torch.float32, f32=1e-6)
            close(h.view(B, n, C), want_h[:, at : at + n], dtype, bf16=5e-3)
            at += n
        assert prev[0].cpu().tolist() == [ids[:, -1].tolist()]


def test_bigram_rows_of_large_multipliers():
    """The product of token and multiplier passes 32 bits."""
    from diff_gpt_b200 import ops

    V, buckets, mp, mc = 50000, 9973, 2**31 - 1, 2**31 - 19
    ids = torch.tensor([49999, 49998, 3, 49999])
    emb, big = torch.zeros(V, 4), torch.arange(buckets + 1.0)[:, None].expand(-1, 4).contiguous()
    e, h = torch.empty(4, 4, device="cuda"), torch.empty(4, 4, device="cuda")
    ops.embed_streams(ids.int().cuda(), None, None, emb.cuda(), big.cuda(), mp, mc, torch.ones(2).cuda(), torch.ones(4).cuda(), 1e-6, e, h,
                      n_seq=1, T=4)
    assert e[:, 0].cpu().tolist() == ref.bigram_rows(ids, buckets, mp, mc).tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,S", [(7, 3), (52, 1), (256, 4), (320, 2), (2048, 5), (1024, 8), (64, 16), (8200, 4)])
def test_streams(dtype, C, S):
    from diff_gpt_b200 import ops

    g, n = gen(C + S), 9
    x, y, mix, out, a, w = rnd(g, S, n, C), rnd(g, n, C, dtype=dtype), rnd(g, S, S), rnd(g, S), rnd(g, S), rnd(g, C)
    dev = [t.cuda() for t in (y, mix, out)]

    def check(xd, x64, new):
        want = ref.stream_out(x64, mix.double(), out.double(), y.double())
        h = torch.empty(n, C, dtype=dtype, device="cuda")
        ops.streams_step(xd, *dev, new, a.cuda(), w.cuda(), 1e-2, h)
        close(new, want, torch.float32)
        close(h, ref.unit_rms(ref.stream_in(want, a.double()), 1e-2) * w.double(), dtype, f32=5e-5, bf16=5e-3)

    check(x.cuda(), x.double(), torch.empty(S, n, C, device="cuda"))
    xd = x.cuda()
    check(xd, x.double(), xd)  # in place
    check(x[0].cuda(), x[:1].double().expand(S, -1, -1), torch.empty(S, n, C, device="cuda"))  # all streams equal
    for rows in (None, torch.tensor([8, 0, 3], dtype=torch.int32)):
        want = ref.unit_rms(ref.stream_out(x.double(), mix.double(), out.double(), y.double()).sum(0), 1e-2) * w.double()
        h = torch.empty(n if rows is None else 3, C, dtype=dtype, device="cuda")
        ops.streams_final(x.cuda(), *dev, w.cuda(), 1e-2, h, rows=None if rows is None else rows.cuda())
        close(h, want if rows is None else want[rows.long()], dtype, f32=5e-5, bf16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_silu_gate_alone_and_in_the_gemm(dtype):
    from diff_gpt_b200 import ops

    g = gen(3)
    x = rnd(g, 33, 2 * 40, dtype=dtype, scale=4.0)
    x[0, :4] = torch.tensor([-80.0, 3.0, 80.0, -2.0])
    out = torch.empty(33, 40, dtype=dtype, device="cuda")
    ops.silu_mul(x.cuda(), out)
    xd = x.double()
    close(out, ref.silu(xd[:, 0::2]) * xd[:, 1::2], dtype, bf16=5e-3)
    odd = torch.empty(3, 5, dtype=dtype, device="cuda")
    ops.silu_mul(x[:3, :10].contiguous().cuda(), odd)
    close(odd, (ref.silu(xd[:, 0::2]) * xd[:, 1::2])[:3, :5], dtype, bf16=5e-3)
    if dtype == torch.bfloat16:
        for M, K, F in ((1, 64, 8), (300, 72, 72), (129, 256, 200), (700, 512, 640)):
            a, w = rnd(g, M, K, dtype=dtype), rnd(g, 2 * F, K, dtype=dtype, scale=K**-0.5)
            out = torch.empty(M, F, dtype=dtype, device="cuda")
            st = torch.zeros(1, dtype=torch.int32, device="cuda")
            ops.linear(a.cuda(), w.cuda(), out, silu_gate=True, status=st)
            p = a.double() @ w.double().T
            close(out, ref.silu(p[:, 0::2]) * p[:, 1::2], dtype, bf16=6e-3)
            assert int(st.item()) == 0


# ---- projection norm, rotation, append -----------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,D,rot,base", [
    (6, 2, 12, 20, 24, 6, 500.0), (8, 2, 64, 64, 64, 64, 1e4), (3, 1, 100, 96, 128, 50, 1e6), (1, 1, 8, 8, 8, 2, 10.0), (40, 8, 128, 128, 128, 96, 5e5),
])
def test_projection_norm_rotation_and_append(dtype, H, G, dim, vdim, D, rot, base):
    """Norm over all heads at once, interleaved pairs on the leading dimensions, rows through a page table and in a dense
    run, positions that differ from slots, padding columns that do not count."""
    for T in (37, 640):  # a CTA per token, a warp per token
        check_append(dtype, H, G, dim, vdim, D, rot, base, T)


def check_append(dtype, H, G, dim, vdim, D, rot, base, T):
    from diff_gpt_b200 import ops

    g, B, pt, eps, pos0, slot0 = gen(H * D), 2, 16, 1e-4, [300, 3], [5, 11]
    q, k, v = rnd(g, B, T, H, dim, dtype=dtype), rnd(g, B, T, G, dim, dtype=dtype), rnd(g, B, T, G, vdim, dtype=dtype)
    qw, kw = rnd(g, H, dim), rnd(g, G, dim)

    def pad(t, to):
        return torch.nn.functional.pad(t, (0, to - t.shape[-1])).flatten(-2)

    x = torch.cat([pad(q, D), pad(k, D), pad(v, D), torch.full((B, T, 8), 9.0).to(dtype)], dim=-1).reshape(B * T, -1).cuda()
    W = 2 * G * D
    per = -(-(T + 11) // pt)
    n_pages = 2 * per + 1
    perm = torch.randperm(n_pages, generator=g).int()[: 2 * per].view(2, per)
    pool = torch.full((n_pages, pt, W + 8), float("nan"), dtype=dtype, device="cuda")
    want_q = torch.stack([ref.rotate_pairs((ref.unit_rms(q[b].double().flatten(1), eps) * qw.double().flatten()).view(T, H, dim), rot, base, pos0[b])
                          for b in range(B)])
    want_k = torch.stack([ref.rotate_pairs((ref.unit_rms(k[b].double().flatten(1), eps) * kw.double().flatten()).view(T, G, dim), rot, base, pos0[b])
                          for b in range(B)])
    step = torch.tensor([2], dtype=torch.int32, device="cuda")
    tab = table(base, rot, 1024)
    for paged in (True, False):
        dense = torch.full((B, T + 20, W + 8), float("nan"), dtype=dtype, device="cuda")
        lay = (ops.kv_layout(pool, pool, pool.stride(0), 0, pt, perm.cuda(), n_pages) if paged
               else ops.kv_layout(dense, dense, dense.stride(0), 0, T + 20))
        out = torch.empty(B * T, H * D, dtype=dtype, device="cuda")
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.proj_norm_rope_append(
            x, pad(qw, D).cuda(), pad(kw, D).cuda(), H * dim, G * dim, eps, tab, out, lay, W + 8,
            torch.tensor([p - 2 for p in pos0], dtype=torch.int32).cuda(), torch.tensor([s - 2 for s in slot0], dtype=torch.int32).cuda(), step,
            n_seq=B, T=T, H=H, G=G, D=D, Dv=D, status=st,
        )
        assert int(st.item()) == 0
        got = out.view(B, T, H, D)
        close(got[..., :dim], want_q, dtype, bf16=6e-3)
        assert bool((got[..., dim:] == 0).all())
        for b in range(B):
            s = slot0[b] + torch.arange(T)
            row = (pool[perm[b].long()[s // pt].cuda(), (s % pt).cuda()] if paged else dense[b, s.cuda()]).cpu()
            kr, vr = row[:, : G * D].view(T, G, D), row[:, G * D : W].view(T, G, D)
            close(kr[..., :dim], want_k[b], dtype, f32=5e-5, bf16=8e-3)
            assert torch.equal(vr[..., :vdim], v[b]) and bool((kr[..., dim:] == 0).all()) and bool((vr[..., vdim:] == 0).all())
    ops.proj_norm_rope_append(x, pad(qw, D).cuda(), pad(kw, D).cuda(), H * dim, G * dim, eps, tab, out, lay, W + 8,
                              torch.tensor([0, 1000], dtype=torch.int32).cuda(), torch.tensor([T, 0], dtype=torch.int32).cuda(), None,
                              n_seq=B, T=T, H=H, G=G, D=D, Dv=D, status=st)
    assert int(st.item()) == 1  # a slot past the run, a position past the table: reported, nothing written there


# ---- attention over cached rows --------------------------------------------------------------
def rows_cache(g, B, n, G, dk, dv, pt, dtype, extra=3, paged=True, prompt=None, pad_cols=0):
    """Keys and values of B sequences, n tokens each, written into a cache of rows; NaN wherever nothing was written.
    prompt: tokens that lie in the first run of slots (the rest starts on a page of its own)."""
    k, v = rnd(g, B, n, G, dk, dtype=dtype), rnd(g, B, n, G, dv, dtype=dtype)
    W = G * (dk + dv) + pad_cols
    p0 = n if prompt is None else prompt
    start1 = -(-p0 // pt) * pt if prompt is not None else 0
    cap = (start1 + (n - p0) if prompt is not None else n) + extra
    pages = -(-cap // pt)
    store = torch.full((B * pages + 2, pt, W), float("nan"), dtype=dtype)
    perm = torch.randperm(B * pages + 2, generator=g)[: B * pages].view(B, pages)
    for b in range(B):
        for t in range(n):
            s = t if prompt is None or t < p0 else start1 + t - p0
            store[perm[b, s // pt], s % pt, : G * dk] = k[b, t].flatten()
            store[perm[b, s // pt], s % pt, G * dk : G * (dk + dv)] = v[b, t].flatten()
            store[perm[b, s // pt], s % pt, G * (dk + dv) :] = 7.0  # columns of a written row are finite
    if not paged:  # the same as one dense run per sequence
        store = torch.stack([store[perm[b]].reshape(pages * pt, W) for b in range(B)])
        return k, v, store.cuda(), None, start1, W
    return k, v, store.cuda(), perm.int().cuda(), start1, W


def plain(q, k, v, first_query, window, keep, scale):
    """q [Tq, H, dk] at logical positions first_query + i; k, v [n, G, *]."""
    n = k.shape[0]
    seen = ref.visible(n, window if window else 10**9, keep)[first_query : first_query + q.shape[0]]
    return ref.softmax_attention(q.double(), k.double(), v.double(), seen, scale)


@pytest.mark.parametrize("dtype,impl", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2)])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 4, 32, 32), (8, 2, 64, 64), (6, 1, 128, 128), (18, 2, 96, 64), (16, 1, 64, 136), (40, 2, 128, 40), (5, 1, 160, 24)])
def test_grouped_attention_over_cached_rows(dtype, impl, H, G, dk, dv):
    """Rows at page borders, prompts in one run and the rest in another, first keys that stay visible in either run, a
    window's first key in either run, several queries per sequence, splits; what nobody wrote is NaN."""
    from diff_gpt_b200 import ops

    g = gen(H + dk)
    scale = 1.3 / math.sqrt(dk)
    cases = [  # n, prompt, T, window, keep, pt, splits
        (300, 130, 1, 64, 5, 16, 1), (300, 130, 1, 200, 5, 16, 3), (300, 7, 1, 60, 20, 16, 1), (300, 290, 4, 129, 300, 64, 1),
        (260, None, 5, 33, 0, 64, 2), (140, None, 1, 0, 9, 8, 1), (129, None, 2, 128, 1, 128, 1), (1, None, 1, 4, 6, 16, 1), (20, 19, 1, 1, 2, 8, 1),
        (700, 513, 3, 256, 130, 32, 5),
    ]
    for n, prompt, T, window, keep, pt, splits in cases:
        B = 3
        for paged in (True, False) if prompt is None else (True,):
            k, v, store, perm, start1, W = rows_cache(g, B, n, G, dk, dv, pt, dtype, paged=paged, prompt=prompt, pad_cols=8)
            q = rnd(g, B, T, H, dk, dtype=dtype)
            lay = (ops.kv_layout(store, store, store.stride(0), 0, pt, perm, store.shape[0]) if paged
                   else ops.kv_layout(store, store, store.stride(0), 0, store.shape[1]))
            p0 = 0 if prompt is None else prompt
            i32 = lambda x: torch.full((B,), x, dtype=torch.int32, device="cuda")  # noqa: E731
            out = torch.full((B * T, H * dv), float("nan"), dtype=dtype, device="cuda")
            ws = torch.empty(max(4, ops.latent_attn_workspace_bytes(B * T, H, dv, splits) // 4), device="cuda") if splits > 1 else None
            st = torch.zeros(1, dtype=torch.int32, device="cuda")
            step = torch.tensor([n - p0 - T], dtype=torch.int32, device="cuda")
            ops.grouped_attn(
                q.reshape(B * T, -1).cuda(), lay, None if prompt is None else i32(p0), i32(start1), i32(1), step, out, row_width=W,
                v_col=G * dk, n_seq=B, T=T, H=H, G=G, dk=dk, dv=dv, window=window, keep_first=keep, scale=scale, workspace=ws,
                n_splits=splits, impl=impl, status=st,
            )
            assert int(st.item()) == 0
            want = torch.stack([plain(q[b], k[b], v[b], n - T, window, keep, scale) for b in range(B)])
            close(out.view(B, T, H, dv), want, dtype, bf16=1.5e-2)


@pytest.mark.parametrize("dtype,impl", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2), (torch.bfloat16, 3)])
@pytest.mark.parametrize("H,G,D", [(4, 2, 32), (8, 2, 64), (3, 1, 128)])
def test_prefill_attention_with_groups_window_and_kept_keys(dtype, impl, H, G, D):
    """Key tiles of kept keys in front of the window's, gaps of several tiles between them, portions behind cached keys,
    dense runs and pages."""
    from diff_gpt_b200 import ops

    g = gen(H * D)
    cases = [  # Tq, context, window, keep, pt (None: dense)
        (300, 0, 64, 5, None), (700, 0, 100, 130, 64), (150, 600, 129, 3, None), (33, 1000, 128, 257, 16), (260, 40, 1, 1, None),
        (128, 512, 256, 128, 128), (400, 0, 50, 0, 32), (200, 100, 0, 7, None), (90, 37, 10**6, 6, 8), (1200, 0, 700, 9, 64),
    ]
    for Tq, context, window, keep, pt in cases:
        B, n = 2, Tq + context
        k, v, store, perm, _, W = rows_cache(g, B, n, G, D, D, pt or 64, dtype, paged=pt is not None)
        q = rnd(g, B, Tq, H, D, dtype=dtype)
        if pt is not None:
            lay = ops.kv_layout(store, store[:, :, G * D :], store.stride(0), D, pt, perm, store.shape[0])
        else:
            lay = ops.kv_layout(store, store[:, :, G * D :], store.stride(0), D, store.shape[1])
        out = torch.full((B * Tq, H * D), float("nan"), dtype=dtype, device="cuda")
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.fmha_grouped(q.reshape(B * Tq, -1).cuda(), lay, out, token_stride=W, n_keys=n, B=B, H=H, G=G, D=D, q_offset=context, window=window,
                         keep_first=keep, scale=0.2, impl=impl, status=st)
        assert int(st.item()) == 0
        want = torch.stack([plain(q[b], k[b], v[b], context, window, keep if window else 0, 0.2) for b in range(B)])
        close(out.view(B, Tq, H, D), want, dtype, bf16=1.5e-2)


@pytest.mark.parametrize("prefill", [True, False])
def test_single_keys_that_carry_all_weight(prefill):
    """One key per query stands out by far: just inside and just outside the window, the last kept key and the one after it,
    page borders.  The result is that key's value, or is untouched by it."""
    from diff_gpt_b200 import ops

    g, H, G, D, n, window, keep, pt = gen(5), 4, 2, 64, 420, 100, 6, 32
    for dtype in DTYPES:
        k = torch.zeros(1, n, G, D)
        v = rnd(g, 1, n, G, D, dtype=dtype).float()
        q = torch.zeros(1, n, H, D)
        target = {}
        for x, i in enumerate(range(150, 420, 9)):
            j = [i - window + 1, i - window, keep - 1, keep, i - (i % pt), i - (i % pt) - 1, 0, i][x % 8]
            target[i] = j
            q[0, i, :, x] = 40.0
            k[0, j, :, x] = 40.0
        store = torch.cat([k.flatten(2), v.flatten(2)], -1).to(dtype).cuda().view(1, n, -1)
        pages = -(-n // pt)
        pool = torch.nn.functional.pad(store[0], (0, 0, 0, pages * pt - n)).view(pages, pt, -1)
        perm = torch.randperm(pages, generator=g)
        shuffled = torch.empty_like(pool)
        shuffled[perm.cuda()] = pool
        tab = perm.int().view(1, -1).cuda()
        out = torch.empty(n, H * D, dtype=dtype, device="cuda")
        qd = q.reshape(n, -1).to(dtype).cuda()
        if prefill:
            lay = ops.kv_layout(shuffled, shuffled[:, :, G * D :], shuffled.stride(0), D, pt, tab, pages)
            ops.fmha_grouped(qd, lay, out, token_stride=2 * G * D, n_keys=n, B=1, H=H, G=G, D=D, q_offset=0, window=window, keep_first=keep, scale=1.0)
        else:
            lay = ops.kv_layout(shuffled, shuffled, shuffled.stride(0), 0, pt, tab, pages)
            one = torch.ones(1, dtype=torch.int32, device="cuda")
            ops.grouped_attn(qd, lay, None, torch.zeros_like(one), one, None, out, row_width=2 * G * D, v_col=G * D, n_seq=1, T=n, H=H, G=G, dk=D,
                             dv=D, window=window, keep_first=keep, scale=1.0)
        got = out.float().cpu().view(n, H, D)
        for i, j in target.items():
            seen = i - j < window or j < keep
            val = v[0, j].repeat_interleave(H // G, 0)
            if seen:
                assert (got[i] - val).abs().max() < 1e-2, (i, j)
            else:
                assert (got[i] - val).abs().max() > 0.3, (i, j)


# ---- retention -----------------------------------------------------------------------------
def run_retention(q, k, v, gate, decay, rot, base, eps, cuts, dtype, impl, pos0, state=None):
    """(y, state) of B sequences through the kernels in portions."""
    from diff_gpt_b200 import ops

    B, T, H, d = q.shape
    e = v.shape[-1]
    parts = [t.flatten(2) for t in (q, k, v, gate)]
    parts = [torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)) for t in parts]
    cols, at = [], 0
    for t in parts:
        cols.append(at)
        at += t.shape[-1]
    x = torch.cat(parts, -1).to(dtype).cuda()
    tab = table(base, rot, 2048)
    bufs = [torch.zeros(B, H, d, e, device="cuda") if state is None else state.clone(), torch.full((B, H, d, e), float("nan"), device="cuda")]
    out, at = [], 0
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    dec = torch.tensor(decay, device="cuda")
    for n in cuts:
        y = torch.full((B * n, H * e), float("nan"), dtype=dtype, device="cuda")
        ws = torch.empty(max(4, ops.retention_workspace_bytes(B, n, H, d, e) // 4), device="cuda")
        ops.retention(
            x[:, at : at + n].reshape(B * n, -1).contiguous(), tuple(cols), tab, torch.tensor([p + at for p in pos0], dtype=torch.int32).cuda(), None,
            dec, min(decay), d**-0.5, bufs[0], bufs[0] if n == 1 else bufs[1], eps, y, ws, n_seq=B, T=n, dim=d, vdim=e,
            impl=impl if n > 1 or impl == 2 else 0, status=st,
        )
        if n > 1:
            bufs.reverse()
        out.append(y.view(B, n, H * e))
        at += n
    assert at == T and int(st.item()) == 0
    return torch.cat(out, 1), bufs[0]


def plain_retention(q, k, v, gate, decay, rot, base, eps, pos0, state=None):
    ys, ss = [], []
    d = q.shape[-1]
    for b in range(q.shape[0]):
        qr = ref.rotate_half(q[b].double(), rot, base, pos0[b])
        kr = ref.rotate_half(k[b].double(), rot, base, pos0[b]) * d**-0.5
        o, S = ref.retention(qr, kr, v[b].double(), torch.tensor(decay).double(), None if state is None else state[b].double().cpu())
        ys.append((ref.unit_rms(o, eps) * ref.silu(gate[b].double())).flatten(1))
        ss.append(S)
    return torch.stack(ys), torch.stack(ss)


RETENTIONS = [  # H, dim, vdim, decay, rot
    (3, 20, 12, (0.9, 0.99, 0.3), 14), (2, 64, 64, (0.96875, 0.9995), 64), (4, 128, 128, (0.97, 0.99, 0.998, 1.0), 128), (2, 96, 40, (0.75, 0.95), 32),
    (1, 32, 200, (0.99,), 32), (2, 136, 24, (0.9, 0.98), 136), (2, 8, 8, (0.125, 0.6), 2), (3, 72, 80, (0.98, 0.9, 0.99), 36), (1, 3, 5, (0.0,), 2),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,vdim,decay,rot", RETENTIONS)
def test_retention_prompts_portions_and_single_tokens(dtype, H, dim, vdim, decay, rot):
    """The same tokens whole, one by one and in portions (around the chunk's 128 and the sizes where kernels change), from
    zero and from a given state; the state left behind is the recurrence's."""
    g, B, T, base, eps, pos0 = gen(dim + vdim), 2, 290, 3000.0, 1e-3, [0, 1000]
    q, k, v, gate = (rnd(g, B, T, H, n, dtype=dtype).float() for n in (dim, dim, vdim, vdim))
    want, S = plain_retention(q, k, v, gate, decay, rot, base, eps, pos0)
    chunked_ok = dtype == torch.bfloat16 and dim <= 128 and dim % 8 == 0 and vdim % 8 == 0 and min(decay) >= 0.0625
    plans = [([T], 0), ([1] * 40 + [250], 0), ([2, 128, 3, 15, 16, 126], 0), ([T], 1), ([129, 161], 1)]
    if chunked_ok:
        plans += [([T], 2), ([2, 1, 127, 128, 32], 2)]
    for cuts, impl in plans:
        y, state = run_retention(q, k, v, gate, decay, rot, base, eps, cuts, dtype, impl, pos0)
        close(y, want, dtype, f32=1e-4, bf16=1e-2)
        close(state, S, torch.float32, f32=2e-4 if impl == 2 or (impl == 0 and chunked_ok) else 2e-5)
    s0 = rnd(g, B, H, dim, vdim, scale=3.0).cuda()
    want, S = plain_retention(q, k, v, gate, decay, rot, base, eps, pos0, s0)
    for cuts in ([T], [1, 1, 288]):
        y, state = run_retention(q, k, v, gate, decay, rot, base, eps, cuts, dtype, 0, pos0, s0)
        close(y, want, dtype, f32=1e-4, bf16=1e-2)
        close(state, S, torch.float32, f32=2e-4)


def test_retention_segments_of_a_long_sequence():
    """Few heads: the tokens are cut into segments that run side by side; sharp keys far back, at chunk and segment borders,
    come through with the decay of their distance."""
    H, d, e, T, base = 2, 64, 48, 6000, 1e4
    decay = (0.9995, 1.0)
    g = gen(9)
    q, k, v, gate = (rnd(g, 1, T, H, n, scale=s, dtype=torch.bfloat16).float() for n, s in ((d, 0.05), (d, 0.05), (e, 1.0), (e, 1.0)))
    for j in (0, 1, 127, 128, 255, 256, 2047, 2048, 5000, 5887, 5888):
        k[0, j] *= 32.0
    want, S = plain_retention(q, k, v, gate, decay, d, base, 1e-6, [0])
    from diff_gpt_b200 import ops
    from diff_gpt_b200.model.rope import rotation_table

    x = torch.cat([t.flatten(2) for t in (q, k, v, gate)], -1)[0].to(torch.bfloat16).cuda()
    cols = (0, H * d, 2 * H * d, 2 * H * d + H * e)
    y = torch.empty(T, H * e, dtype=torch.bfloat16, device="cuda")
    ws = torch.empty(ops.retention_workspace_bytes(1, T, H, d, e) // 4, device="cuda")
    assert ws.numel() > T * H * e  # segments are in use
    out, st = torch.empty(1, H, d, e, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.retention(x, cols, rotation_table(base, d, 8192, "cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"), None,
                  torch.tensor(decay, device="cuda"), min(decay), d**-0.5, None, out, 1e-6, y, ws, n_seq=1, T=T, dim=d, vdim=e, impl=2, status=st)
    assert int(st.item()) == 0
    close(out, S, torch.float32, f32=2e-4)
    close(y, want[0], torch.bfloat16, bf16=1e-2)


def test_refusals():
    from diff_gpt_b200 import ops
    from diff_gpt_b200._lib import DgptError

    x = torch.zeros(4, 64, dtype=torch.bfloat16, device="cuda")
    one, f = torch.ones(1, dtype=torch.int32, device="cuda"), torch.zeros(64, device="cuda")
    lay = ops.kv_layout(x, x, 64, 0, 4)
    kw = dict(n_seq=1, T=4, H=2, G=1, dk=16, dv=16, keep_first=0, scale=1.0)
    with pytest.raises(DgptError, match="cache row"):
        ops.grouped_attn(x[:, :32], lay, None, one, one, None, x[:, 32:], row_width=24, v_col=16, window=0, **kw)
    with pytest.raises(DgptError, match="bad sizes"):
        ops.grouped_attn(x[:, :32], lay, None, one, one, None, x[:, 32:], row_width=32, v_col=16, window=-1, **kw)
    S = torch.zeros(1, 1, 16, 16, device="cuda")
    with pytest.raises(DgptError, match="in place"):
        ops.retention(x, (0, 16, 32, 48), torch.zeros(8, 8, 2, device="cuda"), one, None, f[:1], 0.5, 1.0, S, S, 1e-6, x[:, :16], f, n_seq=1, T=4,
                      dim=16, vdim=16)
    with pytest.raises(DgptError, match="workspace"):
        ops.retention(x, (0, 16, 32, 48), torch.zeros(8, 8, 2, device="cuda"), one, None, f[:1], 0.5, 1.0, None, S, 1e-6, x[:, :16], f[:8], n_seq=1,
                      T=4, dim=16, vdim=16)
    with pytest.raises(DgptError, match="chunked form covers"):
        ops.retention(x.float(), (0, 16, 32, 48), torch.zeros(8, 8, 2, device="cuda"), one, None, f[:1], 0.5, 1.0, None, S, 1e-6,
                      x.float()[:, :16].contiguous(), f, n_seq=1, T=4, dim=16, vdim=16, impl=2)
