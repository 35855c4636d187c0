"""Pesorax on the GPU: every mechanism alone and whole models against the plain implementation in ``pesorax_ref``."""
import pytest
import torch

import pesorax_ref as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.04}


def rel(got, want):
    """RMS of the difference over the spread of the wanted values."""
    got, want = got.detach().cpu().double(), want.double()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()).item()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def pages_of(lens, extra=3):
    """A shuffled page table for sequences of these lengths, and the number of pages."""
    need = [(n + 15) // 16 for n in lens]
    perm = torch.randperm(sum(need) + extra, generator=torch.Generator().manual_seed(5)).tolist()
    table = torch.zeros(len(lens), max(need), dtype=torch.int32)
    for b, n in enumerate(need):
        for j in range(n):
            table[b, j] = perm.pop()
    return table, sum(need) + extra


def slots_of(table, b, n):
    return (table[b, torch.arange(n) // 16] * 16 + torch.arange(n) % 16).long()


# ---------------------------------------------------------------- norm and products
def test_dynamic_tanh():
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(0)
    for T, D, ld in ((3, 72, 72), (5, 100, 104), (4, 93, 96), (2, 2048, 2048), (300, 260, 264), (1, 9000, 9000)):
        x, w, b, alpha = torch.randn(T, D, generator=g) * 3, torch.randn(D, generator=g), torch.randn(D, generator=g), torch.tensor([0.7])
        emb, ids = torch.randn(11, D, generator=g).bfloat16(), torch.randint(0, 11, (T,), generator=g).to(torch.int32)
        W = {"n": w.double(), "n.b": b.double(), "n.alpha": alpha.double()}
        for joins in (False, True):
            want_x = x.double() + (emb[ids.long()].double() if joins else 0)
            want = R.dyt(want_x, W, "n")
            xd, side = x.to(DEV), torch.ones(64, device=DEV)
            kw = dict(ids=ids.to(DEV), emb=emb.to(DEV)) if joins else {}
            hf = torch.full((T, ld), 7.0, device=DEV)
            ops.norm_dyt(xd, alpha.to(DEV), w.to(DEV), b.to(DEV), hf=hf, zero=side, **kw)
            assert rel(xd, want_x) < 1e-6 and rel(hf[:, :D], want) < 1e-6 and not hf[:, D:].any() and not side.any()
            hb = torch.full((T, ld), 7.0, dtype=torch.bfloat16, device=DEV)
            ops.norm_dyt(xd, alpha.to(DEV), w.to(DEV), b.to(DEV), hb=hb)
            assert rel(hb[:, :D].float(), want) < 4e-3 and not hb[:, D:].any()


def test_products_with_gelu_and_scaled_residual():
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(4)
    for M, N, K in ((1, 40, 72), (3, 136, 104), (70, 200, 136), (9, 64, 64), (130, 328, 72), (2, 256, 2048)):
        a, w, x = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g).bfloat16() * K ** -0.5, torch.randn(M, N, generator=g)
        eye = torch.eye(N, dtype=torch.float64)
        want = R.gelu_ff(a.double(), {"up": w.double(), "down": eye}, "")
        want_x = x.double() + 0.3 * (a.double() @ w.double().T)
        ad, wd, st = a.to(DEV), w.to(DEV), i32(0)
        out, xd = torch.empty(M, N, device=DEV), x.to(DEV)
        ops.gemm_f32(ad, wd, out, act=2)
        ops.gemm_f32(ad, wd, xd, alpha=0.3, accumulate=True)
        assert rel(out, want) < 1e-6 and rel(xd, want_x) < 1e-6
        if M <= 8:
            xd = x.to(DEV)
            ops.matvec(ops.WT_BF16, wd, None, N, K, M, xf=ad, epi=ops.EPI_GELU_ERF, y=out, ldy=N)
            ops.matvec(ops.WT_BF16, wd, None, N, K, M, xf=ad, epi=ops.EPI_RESID, resid=xd, y=xd, ldy=N, alpha=0.3)
            assert rel(out, want) < 2e-6 and rel(xd, want_x) < 1e-6
        a16 = a.bfloat16()
        ob, oh, xd = torch.empty(M, N, dtype=torch.bfloat16, device=DEV), torch.empty(M, N, dtype=torch.float16, device=DEV), x.to(DEV)
        ops.gemm_bf16(a16.to(DEV), wd, M, N, K, out_bf16=ob, act=ops.ACT_GELU_ERF, status=st)
        ops.gemm_bf16(a16.to(DEV), wd, M, N, K, out_f16=oh, alpha=2.0, status=st)
        ops.gemm_bf16(a16.to(DEV), wd, M, N, K, out_f32=xd, accumulate=True, alpha=0.3, status=st)
        y16 = a16.double() @ w.double().T
        assert rel(ob.float(), R.gelu_ff(a16.double(), {"up": w.double(), "down": eye}, "")) < 4e-3
        assert rel(oh.float(), 2 * y16) < 1e-3 and rel(xd, x.double() + 0.3 * y16) < 1e-5 and int(st.item()) == 0


@pytest.mark.parametrize("heads,N,K,head_k,head_ldc", [(3, 40, 24, 40, 48), (16, 512, 128, 192, 576), (4, 64, 128, 128, 64), (1, 8, 8, 8, 8), (5, 136, 72, 72, 136), (40, 128, 512, 512, 128)])
def test_one_product_per_head(heads, N, K, head_k, head_ldc):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(6)
    for M in (1, 7, 65, 200):
        a, w = torch.randn(M, heads * head_k, generator=g).bfloat16(), torch.randn(heads * N, K, generator=g).bfloat16() * K ** -0.5
        gate = torch.randn(M, heads * head_ldc + 8, generator=g)
        want = torch.einsum("mhk,hnk->mhn", a.double().view(M, heads, head_k)[..., :K], w.double().view(heads, N, K)) * 0.7
        gates = torch.sigmoid(gate[:, : heads * head_ldc].double().view(M, heads, head_ldc)[..., :N])
        for gd, ref in ((None, want), (gate.to(DEV), want * gates)):
            for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 4e-3), (torch.float16, 1e-3)):
                out, st = torch.full((M, heads * head_ldc), 9.0, dtype=dt, device=DEV), i32(0)
                ops.gemm_heads(a.to(DEV), w.to(DEV), heads, N, K, head_k, out, head_ldc, alpha=0.7, gate=gd, status=st)
                got = out.float().view(M, heads, head_ldc)
                assert rel(got[..., :N], ref) < tol and int(st.item()) == 0
                assert (got[..., N:] == 9.0).all()
            out = torch.full((M, heads * head_ldc), 9.0, device=DEV)
            ops.gemm_f32(a.float().to(DEV), w.to(DEV), out, alpha=0.7, gate=gd, heads=heads, head_k=head_k, head_ldc=head_ldc)
            got = out.view(M, heads, head_ldc)
            assert rel(got[..., :N], ref) < 1e-6 and (got[..., N:] == 9.0).all()
            for rows in (1, 2, 3, 8):
                if rows <= M:
                    out = torch.full((M, heads * head_ldc), 9.0, device=DEV)
                    ops.head_matvec(a[:rows].float().to(DEV), w.to(DEV), out, heads, head_k, head_ldc, alpha=0.7, gate=None if gd is None else gd[:rows])
                    got = out.view(M, heads, head_ldc)
                    assert rel(got[:rows, :, :N], ref[:rows]) < 1e-6 and (got[..., N:] == 9.0).all() and (got[rows:] == 9.0).all()


# ---------------------------------------------------------------- chunked differential attention
def regroup(q, G):
    """[T, H, 2, dim] -> query rows [T, 2 H, dim] in the kernels' order (key/value head, map, head of the group)."""
    T, H, _, dim = q.shape
    return q.view(T, G, H // G, 2, dim).transpose(2, 3).reshape(T, 2 * H, dim)


def differential(kernel, qs, ks, vs, chunk, scale, lam, mult, bias=None):
    """A batch through the projection finish, an attention kernel and the difference of the maps.  qs [T, H, 2, dim] at each sequence's last positions, ks
    [S, G, 2, dim], vs [S, G, vdim]; the cache is filled by the finish kernel itself, all tokens first, then the queries' step."""
    from openagents_b200.ops import cuda_ops as ops
    H, dim, G, vdim, B = qs[0].shape[1], qs[0].shape[3], ks[0].shape[1], vs[0].shape[2], len(qs)
    tc = kernel in ("decode", "tc05")
    DK, DV = ((dim + 63) // 64 * 64, (vdim + 63) // 64 * 64) if tc else ((dim + 7) // 8 * 8, (vdim + 7) // 8 * 8)
    dt = torch.float32 if kernel == "exact32" else torch.float16
    table, n_pages = pages_of([k.shape[0] for k in ks])
    kc, vc = torch.zeros(n_pages, G, 16, 2 * DK, dtype=dt, device=DEV), torch.zeros(n_pages, G, 16, DV, dtype=dt, device=DEV)
    nq, nk, nv = 2 * H * dim, 2 * G * dim, G * vdim
    bias = torch.zeros(nq + nk + nv) if bias is None else bias
    rows = []
    for q, k, v in zip(qs, ks, vs):
        S, T = k.shape[0], q.shape[0]
        full = torch.zeros(S, H, 2, dim)
        full[S - T:] = q
        rows.append(torch.cat([regroup(full, G).reshape(S, -1), k.reshape(S, -1), v.reshape(S, -1)], 1) - bias)
    row = torch.cat(rows).to(DEV)
    slot = torch.cat([slots_of(table, b, k.shape[0]) for b, k in enumerate(ks)]).to(torch.int32).to(DEV)
    pos = torch.cat([torch.arange(k.shape[0]) for k in ks]).to(torch.int32).to(DEV)
    last = torch.cat([torch.arange(k.shape[0]) >= k.shape[0] - q.shape[0] for q, k in zip(qs, ks)]).to(DEV)
    lens = [q.shape[0] for q in qs]
    T = sum(lens)
    fin = lambda r, p, s, **kw: ops.qkv_finish(r, 0, nq, nq + nk, p, s, None, 1.0, 2 * H, G, dim, vdim, DK, DV, 0, 1, False, 1e-5, scale, 16, kc=kc, vc=vc, maps=2,      # noqa: E731
                                               bias=bias.to(DEV), **kw)
    fin(row, pos, slot, q32=torch.empty(row.shape[0], 2 * H * DK, device=DEV))
    q32 = torch.full((T, 2 * H, (2 if kernel == "decode" else 1) * DK), 7.0, device=DEV)
    q16 = torch.full((T, 2 * H, DK), 7.0, dtype=torch.float16, device=DEV) if kernel != "decode" else None
    fin(row[last].contiguous(), pos[last].contiguous(), slot[last].contiguous(), q32=q32, q16=q16, q_wide=kernel == "decode")
    starts, ctx, tab = i32(*[sum(lens[:b]) for b in range(B)]), i32(*[k.shape[0] for k in ks]), table.to(DEV)
    maps_out, st = torch.full((T, 2 * H * DV), 5.0, device=DEV), i32(0)
    if kernel == "decode":
        S = 3
        ops.attn_decode(q32.view(T, -1), kc, vc, tab, ctx, B, 2 * H, G, 2 * DK, dv=DV, S=S, out_f32=maps_out, chunk=chunk, status=st,
                        scratch=torch.empty(ops.attn_decode_scratch_floats(B, 2 * H, G, DV, S), device=DEV), counters=torch.zeros(B * 2 * H, dtype=torch.int32, device=DEV))
    elif kernel == "tc05":
        ops.attn_prefill_tc05(q16.view(T, -1), kc, vc, tab, starts, i32(*lens), ctx, B, max(lens), 2 * H, G, out_f32=maps_out, status=st, dk=DK, dv=DV, chunk=chunk, maps=2)
    else:
        ops.attn_exact(q32.view(T, -1), kc, vc, tab, starts, i32(*lens), ctx, B, max(lens), 2 * H, G, DK, DV, out_f32=maps_out, maps=2, chunk=chunk)
    out = torch.full((T, H * DV), 9.0, device=DEV)
    ops.diff_combine(maps_out, torch.tensor([lam], device=DEV), H, G, vdim, DV, 1e-5, mult, out_f32=out)
    torch.cuda.synchronize()
    assert int(st.item()) == 0
    out = out.view(T, H, DV)
    assert not out[..., vdim:].any()
    return out[..., :vdim].cpu()


def want_differential(qs, ks, vs, chunk, scale, lam, mult):
    out = []
    for q, k, v in zip(qs, ks, vs):
        a1, a2 = R.differential_attention(q.double(), k.double(), v.double(), scale, chunk, k.shape[0] - q.shape[0])
        out.append(R.unit_rms(a1 - lam * a2, 1e-5) * mult)
    return torch.cat(out)


DIFF = [(4, 2, 40, 24), (6, 1, 64, 128), (3, 3, 16, 72), (20, 1, 56, 64), (9, 3, 104, 100), (1, 1, 8, 8)]


@pytest.mark.parametrize("kernel,tol", [("exact32", 2e-5), ("exact16", 3e-3), ("decode", 6e-3), ("tc05", 6e-3)])
@pytest.mark.parametrize("H,G,dim,vdim", DIFF)
@pytest.mark.parametrize("chunk", [0, 1, 16, 50, 128, 1000])
def test_chunked_differential_attention(kernel, tol, H, G, dim, vdim, chunk):
    g = torch.Generator().manual_seed(2)
    f = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    shapes = [(1, 1), (1, 77), (1, 300), (1, 51), (1, 128), (1, 129)] if kernel == "decode" else [(1, 1), (3, 20), (64, 64), (130, 141), (1, 33), (200, 260)]
    qs, ks, vs = [f(t, H, 2, dim) for t, _ in shapes], [f(n, G, 2, dim) for _, n in shapes], [f(n, G, vdim) for _, n in shapes]
    bias = f(2 * H * dim + 2 * G * dim + G * vdim)
    scale = 1.3 * dim ** -0.5
    got = differential(kernel, qs, ks, vs, chunk, scale, 0.6, 0.7, bias)
    want = want_differential(qs, ks, vs, chunk, scale, 0.6, 0.7)
    if chunk == 1 and kernel != "exact32":               # every row sees one key: 0.4 v, the same relative error everywhere
        tol = 2e-3
    assert rel(got, want) < tol


@pytest.mark.parametrize("kernel", ["exact32", "decode", "tc05"])
@pytest.mark.parametrize("chunk", [32, 48, 100, 128])
def test_the_first_key_of_a_chunk_is_seen_and_the_last_of_the_one_before_is_not(kernel, chunk):
    """Two keys stand out, on either side of a chunk's edge: a query of the later chunk takes the inner one's value, however far into the chunk it stands,
    and a query of the earlier chunk the outer one's.  The second map's keys stay dark, so the difference shows the first map."""
    H, G, D = 2, 1, 64
    g = torch.Generator().manual_seed(3)
    qs, ks, vs, want = [], [], [], []
    for edge in (chunk, 2 * chunk):
        for n in (edge, edge + 1, edge + 2, edge + chunk - 1, edge + chunk):           # context length: the query is its last token
            k, v = torch.randn(n, G, 2, D, generator=g), torch.randn(n, G, D, generator=g)
            k[:, :, 1] = 0
            q = torch.zeros(1, H, 2, D)
            q[..., 0, 5] = 1.0
            k[:, 0, 0, 5] = 0
            k[edge - 1, 0, 0, 5] = 80.0
            if n > edge:
                k[edge, 0, 0, 5] = 40.0
            qs.append(q)
            ks.append(k)
            vs.append(v)
            lo = (n - 1) // chunk * chunk
            first = v[edge if n > edge else edge - 1, 0]
            want.append(R.unit_rms(first.double() - 0.5 * v[lo:, 0].double().mean(0), 1e-5))
    got = differential(kernel, qs, ks, vs, chunk, 1.0, 0.5, 1.0)
    for i, w in enumerate(want):
        assert (got[i] - w).abs().max() < 0.03, i


# ---------------------------------------------------------------- latent attention
@pytest.mark.parametrize("style", [0, 1])
def test_latents_are_normed_and_the_shared_part_rotates(style):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(1)
    for q_rank, rank, rd, rot, CR, RR, H, dim in ((20, 36, 10, 10, 40, 16, 3, 24), (96, 130, 64, 64, 192, 64, 5, 128), (7, 64, 6, 4, 64, 64, 1, 9)):
        T, ldq = 5, (q_rank + 7) // 8 * 8
        row = torch.randn(T, q_rank + rank + rd + 3, generator=g)
        qw, cw = torch.randn(q_rank, generator=g), torch.randn(rank, generator=g)
        pos, slot = i32(0, 1, 15, 16, 900), i32(16 * 3 + 1, 0, 16 * 7 + 15, -1, 16 * 2)
        table = ops.rope_table(17, rot, 500.0, DEV)      # 900 lies outside: computed on the spot

        def turn(x):
            if style == 1:
                return R.rotate_half(x, pos.cpu(), rot, 500.0)
            perm = [2 * i for i in range(rot // 2)] + [2 * i + 1 for i in range(rot // 2)] + list(range(rot, rd))
            return R.rotate_half(x[..., perm], pos.cpu(), rot, 500.0)[..., [perm.index(i) for i in range(rd)]]
        r = row.double()
        cq = R.unit_rms(r[:, :q_rank], 1e-4) * qw.double()
        c = R.unit_rms(r[:, q_rank: q_rank + rank], 1e-4) * cw.double()
        kr = turn(r[:, None, q_rank + rank: q_rank + rank + rd])[:, 0]
        for dt, eps in ((torch.float32, 1e-6), (torch.float16, 1e-3)):
            cache = torch.full((8, 16, CR + RR), 3.0, dtype=dt, device=DEV)
            out = torch.full((T, ldq), 9.0, dtype=torch.float32 if dt == torch.float32 else torch.bfloat16, device=DEV)
            ops.latent_finish(row.to(DEV), 0, q_rank, q_rank + rank, q_rank, rank, rd, rot, style, qw.to(DEV), cw.to(DEV), 1e-4, pos, slot, table, 500.0, out, cache, CR, RR)
            assert rel(out[:, :q_rank].float(), cq) < (1e-6 if dt == torch.float32 else 4e-3) and not out[:, q_rank:].any()
            flat = cache.view(-1, CR + RR).float().cpu()
            for t, s in enumerate(slot.tolist()):
                if s >= 0:
                    assert rel(flat[s, :rank], c[t]) < eps and rel(flat[s, CR: CR + rd], kr[t]) < eps
                    assert not flat[s, rank:CR].any() and not flat[s, CR + rd:].any()
            untouched = torch.ones(128, dtype=torch.bool)
            untouched[[s for s in slot.tolist() if s >= 0]] = False
            assert (flat[untouched] == 3.0).all()
        hs = (dim + rd + 7) // 8 * 8
        q = torch.randn(T, H * hs, generator=g)
        parts = q.double().view(T, H, hs)
        NC, width = (dim + 7) // 8 * 8, (dim + 7) // 8 * 8 + CR + RR
        for dt, eps in ((torch.float32, 1e-6), (torch.float16, 1e-3)):
            out = torch.full((T, H, width), 9.0, dtype=dt, device=DEV)
            ops.latent_q(q.to(DEV), hs, H, dim, rd, rot, style, NC, NC + CR, RR, width, pos, table, 500.0, 0.25, out)
            o = out.float().cpu()
            assert rel(o[..., :dim], parts[..., :dim] * 0.25) < eps and rel(o[..., NC + CR: NC + CR + rd], turn(parts[..., dim: dim + rd]) * 0.25) < eps
            assert not o[..., dim:NC].any() and not o[..., NC + CR + rd:].any() and (o[..., NC: NC + CR] == 9.0).all()
            ops.latent_q(q.to(DEV), hs, H, dim, rd, rot, style, 0, NC + CR, RR, width, pos, table, 500.0, 0.25, out.fill_(9.0))
            assert (out[..., : NC + CR] == 9.0).all()


def latent_cache(ctx, W, CR, seed=3, dt=torch.float16):
    """Cached rows [len, W] of sequences of these lengths (the last columns are the rotated part), their pages and the paged cache."""
    g = torch.Generator().manual_seed(seed)
    rows = [torch.randn(n, W, generator=g) for n in ctx]
    table, n_pages = pages_of(ctx)
    cache = torch.zeros(n_pages * 16, W, dtype=dt)
    for b, r in enumerate(rows):
        cache[slots_of(table, b, r.shape[0])] = r.to(dt)
    return rows, table.to(DEV), cache.view(n_pages, 16, W).to(DEV)


def want_latent(q, rows, CR, pos, sink):
    """q [H, W] in the latent space against rows[:pos + 1]."""
    k = rows[: pos + 1].double()
    w = R.weights_over_keys((q.double() @ k.T)[:, None], torch.ones(1, pos + 1, dtype=torch.bool), None if sink is None else sink.double())[:, 0]
    return w @ k[:, :CR]


@pytest.mark.parametrize("H,CR,RR", [(1, 64, 64), (4, 128, 64), (16, 512, 64), (17, 192, 64), (32, 512, 64), (40, 256, 128), (5, 320, 64), (33, 64, 64)])
@pytest.mark.parametrize("S", [1, 2, 7])
def test_decoding_in_the_latent_space(H, CR, RR, S):
    """Rows of several sequences (some share one), block and page edges, fewer key blocks than shares, with and without sinks."""
    from openagents_b200.ops import cuda_ops as ops
    W = CR + RR
    ctx = [1, 16, 63, 64, 65, 129, 400, 700]
    rows, table, cache = latent_cache(ctx, W, CR)
    seq = [0, 1, 2, 3, 4, 5, 6, 7, 7, 7, 6]
    pos = [0, 15, 62, 63, 64, 128, 399, 699, 340, 0, 255]
    g = torch.Generator().manual_seed(4)
    n = len(seq)
    q = torch.randn(n, H, W, generator=g) * 1.5 * W ** -0.5
    sink = torch.randn(H, generator=g) + 1.0
    for sk in (None, sink):
        o32, o16, st = torch.full((n, H * CR), 9.0, device=DEV), torch.zeros(n, H * CR, dtype=torch.bfloat16, device=DEV), i32(0)
        scratch = torch.full((max(1, ops.latent_decode_scratch_floats(n, H, CR, S)),), float("nan"), device=DEV)
        ops.latent_decode(q.to(DEV), cache, table, i32(*seq), i32(*pos), n, H, CR, RR, S, scratch, out_f32=o32, out_bf16=o16, sinks=None if sk is None else sk.to(DEV), status=st)
        torch.cuda.synchronize()
        assert int(st.item()) == 0
        for r in range(n):
            want = want_latent(q[r], rows[seq[r]], CR, pos[r], sk)
            assert rel(o32[r].view(H, CR), want) < 2e-3, r
            assert rel(o16[r].float().view(H, CR), want) < 5e-3, r
    o2 = torch.empty(8, H * CR, device=DEV)
    ops.latent_decode(q[:8].contiguous().to(DEV), cache, table, None, i32(*pos[:8]), 8, H, CR, RR, S, scratch, out_f32=o2, status=st)      # row r is sequence r
    for r in range(8):
        assert rel(o2[r].view(H, CR), want_latent(q[r], rows[r], CR, pos[r], None)) < 2e-3, r


@pytest.mark.parametrize("S", [1, 3])
def test_decoding_in_the_latent_space_finds_one_key_and_moves_its_offset(S):
    """One score stands out far above the others wherever it lies, also late (the running maximum jumps), and just behind the query, where it must not count."""
    from openagents_b200.ops import cuda_ops as ops
    H, CR, RR, n = 3, 128, 64, 500
    places = [0, 1, 15, 16, 63, 64, 65, 127, 128, 255, 256, 430, 498]
    rows, table, cache = latent_cache([n] * len(places), CR + RR, CR)
    q = torch.zeros(len(places), H, CR + RR)
    pos = []
    flat = cache.view(-1, CR + RR)
    for b, p in enumerate(places):
        slots = slots_of(table.cpu(), b, n).to(DEV)
        flat[slots, CR + 3] = 0
        flat[slots[p], CR + 3] = 60.0
        flat[slots[p + 1], CR + 3] = 90.0                # the next one stands out more
        q[b, :, CR + 3] = 1.0
        pos.append(p if b % 2 else n - 1)                # seen by the last token, hidden from the token right ahead of it
    st, out = i32(0), torch.empty(len(places), H * CR, device=DEV)
    scratch = torch.empty(max(1, ops.latent_decode_scratch_floats(len(places), H, CR, S)), device=DEV)
    ops.latent_decode(q.to(DEV), cache, table, None, i32(*pos), len(places), H, CR, RR, S, scratch, out_f32=out, status=st)
    for b, p in enumerate(places):
        want = rows[b][p if b % 2 else p + 1, :CR].half().float()
        assert (out[b].view(H, CR).cpu() - want).abs().max() < 0.01, p
    assert int(st.item()) == 0


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-5), (torch.float16, 1e-3)])
@pytest.mark.parametrize("H,CR,RR", [(3, 40, 16), (2, 136, 8), (5, 520, 64), (1, 1000, 24)])
def test_exact_attention_on_latents(dt, tol, H, CR, RR):
    from openagents_b200.ops import cuda_ops as ops
    W = CR + RR
    lens, ctx = [1, 9, 40], [33, 9, 77]
    rows, table, cache = latent_cache(ctx, W, CR, dt=dt)
    g = torch.Generator().manual_seed(7)
    T = sum(lens)
    q, sink = torch.randn(T, H, W, generator=g) * W ** -0.5, torch.randn(H, generator=g) + 2
    out = torch.empty(T, H * CR, device=DEV)
    ops.attn_exact(q.to(DEV).view(T, -1), cache.view(-1, 1, 16, W), None, table, i32(0, 1, 10), i32(*lens), i32(*ctx), 3, 40, H, 1, W, CR, out_f32=out, sinks=sink.to(DEV))
    at = 0
    for b, n in enumerate(lens):
        for i in range(n):
            assert rel(out[at + i].view(H, CR), want_latent(q[at + i], rows[b], CR, ctx[b] - n + i, sink)) < tol
        at += n


@pytest.mark.parametrize("H,kn,rr,dv", [(3, 64, 64, 64), (2, 128, 64, 128), (5, 64, 128, 128), (1, 128, 128, 64), (2, 64, 64, 128), (2, 192, 64, 128)])
def test_prompts_on_the_expanded_context(H, kn, rr, dv):
    """Own key parts and values in a workspace, the shared part in the paged cache; portions of unequal length, sinks, a gate per element."""
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(8)
    lens, ctx = [17, 64, 130, 2, 200], [17, 100, 141, 290, 200]
    CR = 64
    rows, table, cache = latent_cache(ctx, CR + rr, CR)
    base, n = [sum(ctx[:b]) for b in range(len(ctx))], sum(ctx)
    ws = torch.zeros(n + 5, H * (kn + dv), dtype=torch.float16)
    ws[:n] = torch.randn(n, H * (kn + dv), generator=g).half()
    T = sum(lens)
    q = torch.randn(T, H, kn + rr, generator=g) * (kn + rr) ** -0.5
    gate, sink = torch.randn(T, H * dv, generator=g), torch.randn(H, generator=g) + 1.5
    starts = [sum(lens[:b]) for b in range(len(lens))]
    for gt, sk in ((None, None), (gate, sink)):
        out, st = torch.zeros(T, H * dv, dtype=torch.bfloat16, device=DEV), i32(0)
        ops.attn_prefill_latent(q.half().to(DEV).view(T, -1), ws.to(DEV), H * kn, i32(*base), cache, CR, table, i32(*starts), i32(*lens), i32(*ctx), len(lens), max(lens), H,
                                kn, rr, dv, out, sinks=None if sk is None else sk.to(DEV), gate=None if gt is None else gt.to(DEV), status=st)
        torch.cuda.synchronize()
        assert int(st.item()) == 0
        for b, m in enumerate(lens):
            own = ws[base[b]: base[b] + ctx[b]].double()
            k = torch.cat([own[:, : H * kn].view(-1, H, kn), rows[b][:, None, CR:].double().expand(-1, H, -1)], -1)
            s = torch.einsum("thd,shd->hts", q[starts[b]: starts[b] + m].double(), k)
            w = R.weights_over_keys(s, R.visible(ctx[b] - m, m, ctx[b]), None if sk is None else sk.double())
            want = torch.einsum("hts,shv->thv", w, own[:, H * kn:].view(-1, H, dv)).reshape(m, -1)
            if gt is not None:
                want = want * torch.sigmoid(gt[starts[b]: starts[b] + m].double())
            assert rel(out[starts[b]: starts[b] + m].float(), want) < 6e-3, b


def test_gathered_latents():
    from openagents_b200.ops import cuda_ops as ops
    ctx, CR, W = [5, 130, 16], 72, 136
    rows, table, cache = latent_cache(ctx, W, CR)
    out = torch.full((200, CR), 9.0, dtype=torch.bfloat16, device=DEV)
    ops.latent_gather(cache, CR, table, i32(*ctx), i32(3, 40, 8), 3, 130, out)
    for b, at in enumerate((3, 40, 8)):
        assert rel(out[at: at + ctx[b]].float(), rows[b][:, :CR]) < 4e-3
    assert (out[:3] == 9.0).all() and (out[170:] == 9.0).all() and (out[24:40] == 9.0).all()


# ---------------------------------------------------------------- whole models
A, M = R.layer_attention, R.layer_latent
CONFIGS = {
    # odd sizes, a width and a vocabulary that are no multiples of eight and four, chunks beside the page size, three passes of the loop
    "odd": R.config([A(40, 24, 6, 2, 24, ff=100), M(24, 10, 40, 3, 36, 20, base=500.0, ff=36), A(16, 56, 3, 1, 7, diff=0.1, scale=0.4)], width=100, vocab=131, loop=(1, 3, 3)),
    # latent layers only: one head, many heads, a rotated pair, a query latent wider than the model, the whole stack looped
    "latent": R.config([M(64, 16, 64, 1, 64, 100, ff=96), M(16, 2, 24, 40, 100, 24, base=100.0, scale=0.5), M(128, 64, 128, 2, 192, 40, ff=64)], width=64, vocab=300,
                       loop=(0, 3, 2), residual_mult=1.0),
    # differential layers only, no loop, one key/value head, as many as query heads, groups wider than a tile, a chunk of one token
    "differential": R.config([A(64, 128, 4, 1, 64, ff=96, diff=0.8), A(8, 16, 5, 5, 100), A(48, 80, 12, 1, 33, diff=0.0, ff=40), A(24, 32, 2, 2, 1)], width=128, vocab=260,
                             eps=1e-3, residual_mult=0.3),
    # head sizes and latents beyond the tensor-core kernels
    "wide": R.config([A(136, 72, 2, 1, 40, ff=72), M(200, 8, 24, 2, 40, 16), A(40, 200, 2, 2, 96), M(24, 8, 136, 3, 520, 64, ff=64)], width=96, vocab=264, loop=(2, 4, 2)),
}


def open_model(tmp_path, cfg, W, dtype="float32", max_num_seqs=4, max_ctx=512, max_tokens=512, **kw):
    from openagents_b200.serve.backend import CudaBackend
    return CudaBackend.open(R.save_model(str(tmp_path / "m"), cfg, W), max_num_seqs=max_num_seqs, max_ctx=max_ctx, max_tokens=max_tokens, dtype=dtype, **kw)


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run(be, seq, toks, cuts):
    """Feed ``toks`` in portions of the sizes in ``cuts`` (cycled); logits of every token."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[i % len(cuts)], len(toks) - at)
        out.append(be.forward_at([seq], [toks[at: at + n]], [list(range(n))]))
        at, i = at + n, i + 1
    be.engine.check_status()
    return torch.cat(out)


def close(got, want, dtype):
    """Every position's error within the tolerance (mean taken off, over the logits' spread)."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.double().std()
    assert err.max().item() < TOL[dtype], (err.max().item(), int(err.argmax()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompts_portions_and_decoding(tmp_path, name, dtype):
    cfg = CONFIGS[name]
    W = R.random_weights(cfg, seed=len(name))
    be = open_model(tmp_path, cfg, W, dtype)
    toks = tokens(cfg, 203, 1)
    want = R.forward(cfg, W, toks, R.Sequence())
    for seq, cuts in enumerate(([203], [150] + [1] * 200, [2, 64, 3, 61, 1, 17], [2], [65, 16, 1])):
        be.begin(seq, None)
        close(run(be, seq, toks, cuts), want, dtype)
        be.end(seq)
    be.begin(9, None)                      # token by token from the first
    close(run(be, 9, toks[:40], [1]), want[:40], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_after_every_layer_run(tmp_path, dtype):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=2)
    toks = tokens(cfg, 70, 3)
    layers = []
    R.forward(cfg, W, toks, R.Sequence(), layers)
    e = open_model(tmp_path, cfg, W, dtype).engine
    runs = e.runs
    assert len(runs) == len(layers) == 7
    for n in range(1, len(runs) + 1):
        e.runs = runs[:n]
        e.begin(n)
        e.forward_tokens([n], [toks])
        assert rel(e.x[: len(toks), : cfg["width"]], layers[n - 1]) < TOL[dtype] / 3, n
        assert not e.x[: len(toks), cfg["width"]:].any()
        e.end(n)


@pytest.mark.parametrize("name", ["odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_reuse_pages(tmp_path, name, dtype):
    """Portions beside single tokens in any order, sequences left out of steps, and a pool so tight that pages come round again; each request's logits are those
    it has alone."""
    cfg = CONFIGS[name]
    W = R.random_weights(cfg, seed=5)
    be = open_model(tmp_path, cfg, W, dtype, max_num_seqs=4, n_pages=24, max_ctx=24 * 16, max_tokens=24 * 16)
    want, toks = {}, {}
    for r, n in enumerate((120, 33, 97, 64, 5, 140, 18)):
        toks[r] = tokens(cfg, n, 10 + r)
        want[r] = R.forward(cfg, W, toks[r], R.Sequence())
    g = torch.Generator().manual_seed(8)
    queue, live, at, got, seq = list(toks), [], {}, {r: [] for r in toks}, {}
    nxt = 100
    while queue or live:
        while queue and len(live) < 4 and sum((len(toks[r]) + 15) // 16 for r in live + queue[:1]) <= 24:
            r = queue.pop(0)
            live.append(r)
            at[r], seq[r], nxt = 0, nxt, nxt + 1
            be.begin(seq[r], None)
        step = [r for r in live if torch.rand(1, generator=g).item() < 0.8] or live[:1]
        feeds = []
        for r in step:
            n = [1, 1, 2, 7, 31, 64][int(torch.randint(0, 6, (1,), generator=g))]
            feeds.append(toks[r][at[r]: at[r] + n])
        out = be.forward_at([seq[r] for r in step], feeds, [list(range(len(f))) for f in feeds])
        lo = 0
        for r, f in zip(step, feeds):
            got[r].append(out[lo: lo + len(f)])
            lo += len(f)
            at[r] += len(f)
            if at[r] == len(toks[r]):
                be.end(seq[r])
                live.remove(r)
    be.engine.check_status()
    for r in toks:
        close(torch.cat(got[r]), want[r], dtype)
    assert be.kv_stats()["pages_free"] == 24


def test_contexts_beyond_the_workspace_run_in_groups(tmp_path):
    """The expanded contexts of a step need not fit the workspace together, and a step's answers come back in the caller's order."""
    cfg = CONFIGS["latent"]
    W = R.random_weights(cfg, seed=3)
    be = open_model(tmp_path, cfg, W, "bfloat16", max_num_seqs=4, max_ctx=160, max_tokens=160)
    toks = [tokens(cfg, n, n) for n in (150, 100, 60, 140)]
    want = [R.forward(cfg, W, t, R.Sequence()) for t in toks]
    for b, t in enumerate(toks):
        be.begin(b, None)
        be.forward_at([b], [t[:-30]], [[]])
    cuts = [30, 20, 1, 25]
    feeds = [t[-30:][:n] for t, n in zip(toks, cuts)]
    rows = be.forward_at([0, 1, 2, 3], feeds, [list(range(n)) for n in cuts])
    assert len(be.engine._plan.groups) > 1
    at = 0
    for t, w, n in zip(toks, want, cuts):
        close(rows[at: at + n], w[len(t) - 30: len(t) - 30 + n], "bfloat16")
        at += n
    order = [2, 1, 3]
    logits, ids = be.engine.forward_tokens(order, [toks[2][-29:-27], toks[1][-10:], toks[3][-5:]], all_positions=False)
    for row, i, w in zip(logits, ids, (want[2][-28], want[1][-1], want[3][-1])):
        close(row.cpu()[None], w[None], "bfloat16")
        assert int(i) == int(row.argmax())
    assert be.score(0, toks[0][:3], toks[0][1:4])[0] < 0


def test_stack_shares_prefixes_and_can_be_cut(tmp_path):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=6)
    be = open_model(tmp_path, cfg, W)
    toks = tokens(cfg, 60, 2)
    want = R.forward(cfg, W, toks, R.Sequence())
    assert be.begin(1, toks) == 0
    be.forward_at([1], [toks], [[]])
    be.publish(1, toks)
    assert be.begin(2, toks) == 48
    close(be.forward_at([2], [toks[48:]], [list(range(12))]), want[48:], "float32")
    be.truncate(2, 50)
    close(run(be, 2, toks[50:], [3]), want[50:], "float32")
    be.truncate(2, 20)                     # into a page that both sequences hold
    other = tokens(cfg, 12, 9)
    close(run(be, 2, other, [12]), R.forward(cfg, W, toks[:20] + other, R.Sequence())[20:], "float32")
    close(run(be, 1, other, [12]), R.forward(cfg, W, toks + other, R.Sequence())[60:], "float32")
    assert be.supports_verify
    be.begin(3, None)
    assert be.verify(3, toks[:4]) == want[:4].argmax(-1).tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=7)
    be = open_model(tmp_path, cfg, W, dtype, max_ctx=700, max_tokens=64)
    toks = tokens(cfg, 600, 4)
    want = R.forward(cfg, W, toks, R.Sequence())
    be.begin(1, None)
    got = [run(be, 1, toks[:30], [30])]
    got += [be.forward_at([1], [[t]], [[0]]) for t in toks[30:]]
    close(torch.cat(got), want, dtype)


@pytest.mark.parametrize("name", ["odd", "latent"])
def test_decode_batches_of_every_path(tmp_path, name):
    """Decode batches for the mat-vec path, the one-tile GEMM and beyond it (bf16), each sequence against itself alone."""
    cfg = CONFIGS[name]
    W = R.random_weights(cfg, seed=9)
    for B in (1, 2, 7, 40, 70):
        be = open_model(tmp_path / str(B), cfg, W, "bfloat16", max_num_seqs=B, max_ctx=64, max_tokens=B * 12)
        toks = [tokens(cfg, 3 + b % 9, 50 + b) for b in range(B)]
        more = [tokens(cfg, 3, 500 + b) for b in range(B)]
        for b in range(B):
            be.begin(b, None)
        be.forward_at(list(range(B)), toks, [[] for _ in toks])
        rows = [be.forward_at(list(range(B)), [[m[i]] for m in more], [[0]] * B) for i in range(3)]
        be.engine.check_status()
        for b in range(0, B, max(1, B // 6)):
            want = R.forward(cfg, W, toks[b] + more[b], R.Sequence())[-3:]
            close(torch.stack([r[b] for r in rows]), want, "bfloat16")


@pytest.mark.parametrize("name", ["odd", "latent", "differential"])
def test_greedy_generation_through_the_scheduler(tmp_path, name):
    """Continuous batching end to end in the 32-bit mode: the ids are the plain implementation's."""
    from openagents_b200.serve.generation import SamplingParams, Scheduler

    class Tok:
        eos_id = -1

        def decode(self, ids):
            return ""
    cfg = CONFIGS[name]
    W = R.random_weights(cfg, seed=11)
    be = open_model(tmp_path, cfg, W, max_num_seqs=3)
    sched = Scheduler(be, Tok(), max_num_seqs=3, prefill_chunk=24)
    prompts = [tokens(cfg, n, 20 + n) for n in (50, 9, 31, 2, 70)]
    reqs = [sched.submit(p, SamplingParams(max_tokens=12)) for p in prompts]
    sched.run_until_done(reqs)
    for p, r in zip(prompts, reqs):
        assert r.finish_reason == "length", r.error
        ids, rows = R.generate(cfg, W, p, 12)
        for t, (a, b) in enumerate(zip(r.output, ids)):
            if a != b:                      # only where the two best logits are closer than rounding
                top = rows[t].topk(2).values
                assert (top[0] - top[1]).item() < 1e-3, t
                break
    hot = sched.submit(prompts[0], SamplingParams(max_tokens=5, temperature=0.8, top_k=8, seed=3))
    sched.run_until_done([hot])
    assert len(hot.output) == 5 and all(0 <= t < cfg["vocab"] for t in hot.output)


def test_generate_and_device_side_decode_loop(tmp_path):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=12)
    be = open_model(tmp_path, cfg, W)
    prompt = tokens(cfg, 25, 6)
    ids, rows = R.generate(cfg, W, prompt, 10)
    for graph in (False, True):
        out, logits = be.engine.generate(prompt, 10, seq_id=int(graph), use_graph=graph)
        assert out == ids
        close(logits, rows, "float32")
        be.end(int(graph))
    be.begin(5, None)
    _, nxt = be.engine.forward_tokens([5], [prompt])
    first = int(nxt[0])
    hist = be.engine.decode_steps([5], [first], 9)
    assert [first] + hist[:, 0].tolist() == ids


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_workspace_canaries(tmp_path, name):
    cfg = CONFIGS[name]
    W = R.random_weights(cfg, seed=13)
    for dtype in ("float32", "bfloat16"):
        be = open_model(tmp_path / dtype, cfg, W, dtype, canaries=True, max_tokens=203)
        toks = tokens(cfg, 203, 1)
        be.begin(1, None)
        close(run(be, 1, toks, [100, 1, 64, 1]), R.forward(cfg, W, toks, R.Sequence()), dtype)
        assert be.engine.check_canaries() == []


def test_gguf_round_trip(tmp_path):
    """A GGUF file written by the framework gives the folder's logits."""
    from openagents_b200.models.registry import open_source
    from openagents_b200.models.weights import PLAN_BF16, save_gguf
    from openagents_b200.serve.backend import CudaBackend
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=14)
    be = open_model(tmp_path, cfg, W)
    src = open_source(str(tmp_path / "m"), "cpu")
    path = str(tmp_path / "m.gguf")
    save_gguf(path, src.cfg, {k: v.float().reshape(v.shape or (1,)) for k, v in W.items()}, PLAN_BF16)
    be2 = CudaBackend.open(path, max_num_seqs=4, max_ctx=128, max_tokens=128, dtype="float32")
    assert be2.cfg.layers == src.cfg.layers and be2.cfg.loop == src.cfg.loop
    toks = tokens(cfg, 50, 1)
    for b in (be, be2):
        b.begin(1, None)
    assert torch.equal(be.forward_at([1], [toks], [list(range(50))]), be2.forward_at([1], [toks], [list(range(50))]))


def test_trace_runner(tmp_path):
    """bin/trace_run as a user starts it."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=15)
    folder = R.save_model(str(tmp_path / "m"), cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    ta, tb = tokens(cfg, 40, 1), tokens(cfg, 21, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:20], "want": []}, {"id": "a", "tokens": ta[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ta[31:], "want": [8]}, {"id": "b", "tokens": tb[20:], "want": [0]}], "end": ["a", "b"]}]
    for dtype in ("float32", "bfloat16"):
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (out / "1.f32").exists()
        fa, fb = R.forward(cfg, W, ta, R.Sequence()), R.forward(cfg, W, tb, R.Sequence())
        got = torch.from_numpy(np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in (0, 2)])).view(4, -1)
        close(got, torch.stack([fa[0], fa[29], fa[39], fb[20]]), dtype)


def test_http_server_on_a_checkpoint_folder(tmp_path):
    """The server as `b200-serve -m FOLDER --dtype float32` builds it, speculation included: the answer of the plain implementation."""
    import json
    import threading
    import urllib.request

    from openagents_b200.serve.server import build_state, parse_args, serve
    cfg = dict(CONFIGS["odd"], vocab=300)
    W = R.random_weights(cfg, seed=16)
    a = parse_args(["-m", R.save_model(str(tmp_path / "tiny-pesorax"), cfg, W), "--dtype", "float32", "--max-num-seqs", "2", "--max-ctx", "512",
                    "--speculation", "n_gram"])
    state = build_state(a.model, a.backend, a.max_num_seqs, a.kv_page_size, a.max_ctx, dtype=a.dtype)
    httpd = serve(state, "127.0.0.1", 0)
    threading.Thread(target=httpd.serve_forever, daemon=True).start()
    base = f"http://127.0.0.1:{httpd.server_address[1]}"

    def post(path, obj):
        req = urllib.request.Request(base + path, json.dumps(obj).encode(), {"Content-Type": "application/json"})
        with urllib.request.urlopen(req, timeout=60) as r:
            return json.loads(r.read())
    try:
        out = post("/v1/completions", {"model": "tiny-pesorax", "prompt": "hello there", "max_tokens": 8, "temperature": 0})
        ids, _ = R.generate(cfg, W, list(b"hello there"), 8)
        stop = ids.index(256) if 256 in ids else len(ids)
        assert out["choices"][0]["text"] == bytes(i for i in ids[:stop] if i < 256).decode("utf-8", "replace")
    finally:
        httpd.shutdown()
        for m in state.models.values():
            m.close()
