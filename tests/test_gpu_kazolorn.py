"""Kazolorn on the GPU: every mechanism alone and whole models against the plain implementation in ``kazolorn_ref``."""
import pytest
import torch

import kazolorn_ref as R

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


# ---------------------------------------------------------------- depth average, norms, PolyNorm
@pytest.mark.parametrize("T,D,ld,n", [(3, 72, 72, 1), (5, 100, 104, 4), (4, 93, 96, 3), (300, 260, 264, 9), (2, 2048, 2048, 17), (1, 4096, 4096, 33), (1, 9000, 9000, 2),
                                      (7, 8192, 8192, 5)])
def test_depth_average_and_the_norms_behind_it(T, D, ld, n):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(0)
    xs = torch.zeros(n + 1, T + 2, ld)
    xs[:, :, :D] = torch.randn(n + 1, T + 2, D, generator=g)
    w, bias = torch.randn(n, generator=g), torch.zeros(ld)
    bias[:D] = torch.randn(D, generator=g)
    g1, g2 = torch.randn(ld, generator=g), torch.randn(ld, generator=g)
    x = R.depth_average([s[:T, :D].double() for s in xs[:n]], w.double())
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 4e-3)):
        d = xs.to(DEV)
        h1, h2, side = torch.full((T, ld), 7.0, dtype=dt, device=DEV), torch.full((T, ld), 7.0, dtype=dt, device=DEV), torch.ones(64, device=DEV)
        ops.depth_norm(d[:n, :T], D, 1e-4, weights=w.to(DEV), out=d[n, :T], add=bias.to(DEV), g1=g1.to(DEV), g2=g2.to(DEV), h1=h1, h2=h2, zero=side)
        assert rel(d[n, :T, :D], x + bias[:D].double()) < 2e-6 and torch.equal(d[n, T:].cpu(), xs[n, T:]) and not d[n, :T, D:].any() and not side.any()
        for h, gain in ((h1, g1), (h2, g2)):
            assert rel(h[:, :D].float(), R.rms_norm(x, gain[:D].double(), 1e-4)) < tol and not h[:, D:].any()
        assert torch.equal(d[:n].cpu(), xs[:n])
    for k in (1, 2, 3):                                # sums that later averages start from, and an average that does
        slabs, pw = torch.full((n + 4, T, ld), 7.0, device=DEV), torch.randn(k, n + 2, generator=g)
        slabs[:n] = xs[:n, :T].to(DEV)
        out = torch.empty(T, ld, device=DEV)
        ops.depth_norm(slabs[:n], D, weights=w.to(DEV), out=out, parts=slabs[n: n + k], part_weights=pw.to(DEV))
        assert rel(out[:, :D], x) < 2e-6 and (slabs[n + k:] == 7.0).all()
        for m in range(k):
            want = R.depth_average([s[:T, :D].double() for s in xs[:n]], pw[m, :n].double())
            assert rel(slabs[n + m, :, :D], want) < 2e-6 and not slabs[n + m, :, D:].any()
        ops.depth_norm(slabs[:n], D, weights=w.to(DEV), out=out, base=slabs[n])
        assert rel(out[:, :D], x + R.depth_average([s[:T, :D].double() for s in xs[:n]], pw[0, :n].double())) < 2e-6
    out, h = torch.empty(T, ld, device=DEV), torch.empty(T, ld, device=DEV)
    ops.depth_norm(d[:1, :T], D, 1e-4, out=out, g2=g2.to(DEV), h2=h)                # one slab as it is, one norm
    assert torch.equal(out[:, :D].cpu(), xs[0, :T, :D]) and rel(h[:, :D], R.rms_norm(xs[0, :T, :D].double(), g2[:D].double(), 1e-4)) < 2e-6


@pytest.mark.parametrize("T,F,ld", [(3, 40, 40), (5, 100, 104), (2, 93, 96), (1, 14336, 14336), (130, 1000, 1000), (2, 20004, 20008), (1, 1, 8)])
def test_poly_norm(T, F, ld):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(1)
    z = torch.full((T, ld), 1e3)                      # the padding must not count
    z[:, :F] = torch.randn(T, F, generator=g) * 2 + 0.3
    coef = torch.tensor([0.7, -0.4, 0.9, 0.25])
    want = R.poly_norm(z[:, :F].double(), coef.double(), 1e-4)
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 4e-3)):
        out = torch.full((T, ld), 7.0, dtype=dt, device=DEV)
        ops.poly_norm(z.to(DEV), F, coef.to(DEV), 1e-4, out)
        assert rel(out[:, :F].float(), want) < tol and not out[:, F:].any()
        zb = z.bfloat16()
        ops.poly_norm(zb.to(DEV), F, coef.to(DEV), 1e-4, out.fill_(7.0))
        assert rel(out[:, :F].float(), R.poly_norm(zb[:, :F].double(), coef.double(), 1e-4)) < tol and not out[:, F:].any()
    for k in range(4):                                # each of the four numbers on its own
        one = torch.zeros(4)
        one[k] = 1.5
        out = torch.empty(T, ld, device=DEV)
        ops.poly_norm(z.to(DEV), F, one.to(DEV), 1e-4, out)
        assert rel(out[:, :F], R.poly_norm(z[:, :F].double(), one.double(), 1e-4)) < 3e-6


def test_products_scaled_per_channel():
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(4)
    for M, N, K in ((1, 40, 72), (3, 136, 104), (70, 200, 136), (9, 64, 64), (130, 328, 72), (2, 256, 2048), (64, 512, 4096), (300, 260, 200)):
        a, w, x, ls = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g).bfloat16() * K ** -0.5, torch.randn(M, N, generator=g), torch.randn(N, generator=g)
        a16 = a.bfloat16()
        wd, lsd, st = w.to(DEV), ls.to(DEV), i32(0)
        xd = x.to(DEV)
        ops.gemm_f32(a.to(DEV), wd, xd, accumulate=True, col_scale=lsd)
        want = x.double() + ls.double() * (a.double() @ w.double().T)
        assert rel(xd, want) < 1e-6
        if M <= 8:
            xd = x.to(DEV)
            ops.matvec(ops.WT_BF16, wd, None, N, K, M, xf=a.to(DEV), epi=ops.EPI_RESID, resid=xd, y=xd, ldy=N, col_scale=lsd)
            assert rel(xd, want) < 1e-6
        for split in (0, 1):
            xd = x.to(DEV)
            ops.gemm_bf16(a16.to(DEV), wd, M, N, K, out_f32=xd, accumulate=True, split_k=split, col_scale=lsd, status=st)
            assert rel(xd, x.double() + ls.double() * (a16.double() @ w.double().T)) < 1e-5 and int(st.item()) == 0


# ---------------------------------------------------------------- mixture of experts
def expert_weights(E, F, K, g):
    W = {}
    for e in range(E):
        W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = ((torch.randn(*s, generator=g) * s[1] ** -0.5 * 2).bfloat16().double() for s in ((F, K), (F, K), (K, F)))
    W["router"] = (torch.randn(E, K, generator=g) * 2 * K ** -0.5).bfloat16().double()
    return W


def stacked(W, E, F, FP, K, KP):
    w13, w2, r = torch.zeros(E, FP, 2, KP), torch.zeros(E, KP, FP), torch.zeros(E, KP)
    for e in range(E):
        w13[e, :F, 0, :K], w13[e, :F, 1, :K], w2[e, :K, :F] = W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"]
    r[:, :K] = W["router"]
    return w13.bfloat16().view(-1, KP).to(DEV), w2.bfloat16().view(-1, FP).to(DEV), r.to(DEV)


MOE = [(5, 1, 40, 72), (12, 3, 36, 100), (64, 8, 96, 136), (1, 1, 16, 8), (7, 7, 24, 64), (200, 20, 8, 40)]


@pytest.mark.parametrize("E,top,F,K", MOE)
def test_router_takes_the_largest_sigmoids_as_they_are(E, top, F, K):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(E)
    KP, T = (K + 7) // 8 * 8, 33
    W = expert_weights(E, F, K, g)
    _, _, r = stacked(W, E, F, (F + 15) // 16 * 16, K, KP)
    h = torch.zeros(T, KP)
    h[:, :K] = torch.randn(T, K, generator=g).bfloat16().float()
    for x in (h.to(DEV), h.bfloat16().to(DEV)):
        ids, w = torch.full((T, top), -1, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        ops.moe_choose(x, r, top, ids, w, score=ops.SCORE_SIGMOID)
        e, s = R.route(h[:, :K].double(), W["router"], top)
        assert torch.equal(ids.cpu().long().sort(-1).values, e.sort(-1).values)
        assert rel(w, s) < 1e-6


@pytest.mark.parametrize("E,top,F,K", MOE)
def test_expert_products_of_few_tokens(E, top, F, K):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(E + 1)
    KP, FP = (K + 7) // 8 * 8, (F + 15) // 16 * 16
    W = expert_weights(E, F, K, g)
    w13, w2, r = stacked(W, E, F, FP, K, KP)
    ls = torch.zeros(KP)
    ls[:K] = torch.randn(K, generator=g)
    for T in (1, 2, 21):
        h, x = torch.zeros(T, KP), torch.zeros(T, KP)
        h[:, :K], x[:, :K] = torch.randn(T, K, generator=g), torch.randn(T, K, generator=g)
        hd, xd = h.to(DEV), x.to(DEV)
        ids, w = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        mid = torch.full((T, top, FP), float("nan"), device=DEV)
        ops.moe_choose(hd, r, top, ids, w, score=ops.SCORE_SIGMOID)
        ops.expert_gate_up(hd, w13, FP, ids, w, mid)
        ops.expert_down(mid, w2, KP, ids, xd, scale=ls.to(DEV))
        want = x[:, :K].double() + ls[:K].double() * R.expert_ff(h[:, :K].double(), W, "", top)
        assert rel(xd[:, :K], want) < 3e-6 and not xd[:, K:].any()


@pytest.mark.parametrize("E,top,F,K", MOE)
def test_expert_products_of_gathered_rows(E, top, F, K):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(E + 2)
    KP, FP = (K + 7) // 8 * 8, (F + 15) // 16 * 16
    W = expert_weights(E, F, K, g)
    w13, w2, r = stacked(W, E, F, FP, K, KP)
    ls = torch.zeros(KP)
    ls[:K] = torch.randn(K, generator=g)
    for T in (1, 40, 300):
        cap = (T + 127) // 128 * 128
        h, x = torch.zeros(T, KP), torch.zeros(T, KP)
        h[:, :K], x[:, :K] = torch.randn(T, K, generator=g).bfloat16().float(), torch.randn(T, K, generator=g)
        hd, xd, st = h.bfloat16().to(DEV), x.to(DEV), i32(0)
        rx, mid = torch.empty(E * cap, KP, dtype=torch.bfloat16, device=DEV), torch.empty(E * cap, FP, dtype=torch.bfloat16, device=DEV)
        meta, rw, cnt = torch.zeros(E * cap, 2, dtype=torch.int32, device=DEV), torch.zeros(E * cap, device=DEV), torch.zeros(E, dtype=torch.int32, device=DEV)
        ids, w = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        ops.moe_route_dispatch(hd, None, r, None, top, E, cap, rx.data_ptr(), meta.data_ptr(), rw.data_ptr(), cnt.data_ptr(), None, topk_ids=ids, topk_w=w, status=st,
                               score=ops.SCORE_SIGMOID)
        assert int(cnt.sum()) == T * top and torch.equal(cnt.cpu(), torch.bincount(ids.flatten().cpu(), minlength=E).to(torch.int32))
        ops.moe_gemm(rx, w13, E, cap, 2 * FP, KP, cnt, 1, out_bf16=mid, ldc=FP, gate_w=rw, status=st, live_rows=T * top)
        ops.moe_gemm(mid, w2, E, cap, KP, FP, cnt, 2, ldc=KP, meta=meta, sym_off=xd.data_ptr(), col_scale=ls.to(DEV), status=st, live_rows=T * top)
        want = ls[:K].double() * R.expert_ff(h[:, :K].double(), W, "", top)
        assert rel(xd[:, :K].cpu() - x[:, :K], want) < 8e-3 and not xd[:, K:].any() and int(st.item()) == 0


# ---------------------------------------------------------------- attention with mixed heads
def mixed(kernel, qs, ks, mix, scale, window, bias=None):
    """A batch through the projection finish and an attention kernel.  qs [T, H, dim] at each sequence's last positions, ks [S, G, dim]; the cache is
    filled by the finish kernel itself, all tokens first, then the queries' step."""
    from openagents_b200.ops import cuda_ops as ops
    H, dim, G, B = qs[0].shape[1], qs[0].shape[2], ks[0].shape[1], len(qs)
    tc = kernel in ("decode", "tc05")
    DK = (dim + 63) // 64 * 64 if tc else (dim + 7) // 8 * 8
    if tc and not (ops.mixed_decode_ok(H, G, DK) if kernel == "decode" else ops.mixed_prefill_ok(G, DK)):
        pytest.skip("sizes for the any-size kernel")
    dt = torch.float32 if kernel == "exact32" else torch.float16
    table, n_pages = pages_of([k.shape[0] for k in ks])
    kc = torch.zeros(n_pages, 1, 16, G * DK, dtype=dt, device=DEV)
    nq, nk = H * dim, G * dim
    bias = torch.zeros(nq + nk) if bias is None else bias
    rows = []
    for q, k in zip(qs, ks):
        S, T = k.shape[0], q.shape[0]
        full = torch.zeros(S, H, dim)
        full[S - T:] = q
        rows.append(torch.cat([full.reshape(S, -1), k.reshape(S, -1)], 1) - bias)
    row = torch.cat(rows).to(DEV)
    slot = torch.cat([slots_of(table, b, k.shape[0]) for b, k in enumerate(ks)]).to(torch.int32).to(DEV)
    last = torch.cat([torch.arange(k.shape[0]) >= k.shape[0] - q.shape[0] for q, k in zip(qs, ks)]).to(DEV)
    lens = [q.shape[0] for q in qs]
    T = sum(lens)
    starts, ctx, tab, st = i32(*[sum(lens[:b]) for b in range(B)]), i32(*[k.shape[0] for k in ks]), table.to(DEV), i32(0)
    slopes = (mix.double() @ R.slopes(H)).float().to(DEV)
    args = dict(window=window, sinks=torch.zeros(H, device=DEV), slopes=slopes)
    fin = lambda r, s, q: ops.mixed_finish(r, nq, bias.to(DEV), mix.to(DEV), scale, s, H, G, dim, DK, q, kc)      # noqa: E731
    fin(row, slot, torch.empty(row.shape[0], H * G * DK, device=DEV))
    out = torch.full((T, H * DK), 9.0, device=DEV)
    row, slot = row[last].contiguous(), slot[last].contiguous()
    if kernel == "decode":
        for S in (1, 3, 37):
            q32, before = torch.full((T, H * DK), 7.0, device=DEV), kc.clone()
            ops.qkv_finish(row, 0, nq, -1, slot, slot, None, 1.0, H, 1, dim, dim, DK, DK, 0, 1, False, 0.0, scale, 16, q32=q32, kc=kc, maps=G, bias=bias.to(DEV))
            assert torch.equal(kc, before)               # the very rows the other finish writes
            ops.mixed_decode(q32, kc, ops.mixed_decode_prepare(mix.to(DEV), slopes, H, G, DK), tab, ctx, B, H, G, DK, S=S, out_f32=out, status=st, window=window, sinks=args["sinks"],
                             scratch=torch.full((ops.mixed_decode_scratch_floats(B, H, G, DK, S),), float("nan"), device=DEV))
            assert S == 1 or (out.cpu() - first).abs().max() <= 2e-3 * first.abs().max()
            first = out.clone().cpu()
    elif kernel == "tc05":
        q16 = torch.full((T, H * G * DK), 7.0, dtype=torch.float16, device=DEV)
        fin(row, slot, q16)
        ops.mixed_prefill(q16, kc, slopes, tab, starts, i32(*lens), ctx, B, max(lens), H, G, DK, out_f32=out, status=st, window=window, sinks=args["sinks"])
        o16 = torch.zeros(T, H * DK, dtype=torch.bfloat16, device=DEV)
        ops.mixed_prefill(q16, kc, slopes, tab, starts, i32(*lens), ctx, B, max(lens), H, G, DK, out_bf16=o16, status=st, window=window, sinks=args["sinks"])
        assert torch.allclose(o16.float(), out, rtol=5e-3, atol=1e-6)
    else:
        q32 = torch.full((T, H * G * DK), 7.0, device=DEV)
        fin(row, slot, q32)
        ops.attn_exact(q32, kc, None, tab, starts, i32(*lens), ctx, B, max(lens), H, 1, DK, DK, out_f32=out, slices=G, **args)
    torch.cuda.synchronize()
    assert int(st.item()) == 0
    return out.view(T, H, DK)[..., :dim].cpu()


def want_mixed(qs, ks, mix, scale, window):
    return torch.cat([R.attention(q.double(), k.double(), mix.double(), scale, window, k.shape[0] - q.shape[0]) for q, k in zip(qs, ks)])


KERNELS = [("exact32", 2e-5), ("exact16", 3e-3), ("decode", 6e-3), ("tc05", 6e-3)]
SIZES = [(4, 2, 40), (6, 1, 64), (3, 3, 16), (20, 4, 56), (9, 3, 100), (1, 1, 8), (32, 8, 128), (16, 2, 128), (12, 6, 72), (40, 5, 64), (5, 5, 128), (64, 8, 64), (24, 1, 64), (48, 3, 96),
         (7, 7, 128), (6, 6, 128), (12, 12, 64), (17, 17, 40), (20, 20, 64)]


@pytest.mark.parametrize("kernel,tol", KERNELS)
@pytest.mark.parametrize("H,G,dim", SIZES)
@pytest.mark.parametrize("window", [1, 16, 50, 128, 1000])
def test_attention_with_mixed_heads(kernel, tol, H, G, dim, window):
    g = torch.Generator().manual_seed(2)
    f = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    if kernel == "tc05" and window == 1:
        tol = 1.2e-2                                    # every row sees one key: the same rounding everywhere
    shapes = [(1, 1), (1, 77), (1, 300), (1, 51), (1, 128), (1, 129)] if kernel == "decode" else [(1, 1), (3, 20), (64, 64), (130, 141), (1, 33), (200, 260)]
    qs, ks = [f(t, H, dim) for t, _ in shapes], [f(n, G, dim) for _, n in shapes]
    mix = (f(H, H) * 0.6 * H ** -0.5 + torch.eye(H)).bfloat16().float()          # what a checkpoint holds
    scale = 1.3 * dim ** -0.5
    got = mixed(kernel, qs, ks, mix, scale, window, f(H * dim + G * dim))
    assert rel(got, want_mixed(qs, ks, mix, scale, window)) < tol


@pytest.mark.parametrize("kernel", ["exact32", "decode", "tc05"])
@pytest.mark.parametrize("window", [17, 32, 48, 100, 128])
def test_a_window_starts_with_its_first_key(kernel, window):
    """One key stands out far above the others: a query whose window just holds it takes its value, the next one does not see it."""
    H, G, D = 4, 2, 64
    g = torch.Generator().manual_seed(3)
    qs, ks, inside = [], [], []
    mix = (torch.eye(H) + 0.1 * torch.randn(H, H, generator=g)).bfloat16().float()
    for at in (0, 1, 15, 16, 63, 64, 127, 128, 130):
        for far in (window - 1, window):                # the query's distance from the key
            n = at + far + 1
            k = torch.randn(n, G, D, generator=g) * 0.5
            k[..., 5] = 0
            k[at, :, 5] = 60.0
            q = torch.zeros(1, H, D)
            q[..., 5] = 1.0
            qs.append(q)
            ks.append(k)
            inside.append(far == window - 1)
    got, want = mixed(kernel, qs, ks, mix, 1.0, window), want_mixed(qs, ks, mix, 1.0, window)
    for i, (o, w) in enumerate(zip(got, want)):
        assert (o - w).abs().max() < 0.06 and (o[:, 5].min() > 50) == inside[i], i


@pytest.mark.parametrize("kernel", ["exact32", "decode", "tc05"])
def test_the_silent_sink_takes_its_share(kernel):
    """Scores far below zero leave nothing, scores of zero share with the sink, and it does not depend on how many keys are masked."""
    H, G, D = 4, 2, 64
    g = torch.Generator().manual_seed(6)
    for level in (-200.0, -5.0, 0.0, 5.0, 80.0):
        qs, ks = [], []
        for n in (1, 2, 16, 130):
            k = torch.randn(n, G, D, generator=g)
            k[..., 0] = 1.0
            q = torch.zeros(1, H, D)
            q[..., 0] = level
            qs.append(q)
            ks.append(k)
        got, want = mixed(kernel, qs, ks, torch.eye(H), 1.0, 40), want_mixed(qs, ks, torch.eye(H), 1.0, 40)
        assert torch.isfinite(got).all() and (got - want).abs().max() < 6e-3, level


# ---------------------------------------------------------------- whole models
L = R.layer
CONFIGS = {
    # odd sizes, a width and a vocabulary that are no multiples of eight and four, windows beside the page size, a layer without a feed-forward
    "odd": R.config([L(40, 6, 2, 24, ff=100), L(24, 4, 4, 7, ff=36, experts=5, top=2), L(16, 3, 1, 200, scale=0.4), L(56, 5, 5, 33, ff=44, experts=3, top=3)], width=100, vocab=131),
    # one head, many heads to a key head, a window of one token, one expert
    "few": R.config([L(64, 1, 1, 64, ff=96), L(32, 16, 1, 1, ff=64, experts=1), L(128, 4, 2, 100, ff=48, experts=9, top=4)], width=64, vocab=300, eps=1e-3),
    # heads and windows of a usual kind
    "usual": R.config([L(64, 12, 3, 80, ff=136), L(64, 12, 3, 48, ff=72, experts=10, top=1), L(128, 8, 4, 130, ff=64, experts=6, top=2), L(64, 16, 2, 96, ff=136)], width=128, vocab=260),
    # nothing is a multiple of anything
    "ragged": R.config([L(20, 7, 7, 50, ff=37), L(52, 9, 3, 31, ff=21, experts=7, top=5), L(101, 10, 2, 18, ff=75, scale=0.05)], width=93, vocab=127, eps=1e-2),
    # the head layouts of large models: slices of the queries on both sides of tensor memory, one and two score accumulators
    "heads": R.config([L(128, 32, 8, 150, ff=64), L(128, 20, 5, 60, ff=40, experts=4, top=2), L(64, 64, 8, 90), L(128, 14, 7, 130)], width=80, vocab=144),
    # more key heads than the tensor-core kernels take, head sizes beyond them
    "wide": R.config([L(136, 4, 2, 40, ff=72), L(72, 18, 18, 70, ff=40, experts=4, top=2), L(200, 2, 1, 96, ff=64)], width=96, vocab=264),
}


def model(name, dtype, seed):
    """A configuration and weights.  bf16 rounding may tip a router's close call, which no tolerance on logits covers: there every expert is used (the
    choice is held to the plain one in 32-bit, and by the router's own test)."""
    cfg = CONFIGS[name]
    if dtype == "bfloat16":
        every = lambda m: m if m is None or m["kind"] == "dense" else dict(m, router=dict(m["router"], top=m["router"]["experts"]))      # noqa: E731
        cfg = dict(cfg, layers=[dict(l, mlp=every(l["mlp"])) for l in cfg["layers"]])
    return cfg, R.random_weights(cfg, seed=seed)


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
    cfg, W = model(name, dtype, len(name))
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
@pytest.mark.parametrize("name", ["odd", "usual"])
def test_residual_after_every_layer(tmp_path, name, dtype):
    cfg, W = model(name, dtype, 2)
    toks = tokens(cfg, 70, 3)
    layers = []
    R.forward(cfg, W, toks, R.Sequence(), layers)
    e = open_model(tmp_path, cfg, W, dtype).engine
    runs = e.runs
    assert len(runs) == len(layers) == len(cfg["layers"])
    for n in range(1, len(runs) + 1):
        e.runs = runs[:n]
        e.begin(n)
        e.forward_tokens([n], [toks])
        assert rel(e.x[: len(toks), : cfg["width"]], layers[n - 1]) < TOL[dtype] / 2, n
        assert not e.x[: len(toks), cfg["width"]:].any()
        e.end(n)


@pytest.mark.parametrize("name", ["odd", "usual", "heads"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_reuse_pages(tmp_path, name, dtype):
    """Portions beside single tokens in any order, sequences left out of steps, and a pool so tight that pages come round again; each request's logits are those
    it has alone."""
    cfg, W = model(name, dtype, 5)
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


def test_stack_shares_prefixes_and_can_be_cut(tmp_path):
    cfg, W = model("odd", "float32", 6)
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
@pytest.mark.parametrize("name", ["odd", "usual"])
def test_long_decoding(tmp_path, name, dtype):
    """Every window passes over decoded tokens many times."""
    cfg, W = model(name, dtype, 7)
    be = open_model(tmp_path, cfg, W, dtype, max_ctx=700, max_tokens=64)
    toks = tokens(cfg, 500, 4)
    want = R.forward(cfg, W, toks, R.Sequence())
    be.begin(1, None)
    got = [run(be, 1, toks[:30], [30])]
    got += [be.forward_at([1], [[t]], [[0]]) for t in toks[30:]]
    close(torch.cat(got), want, dtype)


def far_key_model(dtype, window, G):
    """One layer whose first head looks for tokens that hold a mark: a marked token's key meets a query that only the second marked kind has, far above all other
    scores, so that the answer at such a token shows which keys the window holds."""
    H = 2 * G
    cfg = R.config([R.layer(64, H, G, window)], width=96, vocab=40)
    W = R.random_weights(cfg, seed=20)
    W["embed"][:, :2] = 0.0
    W["embed"][38, 0], W["embed"][39, 1] = 8.0, 8.0
    W["l0.norm1"][:2] = 1.0
    for n in ("q", "k"):
        W[f"l0.mix.{n}"][:, :2] = 0.0
    W["l0.mix.k"][5, 0] = 12.0                       # key head 0, dimension 5: the mark
    W["l0.mix.q"][5, 1] = 12.0                       # query head 0 of whoever asks
    W["l0.mix.talk"] = torch.eye(H, dtype=torch.float64)
    return cfg, {k: v.to(torch.bfloat16).double() for k, v in W.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [17, 64, 100])
def test_far_keys_at_the_edges_of_pages_and_windows(tmp_path, window, dtype):
    """A marked key just inside and just outside the window of the token that asks for it, at page borders, asked for in prompts, in short portions and in decoding."""
    cfg, W = far_key_model(dtype, window, 2)
    be = open_model(tmp_path, cfg, W, dtype, max_ctx=400, max_tokens=400)
    seq = 0
    for at in (0, 1, 15, 16, 31, 63, 64, 127, 128):
        for far in (window - 2, window - 1, window):
            toks = [int(t) % 38 for t in tokens(cfg, at + far + 1, 30 + at)]
            toks[at], toks[at + far] = 38, 39
            want = R.forward(cfg, W, toks, R.Sequence())
            plain = R.forward(cfg, W, toks[:at] + [0] + toks[at + 1:], R.Sequence())
            shows = (want[-1] - plain[-1]).abs().max() > 0.5 * want.std()
            assert shows == (far < window)           # the key shows exactly inside the window
            for cuts in ([len(toks)], [len(toks) - 1, 1], [max(1, len(toks) - 2), 2]):
                seq += 1
                be.begin(seq, None)
                close(run(be, seq, toks, cuts)[-1:], want[-1:], dtype)
                be.end(seq)


@pytest.mark.parametrize("name", ["odd", "usual", "few"])
def test_decode_batches_of_every_path(tmp_path, name):
    """Decode batches for the mat-vec path, the one-tile GEMM and beyond it (bf16), each sequence against itself alone."""
    cfg, W = model(name, "bfloat16", 9)
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


@pytest.mark.parametrize("name", ["odd", "few", "usual"])
def test_greedy_generation_through_the_scheduler(tmp_path, name):
    """Continuous batching end to end in the 32-bit mode: the ids are the plain implementation's."""
    from openagents_b200.serve.generation import SamplingParams, Scheduler

    class Tok:
        eos_id = -1

        def decode(self, ids):
            return ""
    cfg, W = model(name, "float32", 11)
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generate_and_device_side_decode_loop(tmp_path, dtype):
    cfg, W = model("usual", dtype, 12)
    be = open_model(tmp_path, cfg, W, dtype)
    prompt = tokens(cfg, 25, 6)
    ids, rows = R.generate(cfg, W, prompt, 10)
    for graph in (False, True):
        out, logits = be.engine.generate(prompt, 10, seq_id=int(graph), use_graph=graph)
        if dtype == "float32":
            assert out == ids
        n = next((t for t, (a, b) in enumerate(zip(out, ids)) if a != b), len(ids) - 1) + 1      # the same tokens up to here
        close(logits[:n], rows[:n], dtype)
        be.end(int(graph))
    be.begin(5, None)
    _, nxt = be.engine.forward_tokens([5], [prompt])
    first = int(nxt[0])
    hist = be.engine.decode_steps([5], [first], 9)
    assert [first] + hist[:, 0].tolist() == out


@pytest.mark.parametrize("name", ["odd", "usual", "wide", "heads", "ragged"])
def test_workspace_canaries(tmp_path, name):
    for dtype in ("float32", "bfloat16"):
        cfg, W = model(name, dtype, 13)
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
    cfg, W = model("odd", "float32", 14)
    be = open_model(tmp_path, cfg, W)
    src = open_source(str(tmp_path / "m"), "cpu")
    path = str(tmp_path / "m.gguf")
    save_gguf(path, src.cfg, {k: v.float() for k, v in W.items()}, PLAN_BF16)
    be2 = CudaBackend.open(path, max_num_seqs=4, max_ctx=128, max_tokens=128, dtype="float32")
    assert be2.cfg.layers == src.cfg.layers
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
    ta, tb = [t % 131 for t in tokens(CONFIGS["odd"], 40, 1)], tokens(CONFIGS["odd"], 21, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:20], "want": []}, {"id": "a", "tokens": ta[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ta[31:], "want": [8]}, {"id": "b", "tokens": tb[20:], "want": [0]}], "end": ["a", "b"]}]
    for dtype in ("float32", "bfloat16"):
        cfg, W = model("odd", dtype, 15)
        folder = R.save_model(str(tmp_path / dtype), cfg, W)
        out = tmp_path / ("out-" + dtype)
        out.mkdir()
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
    a = parse_args(["-m", R.save_model(str(tmp_path / "tiny-kazolorn"), cfg, W), "--dtype", "float32", "--max-num-seqs", "2", "--max-ctx", "512",
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
        out = post("/v1/completions", {"model": "tiny-kazolorn", "prompt": "hello there", "max_tokens": 8, "temperature": 0})
        ids, _ = R.generate(cfg, W, list(b"hello there"), 8)
        stop = ids.index(256) if 256 in ids else len(ids)
        assert out["choices"][0]["text"] == bytes(i for i in ids[:stop] if i < 256).decode("utf-8", "replace")
    finally:
        httpd.shutdown()
        for m in state.models.values():
            m.close()


def test_a_window_of_the_plain_kernels(tmp_path):
    """The same mechanisms without mixed heads: windows, silent sinks and values that are the keys on the other attention kernels, the distance bias on the
    any-size one (the mixer as another design would configure it)."""
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(9)
    H, G, D, window = 12, 4, 64, 40
    lens, ctx = [1, 30, 70, 1], [77, 30, 141, 33]
    table, n_pages = pages_of(ctx)
    kc = torch.zeros(n_pages, G, 16, D, dtype=torch.float16, device=DEV)
    ks = [torch.randn(n, G, D, generator=g).half() for n in ctx]
    for b, k in enumerate(ks):
        for n in range(ctx[b]):
            kc[int(table[b, n // 16]), :, n % 16] = k[n].to(DEV)
    qs = [torch.randn(t, H, D, generator=g) * D ** -0.5 for t in lens]
    q, starts = torch.cat(qs).to(DEV), i32(*[sum(lens[:b]) for b in range(4)])
    zero, sl = torch.zeros(H, device=DEV), R.slopes(H).float().to(DEV)

    def want(bias):
        out = []
        for a, k in zip(qs, ks):
            T, S = a.shape[0], k.shape[0]
            s = R.raw_scores(a.double(), k.double(), 1.0)
            s = R.distance_bias(s, S - T) if bias else s
            p = R.weights_with_silent_sink(s, R.visible(S - T, T, S, window))
            out.append(torch.stack([p[h] @ k[:, h // (H // G)].double() for h in range(H)], 1))
        return torch.cat(out)
    tab, st, T = table.to(DEV), i32(0), sum(lens)
    out = torch.empty(T, H * D, device=DEV)
    ops.attn_prefill_tc05(q.half().view(T, -1), kc, kc, tab, starts, i32(*lens), i32(*ctx), 4, max(lens), H, G, window=window, sinks=zero, out_f32=out, status=st, dk=D, dv=D)
    assert rel(out.view(T, H, D), want(False)) < 6e-3
    for bias in (False, True):
        ops.attn_exact(q.view(T, -1), kc, kc, tab, starts, i32(*lens), i32(*ctx), 4, max(lens), H, G, D, D, out_f32=out, window=window, sinks=zero, slopes=sl if bias else None)
        assert rel(out.view(T, H, D), want(bias)) < 1e-5
    last = [sum(lens[: b + 1]) - 1 for b in range(4)]
    ops.attn_decode(q[last].contiguous().view(4, -1), kc, kc, tab, i32(*ctx), 4, H, G, D, window=window, S=1, sinks=zero, out_f32=out, status=st)
    assert rel(out[:4].view(4, H, D), want(False)[last]) < 6e-3 and int(st.item()) == 0
