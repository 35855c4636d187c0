"""Folirax on the GPU: every mechanism alone and whole models against the plain implementation in ``folirax_ref``."""
import math

import pytest
import torch

import folirax_ref as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 3e-5, "bfloat16": 0.04}


def rel(got, want):
    """RMS of the difference over the spread of the wanted values."""
    got, want = got.detach().cpu().double(), want.double()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()).item()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- mechanisms
def test_norm_on_both_sides_of_a_sublayer():
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(0)
    for T, D, ld in ((3, 72, 72), (5, 100, 104), (4, 93, 96), (2, 2048, 2048), (3, 4096, 4096), (2, 4100, 4104), (1, 9000, 9000)):
        x, y = torch.randn(T, D, generator=g), torch.randn(T, ld, generator=g) * 3
        gy, gh = 1 + 0.3 * torch.randn(D, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
        want_x = x.double() + R.centred_norm(y[:, :D].double(), gy.double() - 1, 1e-3)
        want_h = R.centred_norm(want_x, gh.double() - 1, 1e-3)
        xd, yd = x.to(DEV), y.to(DEV)
        hf, side = torch.full((T, ld), 7.0, device=DEV), torch.ones(64, device=DEV)
        ops.norm_residual(xd, 1e-3, y=yd, gy=gy.to(DEV), gh=gh.to(DEV), hf=hf, y_clear=True, zero=side)
        assert rel(xd, want_x) < 1e-6 and rel(hf[:, :D], want_h) < 1e-6
        assert not hf[:, D:].any() and not yd.any() and not side.any()
        hb = torch.full((T, ld), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.norm_residual(xd, 1e-3, gh=gh.to(DEV), hb=hb)
        assert rel(hb[:, :D].float(), want_h) < 4e-3 and not hb[:, D:].any()


@pytest.mark.parametrize("style", [0, 1])
def test_rotation_then_unit_norm_then_cache(style):
    """Partial rotation, unit-RMS queries and keys, the padded cache rows, and a layer without keys of its own."""
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(1)
    for H, G, dim, vdim, DK, DV, rot in ((6, 2, 40, 24, 64, 64, 16), (4, 4, 104, 56, 104, 56, 104), (2, 1, 10, 6, 16, 8, 2), (3, 1, 72, 130, 72, 136, 0)):
        T = 5
        ld = H * dim + G * (dim + vdim) + 3
        row = torch.randn(T, ld, generator=g)
        pos, pages = i32(0, 1, 15, 16, 900), 8
        slot = i32(16 * 3 + 1, 0, 16 * 7 + 15, -1, 16 * 2)
        table = ops.rope_table(17, rot, 500.0, DEV) if rot else None      # 900 lies outside: computed on the spot
        for dt in (torch.float16, torch.float32):
            kc, vc = torch.full((pages, G, 16, DK), 3.0, dtype=dt, device=DEV), torch.full((pages, G, 16, DV), 3.0, dtype=dt, device=DEV)
            q32, q16 = torch.full((T, H, DK), 5.0, device=DEV), torch.full((T, H, DK), 5.0, dtype=torch.float16, device=DEV)
            k_off, v_off = H * dim, H * dim + G * dim
            ops.qkv_finish(row.to(DEV), 0, k_off, v_off, pos, slot, table, 500.0, H, G, dim, vdim, DK, DV, rot, style, True, 1e-4, 0.25, 16,
                           q32=q32, q16=q16, kc=kc, vc=vc)

            def turn(x):
                if style == 1 and rot:       # halves layout = the pairs layout after a permutation
                    perm = [i // 2 + (i % 2) * (rot // 2) for i in range(rot)] + list(range(rot, dim))
                    inv = [perm.index(i) for i in range(dim)]
                    return R.rotate(x[..., perm], pos.cpu(), rot, 500.0)[..., inv]
                return R.rotate(x, pos.cpu(), rot, 500.0)
            q = R.rms(turn(row[:, :k_off].double().view(T, H, dim)), 1e-4) * 0.25
            k = R.rms(turn(row[:, k_off:v_off].double().view(T, G, dim)), 1e-4)
            v = row[:, v_off: v_off + G * vdim].double().view(T, G, vdim)
            assert rel(q32[..., :dim], q) < 1e-6 and not q32[..., dim:].any()
            assert rel(q16[..., :dim].float(), q) < 1e-3 and not q16[..., dim:].any()
            eps = 1e-6 if dt == torch.float32 else 1e-3
            for t, s in enumerate(slot.tolist()):
                if s >= 0:
                    assert rel(kc[s // 16, :, s % 16, :dim].float(), k[t]) < eps and not kc[s // 16, :, s % 16, dim:].any()
                    assert rel(vc[s // 16, :, s % 16, :vdim].float(), v[t]) < eps and not vc[s // 16, :, s % 16, vdim:].any()
            untouched = torch.ones(pages * 16, dtype=torch.bool)
            untouched[[s for s in slot.tolist() if s >= 0]] = False
            assert (kc.transpose(1, 2).reshape(pages * 16, -1)[untouched] == 3.0).all()
            before = kc.clone()
            ops.qkv_finish(row.to(DEV), 0, -1, -1, pos, slot, table, 500.0, H, G, dim, vdim, DK, DV, rot, style, True, 1e-4, 0.25, 16, q32=q32,
                           kc=kc, vc=vc)
            assert torch.equal(before, kc) and rel(q32[..., :dim], q) < 1e-6


ATTN = [(6, 2, 64, 64), (1, 1, 128, 128), (5, 1, 128, 64), (12, 12, 64, 128), (20, 1, 64, 64), (9, 1, 128, 128), (14, 2, 192, 128), (4, 4, 256, 64)]


def _paged(ks, vs, dt, DK, DV):
    """Scatter sequences' keys and values over shuffled pages; returns caches, page table, lengths."""
    G = ks[0].shape[1]
    need = [(k.shape[0] + 15) // 16 for k in ks]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(5)).tolist()
    kc, vc = torch.zeros(len(perm), G, 16, DK, dtype=dt), torch.zeros(len(perm), G, 16, DV, dtype=dt)
    table = torch.zeros(len(ks), max(need), dtype=torch.int32)
    for b, (k, v) in enumerate(zip(ks, vs)):
        for j in range(need[b]):
            pg = perm.pop()
            table[b, j] = pg
            kk, vv = k[16 * j: 16 * j + 16], v[16 * j: 16 * j + 16]
            kc[pg, :, : len(kk), : k.shape[2]] = kk.transpose(0, 1).to(dt)
            vc[pg, :, : len(vv), : v.shape[2]] = vv.transpose(0, 1).to(dt)
    return kc.to(DEV), vc.to(DEV), table.to(DEV), i32(*[k.shape[0] for k in ks])


def _attend(kernel, qs, ks, vs, gates, DK, DV):
    """One batch through a kernel; q [T, H, dim] of each sequence stands at its last T positions."""
    from openagents_b200.ops import cuda_ops as ops
    H, G, B = qs[0].shape[1], ks[0].shape[1], len(qs)
    dt = torch.float32 if kernel == "exact32" else torch.float16
    kc, vc, table, ctx = _paged(ks, vs, dt, DK, DV)
    lens = [q.shape[0] for q in qs]
    starts = [sum(lens[:b]) for b in range(B)]
    T = sum(lens)
    q = torch.zeros(T, H, DK)
    q[..., : qs[0].shape[2]] = torch.cat(qs)
    gate = torch.cat(gates).to(DEV)
    st = i32(0)
    if kernel == "decode":
        S = 3
        out = torch.empty(T, H * DV, device=DEV)
        ops.attn_decode(q.to(DEV).view(T, -1), kc, vc, table, ctx, B, H, G, DK, dv=DV, S=S, gate=gate, out_f32=out,
                        scratch=torch.empty(ops.attn_decode_scratch_floats(B, H, G, DV, S), device=DEV),
                        counters=torch.zeros(B * H, dtype=torch.int32, device=DEV), status=st)
    elif kernel == "tc05":
        out = torch.empty(T, H * DV, dtype=torch.bfloat16, device=DEV)
        ops.attn_prefill_tc05(q.to(DEV).half().view(T, -1), kc, vc, table, i32(*starts), i32(*lens), ctx, B, max(lens), H, G, out_bf16=out,
                              status=st, dk=DK, dv=DV, gate=gate)
    else:
        out = torch.empty(T, H * DV, device=DEV)
        ops.attn_exact(q.to(DEV).view(T, -1), kc, vc, table, i32(*starts), i32(*lens), ctx, B, max(lens), H, G, DK, DV, gate=gate, out_f32=out)
    torch.cuda.synchronize()
    assert int(st.item()) == 0
    return out.float().view(T, H, DV)


def _want(qs, ks, vs, gates):
    return torch.cat([R.softmax_attention(q.double(), k.double(), v.double(), 1.0, k.shape[0] - q.shape[0]) * torch.sigmoid(g.double())[..., None]
                      for q, k, v, g in zip(qs, ks, vs, gates)])


@pytest.mark.parametrize("kernel,tol", [("exact32", 1e-5), ("exact16", 1e-3), ("decode", 2e-3), ("tc05", 6e-3)])
@pytest.mark.parametrize("H,G,DK,DV", ATTN)
def test_gated_attention(kernel, tol, H, G, DK, DV):
    g = torch.Generator().manual_seed(2)
    dim, vdim = DK - 8, DV - 16                        # padded columns
    one = kernel == "decode"
    shapes = [(1, 1), (1, 77), (1, 300)] if one else [(1, 1), (3, 20), (64, 64), (130, 141), (1, 33), (200, 200)]
    f = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    qs, ks = [f(t, H, dim) * dim ** -0.5 for t, _ in shapes], [f(n, G, dim) for _, n in shapes]
    vs, gates = [f(n, G, vdim) for _, n in shapes], [f(t, H) for t, _ in shapes]
    got = _attend(kernel, qs, ks, vs, gates, DK, DV)
    assert rel(got[..., :vdim], _want(qs, ks, vs, gates)) < tol
    assert not got[..., vdim:].any()


@pytest.mark.parametrize("kernel", ["exact32", "decode", "tc05"])
def test_one_key_stands_out_wherever_it_lies(kernel):
    """A query aligned with one key far back (page and tile borders, the first tokens, itself) and with the key just behind it, which
    it must not see: the output is that key's value."""
    H, G, D, n = 2, 1, 64, 300
    g = torch.Generator().manual_seed(3)
    places = [0, 1, 15, 16, 17, 31, 63, 64, 127, 128, 129, 255, 256, 298]
    qs, ks, vs, gates, want = [], [], [], [], []
    for p in places:
        k, v = torch.randn(n, G, D, generator=g), torch.randn(n, G, D, generator=g)
        q = torch.randn(n - p if kernel != "decode" else 1, H, D, generator=g) * 0.05
        k[p, 0] = 0
        k[p, 0, p % D] = 40.0
        q[-1] = 0
        q[-1, :, p % D] = 1.0
        if kernel != "decode":                           # the row just ahead of the key: aligned with it, but it lies in its future
            q[0, :, p % D] = 1.0
            k[p + 1:, 0, p % D] = 80.0
            k[p + 1:, 0, (p + 1) % D] = 0
            q[-1] = 0
            q[-1, :, (p + 1) % D] = 1.0
            k[p, 0, (p + 1) % D] = 60.0
        qs.append(q)
        ks.append(k)
        vs.append(v)
        gates.append(torch.zeros(q.shape[0], H))
        want.append(v[p, 0] * 0.5)
    got = _attend(kernel, qs, ks, vs, gates, D, D).cpu()
    at = 0
    for q, w, p in zip(qs, want, places):
        assert (got[at + len(q) - 1] - w).abs().max() < 0.02, p
        if kernel != "decode":
            assert (got[at] - w).abs().max() < 0.02, p
        at += len(q)


def _gla_case(T_list, pos_list, H, dim, vdim, rank, tau, z_shift, seed=0, z_scale=1.0):
    """A batch for the linear-attention kernels: fused rows, weights, states; returns everything plus the plain result."""
    g = torch.Generator().manual_seed(seed)
    VP = (vdim + 7) // 8 * 8
    T = sum(T_list)
    qk, vv = H * dim, H * vdim
    offs = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
    ld = (2 * qk + 2 * vv + rank + 7) // 8 * 8
    row = torch.randn(T, ld, generator=g)
    row[:, offs[2]: offs[3]] = row[:, offs[2]: offs[3]].bfloat16().float()       # v is exact in bf16: the rest is what is measured
    a2 = torch.randn(H * dim, rank, generator=g) * z_scale * rank ** -0.5
    b2 = torch.randn(H * dim, generator=g) + z_shift
    w = 1 + 0.2 * torch.randn(vdim, generator=g)
    slots = torch.randperm(len(T_list) + 2, generator=g)[: len(T_list)].to(torch.int32)
    state = torch.randn(len(T_list) + 2, H, dim, VP, generator=g)
    state[..., vdim:] = 0
    want, want_state, at = [], state.clone().double(), 0
    for n, p0, s in zip(T_list, pos_list, slots.tolist()):
        r = row[at: at + n].double()
        at += n
        q = r[:, :qk].view(n, H, dim) * dim ** -0.5
        k, v = r[:, qk: 2 * qk].view(n, H, dim), r[:, offs[2]: offs[3]].view(n, H, vdim)
        gl = torch.nn.functional.logsigmoid(r[:, offs[4]: offs[4] + rank] @ a2.double().T + b2.double()) / tau
        S0 = state[s, :, :, :vdim].double() if p0 else torch.zeros(H, dim, vdim, dtype=torch.float64)
        o, S = R.gla_recurrence(q, k, v, gl.view(n, H, dim), S0)
        want_state[s, :, :, :vdim] = S
        want_state[s, :, :, vdim:] = 0
        want.append(R.rms(o, 1e-5) * w.double() * torch.nn.functional.silu(r[:, offs[3]: offs[4]].view(n, H, vdim)))
    d = lambda x: x.to(DEV).contiguous()        # noqa: E731
    starts = [sum(T_list[:b]) for b in range(len(T_list))]
    args = (d(row), offs, rank, d(a2.T), d(b2), d(w), d(state), i32(*starts), i32(*T_list), i32(*[a + b for a, b in zip(T_list, pos_list)]),
            d(slots), len(T_list), H, dim, vdim, VP, tau, dim ** -0.5, 1e-5)
    return args, VP, torch.cat(want), want_state, args[6], slots


GLA_SIZES = [(3, 32, 56, 12), (4, 128, 256, 16), (2, 24, 40, 5), (1, 128, 72, 20), (5, 64, 8, 1), (2, 160, 136, 33), (1, 256, 64, 16)]


@pytest.mark.parametrize("kind", ["recurrent", "chunked"])
@pytest.mark.parametrize("H,dim,vdim,rank", GLA_SIZES)
@pytest.mark.parametrize("tau,shift,scale", [(16.0, 0.0, 1.0), (1.0, 20.0, 1.0), (1.0, -30.0, 3.0), (4.0, -4.0, 8.0)])
def test_gated_linear_attention(kind, H, dim, vdim, rank, tau, shift, scale):
    """Mild decays, none, total forgetting and mixtures; fresh and continued sequences of unequal length, chunk edges."""
    from openagents_b200.ops import cuda_ops as ops
    lens, pos = [1, 63, 64, 65, 130, 2], [0, 7, 0, 64, 0, 1000]
    args, VP, want, want_state, state, slots = _gla_case(lens, pos, H, dim, vdim, rank, tau, shift, z_scale=scale)
    T = sum(lens)
    out = torch.full((T, H * VP), 9.0, device=DEV)
    if kind == "recurrent":
        ops.gla_recurrent(*args, out_f32=out)
    else:
        n = ops.gla_chunk_bytes(T, len(lens), H, dim, VP, rank)
        assert n > 0
        ops.gla_chunked(*args, max(lens), torch.empty(n, dtype=torch.uint8, device=DEV), out_f32=out)
    torch.cuda.synchronize()
    out = out.view(T, H, VP)
    tol = 2e-5 if kind == "recurrent" else 2e-4        # the chunked operands carry 16 bits of mantissa
    assert torch.isfinite(out).all() and not out[..., vdim:].any()
    at = 0
    for n in lens:
        assert rel(out[at: at + n, :, :vdim], want[at: at + n]) < tol, n
        at += n
    assert rel(state, want_state) < tol


def test_linear_attention_without_a_slot_keeps_nothing():
    from openagents_b200.ops import cuda_ops as ops
    args, VP, _, _, state, _ = _gla_case([1, 1], [5, 0], 2, 32, 16, 4, 16.0, 0.0)
    before = state.clone()
    out = torch.empty(2, 2 * VP, device=DEV)
    ops.gla_recurrent(*args[:10], i32(-1, -1), *args[11:], out_f32=out)
    torch.cuda.synchronize()
    assert torch.equal(before, state) and torch.isfinite(out).all()


def test_products_and_squared_relu():
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(4)
    for M, N, K in ((1, 40, 72), (3, 136, 104), (70, 200, 136), (9, 64, 64), (130, 328, 72)):
        a, w = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g).bfloat16()
        want = R.relu2_ff(a.double(), {"up": w.double(), "down": torch.eye(N, dtype=torch.float64)}, "")
        out = torch.empty(M, N, device=DEV)
        ops.gemm_f32(a.to(DEV), w.to(DEV), out, act=1)
        assert rel(out, want) < 1e-6
        if M <= 8:
            ops.matvec(ops.WT_BF16, w.to(DEV), None, N, K, M, xf=a.to(DEV), epi=ops.EPI_RELU2, y=out, ldy=N)
            assert rel(out, want) < 1e-6
        ob, st = torch.empty(M, N, dtype=torch.bfloat16, device=DEV), i32(0)
        ops.gemm_bf16(a.bfloat16().to(DEV), w.to(DEV), M, N, K, out_bf16=ob, act=ops.ACT_RELU2, status=st)
        want16 = R.relu2_ff(a.bfloat16().double(), {"up": w.double(), "down": torch.eye(N, dtype=torch.float64)}, "")
        assert rel(ob.float(), want16) < 4e-3 and int(st.item()) == 0


def test_scaled_and_capped_logits():
    from openagents_b200.ops import cuda_ops as ops
    x = torch.randn(3, 1001, generator=torch.Generator().manual_seed(0)) * 40
    for scale, cap in ((0.5, 30.0), (2.0, 0.0), (1.0, 3.0)):
        y = x.to(DEV).clone()
        ops.logits_finish(y, scale, cap)
        want = x.double() * scale
        assert rel(y, cap * torch.tanh(want / cap) if cap else want) < 1e-6


# ---------------------------------------------------------------- whole models
A, L = R.layer_attention, R.layer_gla
CONFIGS = {
    # odd sizes, groups of three, shared keys, a vocabulary that is no multiple of four
    "odd": R.config([L(24, 40, 3, tau=8.0), A(40, 24, 6, 2, 16, ff=100), L(24, 40, 3, tau=8.0, ff=36), A(40, 24, 6, 2, 16, kv_from=1, scale=0.3)],
                    width=72, vocab=131),
    # everything rotates, one kv head, keys shared twice, feed-forwards everywhere
    "attention": R.config([A(64, 64, 4, 1, 64, base=1000.0, ff=96), A(64, 64, 4, 1, 64, base=1000.0, kv_from=0, scale=1.0), A(96, 80, 5, 5, 32, ff=64),
                           A(64, 64, 8, 1, 64, base=1000.0, kv_from=0, ff=40)], width=100, vocab=260, eps=1e-4),
    "recurrent": R.config([L(20, 16, 5, tau=1.0), L(48, 128, 2, tau=4.0, ff=64), L(144, 64, 3)], width=64, vocab=300, logit_scale=1.0),
    # head sizes beyond the tensor-core kernels, no rotation
    "wide": R.config([A(264, 136, 2, 1, 0, ff=72), L(264, 24, 2, ff=64), A(128, 192, 2, 2, 48)], width=128, vocab=264, softcap=8.0),
}


def open_model(tmp_path, cfg, W, dtype="float32", max_num_seqs=4, max_ctx=512, max_tokens=512, **kw):
    from openagents_b200.serve.backend import CudaBackend
    kw.setdefault("state_slots", max_num_seqs)
    return CudaBackend.open(R.save_model(str(tmp_path / "m"), cfg, W), max_num_seqs=max_num_seqs, max_ctx=max_ctx, max_tokens=max_tokens,
                            dtype=dtype, **kw)


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
    if name == "odd":
        be.begin(9, None)                  # token by token from the first
        close(run(be, 9, toks[:40], [1]), want[:40], dtype)


def test_residual_after_every_layer(tmp_path):
    """The residual stream itself (both modes), cut to the first layers one by one."""
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=2)
    toks = tokens(cfg, 70, 3)
    layers = []
    R.forward(cfg, W, toks, R.Sequence(), layers)
    for n in range(1, len(cfg["layers"]) + 1):
        for dtype in ("float32", "bfloat16"):
            be = open_model(tmp_path / f"{n}{dtype}", dict(cfg, layers=cfg["layers"][:n]), W, dtype)
            be.begin(1, None)
            be.engine.forward_tokens([1], [toks])
            assert rel(be.engine.x[: len(toks)], layers[n - 1]) < TOL[dtype] / 3, (n, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_reuse_pages_and_slots(tmp_path, dtype):
    """Portions beside single tokens, sequences left out of steps, and a pool so tight that pages and slots come round again; each
    request's logits are those it has alone."""
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=5)
    be = open_model(tmp_path, cfg, W, dtype, max_num_seqs=3, n_pages=24, max_ctx=24 * 16, max_tokens=24 * 16)
    want, toks = {}, {}
    for r, n in enumerate((120, 33, 97, 64, 5, 140, 18)):
        toks[r] = tokens(cfg, n, 10 + r)
        want[r] = R.forward(cfg, W, toks[r], R.Sequence())
    g = torch.Generator().manual_seed(8)
    queue, live, at, got, seq = list(toks), [], {}, {r: [] for r in toks}, {}
    nxt = 100
    while queue or live:
        while queue and len(live) < 3 and sum((len(toks[r]) + 15) // 16 for r in live + queue[:1]) <= 24:
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
    st = be.kv_stats()
    assert st["pages_free"] == 24 and st["state_slots_free"] == st["state_slots_total"] == 3


def test_slots_run_out_and_come_back(tmp_path):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=5)
    be = open_model(tmp_path, cfg, W, max_num_seqs=2)
    be.begin(1, None)
    be.begin(2, None)
    with pytest.raises(MemoryError):
        be.begin(3, None)
    toks = tokens(cfg, 20, 1)
    be.forward_at([1, 2], [toks, toks[:7]], [[], []])
    be.end(1)
    be.begin(3, None)
    close(run(be, 3, toks, [20]), R.forward(cfg, W, toks, R.Sequence()), "float32")
    with pytest.raises(ValueError):
        be.truncate(3, 10)                 # a recurrent state cannot be cut
    be.truncate(3, 0)
    close(run(be, 3, toks, [9]), R.forward(cfg, W, toks, R.Sequence()), "float32")
    assert not be.supports_verify


def test_attention_only_stack_shares_prefixes_and_can_be_cut(tmp_path):
    cfg = CONFIGS["attention"]
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
    assert be.supports_verify


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


def test_decode_batches_of_every_path(tmp_path):
    """Decode batches for the mat-vec path, the one-tile GEMM and beyond it (bf16), each sequence against itself alone."""
    cfg = CONFIGS["odd"]
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


@pytest.mark.parametrize("name", ["odd", "recurrent", "attention"])
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
                assert (top[0] - top[1]).item() < 1e-4, t
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


def test_workspace_canaries(tmp_path):
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=13)
    for dtype in ("float32", "bfloat16"):
        be = open_model(tmp_path / dtype, cfg, W, dtype, canaries=True, max_tokens=203)
        toks = tokens(cfg, 203, 1)
        be.begin(1, None)
        close(run(be, 1, toks, [100, 1, 64, 1]), R.forward(cfg, W, toks, R.Sequence()), dtype)
        assert be.engine.check_canaries() == []


def test_random_source_and_gguf_round_trip(tmp_path):
    """The design through the framework's other ways in: a GGUF file written by the framework gives the folder's logits."""
    from openagents_b200.models.registry import open_source
    from openagents_b200.models.weights import PLAN_BF16, save_gguf
    from openagents_b200.serve.backend import CudaBackend
    cfg = CONFIGS["odd"]
    W = R.random_weights(cfg, seed=14)
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
    assert math.isfinite(be2.score(1, toks[:8], toks[1:9])[0])


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
    """The server as `b200-serve -m FOLDER --dtype float32` builds it: completions, sessions beyond the state slots (idle ones give
    theirs up), log-probabilities, and the answer of the plain implementation."""
    import json
    import threading
    import urllib.request

    from openagents_b200.serve.server import build_state, parse_args, serve
    cfg = dict(CONFIGS["recurrent"], vocab=300)
    W = R.random_weights(cfg, seed=16)
    a = parse_args(["-m", R.save_model(str(tmp_path / "tiny-folirax"), cfg, W), "--dtype", "float32", "--max-num-seqs", "2", "--max-ctx", "512",
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
        rows = json.loads(urllib.request.urlopen(base + "/v1/models", timeout=30).read())["data"]
        assert [m["id"] for m in rows] == ["tiny-folirax"]
        out = post("/v1/completions", {"model": "tiny-folirax", "prompt": "hello there", "max_tokens": 8, "temperature": 0})
        ids, _ = R.generate(cfg, W, list(b"hello there"), 8)
        stop = ids.index(256) if 256 in ids else len(ids)
        assert out["choices"][0]["text"] == bytes(i for i in ids[:stop] if i < 256).decode("utf-8", "replace")
        slots = state.models["tiny-folirax"].backend.kv_stats()["state_slots_total"]
        for _ in range(slots + 3):
            sid = post("/v1/sessions", {"model": "tiny-folirax"})["id"]
            assert "output_text" in post(f"/v1/sessions/{sid}/responses", {"prompt": "again", "max_tokens": 3})
        assert state.sessions_evicted > 0
    finally:
        httpd.shutdown()
        for m in state.models.values():
            m.close()
