"""Tekosun on the GPU: every mechanism alone and whole models against the plain implementation in ``tekosun_ref``."""
import math

import pytest
import torch

import tekosun_ref as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.04}
DECAY = math.exp(-0.5)


def rel(got, want):
    """RMS of the difference over the spread of the wanted values."""
    got, want = got.detach().cpu().double(), want.double()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()).item()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- residual step, embedding, norms
@pytest.mark.parametrize("T,D,ld", [(3, 72, 72), (5, 100, 104), (4, 93, 96), (2, 2048, 2048), (3, 4096, 4096), (1, 9000, 9000)])
def test_norm_behind_a_sublayer_and_the_plain_row(T, D, ld):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(0)
    x, y, gy = torch.randn(T, D, generator=g), torch.randn(T, ld, generator=g) * 3, 1 + 0.3 * torch.randn(D, generator=g)
    want = x.double() + R.rms_norm(y[:, :D].double(), gy.double(), 1e-3)
    for clear in (False, True):
        for h in (torch.full((T, ld), 7.0, device=DEV), torch.full((T, ld), 7.0, dtype=torch.bfloat16, device=DEV)):
            xd, yd = x.to(DEV), y.to(DEV)
            ops.norm_residual(xd, 1e-3, y=yd, gy=gy.to(DEV), y_clear=clear, **{"hf" if h.dtype == torch.float32 else "hb": h})
            assert rel(xd, want) < 1e-6 and torch.equal(h[:, :D], xd.to(h.dtype)) and not h[:, D:].any()
            assert not yd.any() if clear else torch.equal(yd.cpu(), y)
            ops.norm_residual(xd, 1e-3, **{"hf" if h.dtype == torch.float32 else "hb": h.fill_(7.0)})            # nothing to add
            assert torch.equal(h[:, :D], xd.to(h.dtype)) and not h[:, D:].any()


def test_scaled_embedding():
    from openagents_b200.ops import cuda_ops as ops
    emb = torch.randn(50, 72, generator=torch.Generator().manual_seed(1)).bfloat16()
    out = torch.empty(4, 72, device=DEV)
    ops.embedding(i32(3, 49, 0, 3), out, ops.EMB_BF16, emb.to(DEV), vocab_n=50, scale=3.7)
    assert rel(out, emb[[3, 49, 0, 3]].double() * 3.7) < 1e-7


@pytest.mark.parametrize("T,D,ng,ldo", [(3, 72, 1, 72), (5, 100, 4, 104), (4, 93, 3, 96), (2, 8192, 1, 8192), (70, 1024, 8, 1024), (1, 60, 60, 64)])
def test_gated_norm_in_parts(T, D, ng, ldo):
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(2)
    y, z, w = torch.randn(T, D, generator=g) * 2, torch.randn(T, D + 7, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
    for gate in (z, None):
        v = y.double() if gate is None else y.double() * R.silu(z[:, :D].double())
        want = R.group_rms_norm(v, w.double(), ng, 1e-3)
        for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 4e-3)):
            out = torch.full((T, ldo), 7.0, dtype=dt, device=DEV)
            ops.group_norm(y.to(DEV), D, ng, w.to(DEV), 1e-3, out, gate=None if gate is None else gate.to(DEV)[:, :D])
            assert rel(out[:, :D].float(), want) < tol and not out[:, D:].any()


# ---------------------------------------------------------------- attention's projections
QKV = [(6, 2, 40, 24, 64, 64, 16, None), (4, 4, 104, 56, 104, 56, 104, (8.0, 1.0, 4.0, 64.0)), (2, 1, 10, 6, 16, 8, 2, None), (3, 1, 72, 130, 72, 136, 0, None),
       (32, 8, 128, 128, 128, 128, 128, (8.0, 1.0, 4.0, 512.0)), (9, 3, 24, 20, 64, 64, 24, (2.0, 0.5, 1.5, 30.0))]


@pytest.mark.parametrize("H,G,dim,vdim,DK,DV,rot,scaling", QKV)
def test_whole_row_norms_rotation_and_mixed_values(H, G, dim, vdim, DK, DV, rot, scaling):
    from openagents_b200.models.config import MixerSpec
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(3)
    T, pages, nq, nk = 5, 8, H * dim, G * dim
    for extra in (0, 3):                               # rows of whole float4s, and others
        row = torch.randn(T, nq + nk + G * vdim + extra, generator=g) * 2
        first = torch.randn(T, G * vdim, generator=g)
        wq, wk, lam = 1 + 0.4 * torch.randn(nq, generator=g), 1 + 0.4 * torch.randn(nk, generator=g), torch.tensor([0.3])
        pos, slot = [0, 1, 15, 16, 900], [16 * 3 + 1, 0, 16 * 7 + 15, -1, 16 * 2]
        spec = MixerSpec("attention", H, dim, vdim, kv_heads=G, rope_base=500.0, rope_dims=rot, rope_style="half", row_norm=True, rope_scaling=scaling)
        table = ops.rope_table(901, rot, 500.0, DEV, spec.rope_frequencies()) if rot else None
        turn = {"dims": rot, "base": 500.0, "scaling": dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None}
        r = row.double()
        q = R.rms_norm(r[:, :nq], wq.double(), 1e-4).view(T, H, dim)
        k = R.rms_norm(r[:, nq: nq + nk], wk.double(), 1e-4).view(T, G, dim)
        q, k = (R.rotate(x, pos, turn) if rot else x for x in (q, k))
        v = R.unit_rms(r[:, nq + nk: nq + nk + G * vdim].view(T, G, vdim), 1e-4)
        mixed = R.mix_values(v, first.double().view(T, G, vdim), 0.3)
        for dt, tol in ((torch.float32, 1e-6), (torch.float16, 1e-3)):
            for mode in ("none", "writes", "mixes"):
                kc, vc = torch.full((pages, G, 16, DK), 3.0, dtype=dt, device=DEV), torch.full((pages, G, 16, DV), 3.0, dtype=dt, device=DEV)
                q32, q16 = torch.full((T, H, DK), 5.0, device=DEV), torch.full((T, H, DK), 5.0, dtype=torch.float16, device=DEV)
                vf = None if mode == "none" else torch.full((T, G * vdim), 9.0, device=DEV) if mode == "writes" else first.to(DEV)
                ops.row_qkv_finish(row.to(DEV), 0, nq, nq + nk, wq.to(DEV), wk.to(DEV), i32(*pos), i32(*slot), table, H, G, dim, vdim, DK, DV, rot, 1, True, 1e-4, 0.25,
                                   16, kc, vc, q32=q32, q16=q16, lam=lam.to(DEV) if mode == "mixes" else None, v_first=vf)
                assert rel(q32[..., :dim], q * 0.25) < 1e-6 and not q32[..., dim:].any()
                assert rel(q16[..., :dim].float(), q * 0.25) < 1e-3 and not q16[..., dim:].any()
                if mode == "writes":
                    assert rel(vf, v.reshape(T, -1)) < 1e-6
                want = mixed if mode == "mixes" else v
                for t, s in enumerate(slot):
                    if s >= 0:
                        assert rel(kc[s // 16, :, s % 16, :dim].float(), k[t]) < tol and not kc[s // 16, :, s % 16, dim:].any()
                        assert rel(vc[s // 16, :, s % 16, :vdim].float(), want[t]) < tol and not vc[s // 16, :, s % 16, vdim:].any()
                untouched = torch.ones(pages * 16, dtype=torch.bool)
                untouched[[s for s in slot if s >= 0]] = False
                assert (kc.transpose(1, 2).reshape(pages * 16, -1)[untouched] == 3.0).all() and (vc.transpose(1, 2).reshape(pages * 16, -1)[untouched] == 3.0).all()


# ---------------------------------------------------------------- generalized delta rule
def batch_of(lens, ctx=None):
    """q_start, q_len, tokens behind the portion."""
    return i32(*[sum(lens[:b]) for b in range(len(lens))]), i32(*lens), i32(*[n + (0 if ctx is None else ctx[b]) for b, n in enumerate(lens)])


class Delta:
    """Random projections and weights of one delta-rule layer."""

    def __init__(self, H, D, rank, T, seed, keep=-3.0):
        g = torch.Generator().manual_seed(seed)
        f = lambda *s: torch.randn(*s, generator=g)    # noqa: E731
        self.H, self.D, self.rank, self.VP = H, D, rank, (D + 7) // 8 * 8 if D <= 128 else (D + 31) // 32 * 32
        hd, self.w = H * D, {}
        self.row = f(T, 5 * hd + rank)
        self.offs = tuple(i * hd for i in range(6))
        self.row[:, self.offs[2]: self.offs[3]] = self.row[:, self.offs[2]: self.offs[3]].bfloat16().float()      # v, which the chunked kernels round
        r8 = (rank + 7) // 8 * 8
        self.w2 = torch.zeros(hd, r8)
        self.w2[:, :rank] = f(hd, rank) * rank ** -0.5 * 2
        self.w2 = self.w2.bfloat16()
        self.w0, self.ab, self.norm = f(hd) * 2 + keep, f(hd), 1 + 0.3 * f(hd)

    def want(self, lo, hi, S, eps=1e-4):
        H, D = self.H, self.D
        r, k, v, g, a = (self.row[lo:hi, o: o + H * D].double() for o in self.offs[:5])
        w = torch.exp(-DECAY * torch.sigmoid(torch.tanh(self.row[lo:hi, self.offs[5]:].double()) @ self.w2[:, : self.rank].double().T + self.w0.double()))
        a = torch.sigmoid(a + self.ab.double())
        o, S = R.delta_rule(*(x.view(-1, H, D) for x in (r, w, a, k, v)), S)
        return (R.unit_rms(o, eps).reshape(-1, H * D) * self.norm.double() * torch.sigmoid(g)).view(-1, H, D), S

    def run(self, kernel, portions, state, slots, out_dtype=torch.float32):
        """``portions``: (first, last, tokens before) of each sequence among the rows."""
        from openagents_b200.ops import cuda_ops as ops
        lens = [hi - lo for lo, hi, _ in portions]
        rows = torch.cat([self.row[lo:hi] for lo, hi, _ in portions]).to(DEV)
        qs, ql, ctx = batch_of(lens, [c for _, _, c in portions])
        out = torch.full((rows.shape[0], self.H * self.VP), 7.0, dtype=out_dtype, device=DEV)
        args = (rows, self.offs, self.rank, self.w2.to(DEV), self.w0.to(DEV), self.ab.to(DEV), self.norm.to(DEV), state, qs, ql, ctx, i32(*slots), len(lens), self.H, self.D,
                self.D, self.VP, DECAY, 1e-4, out)
        if kernel == "recurrent":
            ops.delta_recurrent(*args)
        else:
            n = ops.delta_chunk_bytes(rows.shape[0], len(lens), self.H, self.D, self.VP, DECAY)
            if not n:
                pytest.skip("sizes for the token-by-token kernel")
            ops.delta_chunked(*args, max_q=max(lens), ws=torch.full((n,), 255, dtype=torch.uint8, device=DEV))
        out = out.view(-1, self.H, self.VP)
        assert not out[..., self.D:].any()
        return out[..., : self.D].float().cpu()


DELTA = [(2, 24, 8), (3, 64, 16), (1, 100, 5), (5, 128, 70), (4, 40, 130), (2, 8, 1), (1, 200, 32), (2, 256, 24), (7, 16, 12), (40, 64, 64)]


@pytest.mark.parametrize("kernel,tol", [("recurrent", 2e-5), ("chunked", 3e-4)])
@pytest.mark.parametrize("H,D,rank", DELTA)
def test_delta_rule(kernel, tol, H, D, rank):
    """Unequal sequences from zero and from a state, in slots of their own; the state behind them, and a slot that keeps nothing."""
    lens = [1, 2, 63, 64, 65, 130, 200] if H < 20 else [3, 70]
    d = Delta(H, D, rank, max(lens) + 5, H * D)
    for before in (0, 5):
        B = len(lens)
        state = torch.zeros(B + 3, H, D, d.VP)
        slots = list(torch.randperm(B + 3, generator=torch.Generator().manual_seed(1))[:B])
        state.normal_(generator=torch.Generator().manual_seed(2))        # what a fresh sequence must not read
        state[..., D:] = 0.0
        start = state.clone()
        dev = state.to(DEV)
        got = d.run(kernel, [(0, n, before) for n in lens], dev, slots)
        at = 0
        for b, n in enumerate(lens):
            S0 = start[slots[b], :, :, :D].double() if before else torch.zeros(H, D, D, dtype=torch.float64)
            want, S = d.want(0, n, S0)
            assert rel(got[at: at + n], want) < tol, (n, before)
            assert rel(dev[slots[b], :, :, :D], S) < tol and not dev[slots[b], :, :, D:].any()
            at += n
        rest = [s for s in range(B + 3) if s not in slots]
        assert torch.equal(dev[rest].cpu(), start[rest])
    dev = start.to(DEV)
    got = d.run(kernel, [(0, 3, 5)], dev, [-1])          # starts from zero, keeps nothing
    assert rel(got, d.want(0, 3, torch.zeros(H, D, D, dtype=torch.float64))[0]) < tol and torch.equal(dev.cpu(), start)


@pytest.mark.parametrize("H,D,rank", [(3, 24, 8), (2, 64, 64), (2, 128, 20)])
def test_delta_rule_in_portions(H, D, rank):
    """The same sequence whole, in portions of several sizes (down to one and two tokens), by either kernel, and token by token."""
    n = 150
    d = Delta(H, D, rank, n, 5)
    want, S = d.want(0, n, torch.zeros(H, D, D, dtype=torch.float64))
    for kernels, cuts in ((("chunked",), [150]), (("chunked",), [2]), (("chunked",), [64, 3, 65, 1]), (("recurrent", "chunked"), [1, 31, 2, 40]), (("recurrent",), [1])):
        dev, out, at, i = torch.randn(1, H, D, d.VP, device=DEV), [], 0, 0
        while at < n:
            m = min(cuts[i % len(cuts)], n - at)
            out.append(d.run(kernels[i % len(kernels)], [(at, at + m, at)], dev, [0]))
            at, i = at + m, i + 1
        assert rel(torch.cat(out), want) < 3e-4 and rel(dev[0, :, :, :D], S) < 3e-4


def test_delta_rule_remembers_and_forgets():
    """A key written long ago is read back by a query that matches it, unless a later token with the same key and a full rate has taken it away; strongest and
    weakest decays."""
    H, D, n = 2, 64, 200
    for kernel in ("recurrent", "chunked"):
        for keep in (-40.0, -9.0, 40.0):                 # decays of one, of nearly one, of e^-0.6
            d = Delta(H, D, 8, n, 7, keep)
            d.w2.zero_()
            d.w0.fill_(keep)
            for t in range(n):
                d.row[t, d.offs[1]: d.offs[2]].mul_(0.05)
            for at in (3, 64, 130):                      # the written key, and who asks for it
                d.row[at, d.offs[1]: d.offs[2]] = 0.0
                d.row[at, d.offs[1] + at % D] = 4.0
                d.row[at + 1: at + 60, d.offs[1] + at % D] = 0.0
                d.row[at + 50, d.offs[0]: d.offs[1]] = 0.0
                d.row[at + 50, d.offs[0] + at % D] = 3.0
            d.row[90, d.offs[1]: d.offs[2]] = d.row[64, d.offs[1]: d.offs[2]]
            d.row[90, d.offs[4]: d.offs[5]] = 30.0       # the rate: one
            want, S = d.want(0, n, torch.zeros(H, D, D, dtype=torch.float64))
            dev = torch.zeros(1, H, D, d.VP, device=DEV)
            got = d.run(kernel, [(0, n, 0)], dev, [0])
            for t in range(n):                           # a tiny output is divided by its size: the noise of the long sums shows there
                assert rel(got[t], want[t]) < (2e-2 if kernel == "chunked" else 1e-3), (kernel, keep, t)
            assert rel(dev[0, :, :, :D], S) < 1e-3


# ---------------------------------------------------------------- state-space duality
class Ssd:
    """Random projections and weights of one Mamba-2 layer."""

    def __init__(self, H, P, N, G, taps, T, seed, fast=0.0):
        g = torch.Generator().manual_seed(seed)
        f = lambda *s: torch.randn(*s, generator=g)    # noqa: E731
        self.H, self.P, self.N, self.G, self.taps, self.inner = H, P, N, G, taps, H * P
        self.CC, self.PP = H * P + 2 * G * N, (P + 7) // 8 * 8 if P <= 128 else (P + 31) // 32 * 32
        self.row = f(T, self.inner + self.CC + H + (-(self.inner + self.CC + H)) % 8)
        self.conv, self.cb, self.dtb, self.A, self.D = f(self.CC, taps) * 0.7, f(self.CC) * 0.3, f(H) - 2 + fast, f(H) + fast, f(H)

    def blank(self, slots):
        return torch.randn(slots, self.H, self.N, self.PP, device=DEV), torch.randn(slots, self.taps, self.CC, device=DEV)

    def want(self, lo, hi, carry=None, rounded=False):
        """``rounded``: the filter's results as the chunked kernels keep them."""
        before, S = carry or (torch.zeros(self.taps - 1, self.CC, dtype=torch.float64), torch.zeros(self.H, self.N, self.P, dtype=torch.float64))
        x = self.row[lo:hi].double()
        xbc, before = R.causal_conv(x[:, self.inner: self.inner + self.CC], before, self.conv.double(), self.cb.double())
        xbc = R.silu(xbc).bfloat16().double() if rounded else R.silu(xbc)
        u, B, C = xbc.split([self.inner, self.G * self.N, self.G * self.N], -1)
        dt = R.softplus(x[:, self.inner + self.CC: self.inner + self.CC + self.H] + self.dtb.double())
        y, S = R.ssd(u.view(-1, self.H, self.P), B.view(-1, self.G, self.N), C.view(-1, self.G, self.N), dt, self.A.double(), self.D.double(), S)
        return y.reshape(-1, self.inner), (before, S)

    def run(self, kernel, portions, state, ring, slots):
        from openagents_b200.ops import cuda_ops as ops
        lens = [hi - lo for lo, hi, _ in portions]
        rows = torch.cat([self.row[lo:hi] for lo, hi, _ in portions]).to(DEV)
        qs, ql, ctx = batch_of(lens, [c for _, _, c in portions])
        y = torch.full((rows.shape[0], self.inner), 7.0, device=DEV)
        args = (rows, self.inner, self.inner + self.CC, self.conv.to(DEV), self.cb.to(DEV), self.dtb.to(DEV), self.A.to(DEV), self.D.to(DEV), state, ring, qs, ql, ctx, i32(*slots),
                len(lens), self.H, self.P, self.N, self.G, self.PP, y)
        if kernel == "decode":
            n = ops.ssd_decode_bytes(len(lens), self.H, self.PP, self.N, self.G)
            ops.ssd_decode(*args, ws=torch.full((n,), 255, dtype=torch.uint8, device=DEV))
        else:
            exact = kernel == "exact"
            n = ops.ssd_prefill_bytes(rows.shape[0], len(lens), self.H, self.PP, self.N, self.G, exact)
            ops.ssd_prefill(*args, max_q=max(lens), ws=torch.full((n,), 255, dtype=torch.uint8, device=DEV), exact=exact)
        return y.cpu()


SSD = [(6, 20, 12, 3, 3), (4, 64, 128, 1, 4), (2, 48, 80, 2, 2), (1, 8, 16, 1, 1), (3, 100, 33, 1, 6), (8, 16, 24, 4, 4), (2, 128, 64, 1, 4), (2, 200, 256, 2, 4), (1, 256, 20, 1, 3),
       (32, 64, 64, 8, 4)]


@pytest.mark.parametrize("kernel,tol", [("exact", 1e-5), ("chunked", 1e-3)])
@pytest.mark.parametrize("H,P,N,G,taps", SSD)
def test_state_space_duality(kernel, tol, H, P, N, G, taps):
    lens = [1, 2, 63, 64, 65, 130, 200] if H < 20 else [3, 70]
    s = Ssd(H, P, N, G, taps, max(lens), H + P)
    B = len(lens)
    state, ring = s.blank(B + 2)
    kept = state[[1, B + 1]].clone(), ring[[1, B + 1]].clone()
    slots = [0, *range(2, B + 1)]
    got, at = s.run(kernel, [(0, n, 0) for n in lens], state, ring, slots), 0
    for b, n in enumerate(lens):
        want, (_, S) = s.want(0, n, rounded=kernel == "chunked")
        assert rel(got[at: at + n], want) < tol, n
        assert rel(state[slots[b], :, :, :P], S) < tol and not state[slots[b], :, :, P:].any()
        for p in range(max(0, n - taps + 1), n):         # the filter's latest inputs, by position
            assert torch.equal(ring[slots[b], p % taps].cpu(), s.row[p, s.inner: s.inner + s.CC])
        at += n
    assert torch.equal(state[[1, B + 1]], kept[0]) and torch.equal(ring[[1, B + 1]], kept[1])
    before = state.clone(), ring.clone()
    for k in (kernel, "decode"):
        m = 1 if k == "decode" else 3
        assert rel(s.run(k, [(0, m, 5)], state, ring, [-1]), s.want(0, m, rounded=k == "chunked")[0]) < tol          # starts from zero, keeps nothing
        assert torch.equal(state, before[0]) and torch.equal(ring, before[1])


@pytest.mark.parametrize("H,P,N,G,taps", [(6, 20, 12, 3, 3), (4, 64, 128, 1, 4), (3, 40, 36, 1, 6), (2, 24, 16, 2, 1)])
def test_state_space_duality_in_portions(H, P, N, G, taps):
    n = 150
    s = Ssd(H, P, N, G, taps, n, 3)
    want, (_, S) = s.want(0, n)
    for kernels, cuts in ((("chunked",), [150]), (("chunked",), [2]), (("chunked",), [64, 3, 65, 1]), (("decode", "chunked"), [1, 31, 1, 2]), (("exact", "decode"), [2, 1, 50, 1]),
                          (("decode",), [1])):
        (state, ring), out, at, i = s.blank(2), [], 0, 0
        while at < n:
            m = min(cuts[i % len(cuts)], n - at)
            out.append(s.run(kernels[i % len(kernels)], [(at, at + m, at)], state, ring, [1]))
            at, i = at + m, i + 1
        assert rel(torch.cat(out), want) < 6e-3 and rel(state[1, :, :, :P], S) < 6e-3


def test_state_space_decode_batches():
    """Sequences of different lengths decode together, in slots that others have used."""
    for H, P, N, G, taps in ((6, 20, 12, 3, 3), (64, 64, 128, 1, 4), (2, 256, 256, 1, 4), (3, 8, 200, 3, 5)):
        s = Ssd(H, P, N, G, taps, 60, 9)
        lens, slots = [1, 2, 5, 17, 40], [3, 0, 5, 1, 4]
        state, ring = s.blank(6)
        s.run("exact", [(0, n, 0) for n in lens], state, ring, slots)
        carry = [s.want(0, n)[1] for n in lens]
        for step in range(8):
            got = s.run("decode", [(n + step, n + step + 1, n + step) for n in lens], state, ring, slots)
            for b, n in enumerate(lens):
                want, carry[b] = s.want(n + step, n + step + 1, carry[b])
                assert rel(got[b], want[0]) < 2e-5, (H, b, step)


def test_state_space_strong_and_weak_decays():
    """Steps and rates so large that a token wipes the state, and so small that the first one stays."""
    for fast in (4.0, -6.0):
        s = Ssd(3, 24, 16, 1, 4, 140, 11, fast)
        for kernel, tol in (("exact", 1e-5), ("chunked", 1e-3)):
            want, (_, S) = s.want(0, 140, rounded=kernel == "chunked")
            state, ring = s.blank(1)
            assert rel(s.run(kernel, [(0, 140, 0)], state, ring, [0]), want) < tol and rel(state[0, :, :, :24], S) < tol


# ---------------------------------------------------------------- mixture of experts
def expert_weights(E, F, K, g):
    W = {}
    for e in range(E):
        W[f"e{e}.up"], W[f"e{e}.down"] = ((torch.randn(*s, generator=g) * s[1] ** -0.5 * 2).bfloat16().double() for s in ((F, K), (K, F)))
    W["router"] = (torch.randn(E, K, generator=g) * 2 * K ** -0.5).bfloat16().double()
    return W


MOE = [(5, 1, 40, 72), (12, 3, 36, 100), (64, 8, 96, 136), (1, 1, 16, 8), (7, 7, 24, 64), (200, 20, 8, 40)]


@pytest.mark.parametrize("E,top,F,K", MOE)
def test_experts_without_a_gate(E, top, F, K):
    """Router (softmax over all, renormalised over the chosen, scaled) and experts weighted at their output: few fp32 rows, and gathered bf16 rows."""
    from openagents_b200.ops import cuda_ops as ops
    g = torch.Generator().manual_seed(E)
    KP, FP, scale = (K + 7) // 8 * 8, (F + 15) // 16 * 16, 1.7
    W = expert_weights(E, F, K, g)
    w1, w2, r = torch.zeros(E, FP, KP), torch.zeros(E, KP, FP), torch.zeros(E, KP)
    for e in range(E):
        w1[e, :F, :K], w2[e, :K, :F] = W[f"e{e}.up"], W[f"e{e}.down"]
    r[:, :K] = W["router"]
    w1, w2, r = w1.bfloat16().view(-1, KP).to(DEV), w2.bfloat16().view(-1, FP).to(DEV), r.to(DEV)
    mlp = {"router": {"top": top, "scale": scale}}
    how = dict(score=ops.SCORE_SOFTMAX, scale=scale)
    for T in (1, 2, 40, 300):
        cap = (T + 127) // 128 * 128
        h, y = torch.zeros(T, KP), torch.zeros(T, KP)
        h[:, :K], y[:, :K] = torch.randn(T, K, generator=g).bfloat16().float(), torch.randn(T, K, generator=g)
        want_e, want_w = R.route(h[:, :K].double(), W["router"], top, scale)
        want = R.expert_ff(h[:, :K].double(), W, "", mlp)
        ids, w = torch.full((T, top), -1, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        ops.moe_choose(h.to(DEV), r, top, ids, w, **how)
        assert torch.equal(ids.cpu().long().sort(-1).values, want_e.sort(-1).values) and rel(w, want_w) < 1e-6
        mid, yd = torch.full((T, top, FP), float("nan"), device=DEV), y.to(DEV)
        ops.expert_up(h.to(DEV), w1, FP, ids, w, mid)
        ops.expert_down(mid, w2, KP, ids, yd)
        assert rel(yd[:, :K].cpu() - y[:, :K], want) < 3e-6 and not yd[:, K:].any()
        st, yd = i32(0), y.to(DEV)
        rx, mid = torch.empty(E * cap, KP, dtype=torch.bfloat16, device=DEV), torch.empty(E * cap, FP, dtype=torch.bfloat16, device=DEV)
        meta, rw, cnt = torch.zeros(E * cap, 2, dtype=torch.int32, device=DEV), torch.zeros(E * cap, device=DEV), torch.zeros(E, dtype=torch.int32, device=DEV)
        ops.moe_route_dispatch(h.bfloat16().to(DEV), None, r, None, top, E, cap, rx.data_ptr(), meta.data_ptr(), rw.data_ptr(), cnt.data_ptr(), None, topk_ids=ids, topk_w=w,
                               status=st, **how)
        ops.moe_gemm(rx, w1, E, cap, FP, KP, cnt, 3, out_bf16=mid, ldc=FP, status=st, live_rows=T * top)
        ops.moe_gemm(mid, w2, E, cap, KP, FP, cnt, 2, ldc=KP, meta=meta, gate_w=rw, sym_off=yd.data_ptr(), status=st, live_rows=T * top)
        assert rel(yd[:, :K].cpu() - y[:, :K], want) < 8e-3 and not yd[:, K:].any() and int(st.item()) == 0


# ---------------------------------------------------------------- whole models
D, M, A, X = R.layer_delta, R.layer_mamba, R.layer_attention, R.moe
CONFIGS = {
    # odd sizes, a width and a vocabulary that are no multiples of eight and four, windows beside the page size, layers without a feed-forward
    "odd": R.config([D(24, 3, X(40, 5, 2, 2.5, 56)), A(40, 24, 6, 2, 16, 24, 5000.0, (4.0, 1.0, 3.0, 64), mlp=X(36, 3, 1)), M(6, 20, 12, 3, 4, 3), A(16, 24, 4, 2, 8, 7, scale=0.4),
                     D(40, 2), A(24, 40, 3, 1, 0, v_mix=False, mlp=X(20, 4, 4, 0.5, 100))], width=100, vocab=131, scale=3.0),
    # one head of each kind, one expert, a filter of one tap, a window of one token, no window
    "few": R.config([A(64, 64, 1, 1, 64, 1, mlp=X(64, 1, 1)), M(1, 64, 16, 1, 1, 1, X(32, 2, 1, 1.0, 0)), D(64, 1, X(48, 9, 4)), A(32, 64, 16, 1, 16, mlp=None)], width=64, vocab=300,
                    eps=1e-3),
    # sizes of a usual kind
    "usual": R.config([D(64, 4, X(64, 8, 2, 1.5, 128)), A(64, 64, 12, 3, 64, 80, 500000.0, (8.0, 1.0, 4.0, 128), mlp=X(64, 8, 2, 1.5, 128)), D(64, 4, X(64, 8, 2, 1.5, 128)),
                       M(8, 64, 64, 2, 2, 4, X(64, 8, 2, 1.5, 128)), A(64, 64, 12, 3, 64, 48, mlp=X(72, 10, 1))], width=128, vocab=260, scale=8.0),
    # nothing is a multiple of anything
    "ragged": R.config([M(5, 13, 19, 5, 13, 5, X(21, 7, 5, 0.3, 37)), D(37, 3, X(75, 3, 2)), A(52, 20, 9, 3, 18, 31, 100.0, (2.0, 0.5, 1.5, 30), 0.05, mlp=X(13, 3, 3)), D(11, 7),
                        A(101, 20, 6, 3, 100, 50)], width=93, vocab=127, eps=1e-2, scale=0.7),
    # the sizes at which large models' kernels run, and beyond them: long rows, heads that only the token-by-token and any-size kernels take
    "wide": R.config([D(128, 2, X(64, 4, 2)), M(2, 200, 144, 1, 8, 4), A(136, 136, 4, 2, 72, 40), D(160, 2), M(3, 128, 256, 1, 3, 2, X(40, 3, 2))], width=96, vocab=264),
    # no attention at all, and nothing but attention
    "recurrent": R.config([M(4, 32, 40, 4, 1, 4, X(40, 4, 2)), D(32, 4), M(2, 96, 24, 1, 2, 7)], width=80, vocab=100),
    "attention": R.config([A(48, 48, 4, 4, 48, 20, v_mix=False), A(48, 32, 8, 2, 32, 33, mlp=X(40, 4, 1)), A(16, 32, 2, 2, 16), A(80, 32, 6, 2, 40, 17)], width=72, vocab=100),
}


def model(name, dtype, seed):
    """A configuration and weights.  bf16 rounding may tip a router's close call, which no tolerance on logits covers: there every expert is used (the
    choice is held to the plain one in 32-bit, and by the router's own test)."""
    cfg = CONFIGS[name]
    if dtype == "bfloat16":
        every = lambda m: m if m is None else dict(m, router=dict(m["router"], top=m["router"]["experts"]))      # noqa: E731
        cfg = dict(cfg, layers=[dict(l, mlp=every(l["mlp"])) for l in cfg["layers"]])
    return cfg, R.random_weights(cfg, seed=seed, rank=5 if name == "ragged" else 24)


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


def error(got, want, spread):
    """Per position: mean taken off, over the logits' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / spread


class Wanted:
    """The plain implementation's logits of every token, and how far each may be off.  A head's output is divided by its own size, so where it cancels, rounding
    shows: in bf16 a position may be off by what weights changed by about half a bf16 step cause there, three times over."""

    def __init__(self, cfg, W, toks, dtype):
        self.rows = R.forward(cfg, W, toks, R.Sequence())
        self.spread, self.limit = self.rows.std(), torch.full((len(toks),), TOL[dtype], dtype=torch.float64)
        for seed in range(4 if dtype == "bfloat16" else 0):
            g = torch.Generator().manual_seed(seed)
            shaken = {k: v * (1 + (torch.rand(v.shape, generator=g, dtype=torch.float64) - 0.5) * 2 ** -7) for k, v in W.items()}
            self.limit = torch.maximum(self.limit, 3 * error(R.forward(cfg, shaken, toks, R.Sequence()), self.rows, self.spread))


def close(got, want, rows=slice(None)):
    err, limit = error(got, want.rows[rows], want.spread), want.limit[rows]
    assert (err < limit).all(), (err.max().item(), int((err / limit).argmax()), int((err >= limit).sum()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompts_portions_and_decoding(tmp_path, name, dtype):
    cfg, W = model(name, dtype, len(name))
    be = open_model(tmp_path, cfg, W, dtype)
    toks = tokens(cfg, 203, 1)
    want = Wanted(cfg, W, toks, dtype)
    for seq, cuts in enumerate(([203], [150] + [1] * 200, [2, 64, 3, 61, 1, 17], [2], [65, 16, 1])):
        be.begin(seq, None)
        close(run(be, seq, toks, cuts), want)
        be.end(seq)
    be.begin(9, None)                      # token by token from the first
    close(run(be, 9, toks[:40], [1]), want, slice(40))


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
        assert rel(e.x[: len(toks)], layers[n - 1]) < TOL[dtype] / 2, n
        e.end(n)


@pytest.mark.parametrize("name", ["odd", "usual"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_reuse_pages_and_slots(tmp_path, name, dtype):
    """Portions beside single tokens in any order, sequences left out of steps, and a pool so tight that pages and state slots come round again; each request's
    logits are those it has alone."""
    cfg, W = model(name, dtype, 5)
    be = open_model(tmp_path, cfg, W, dtype, max_num_seqs=4, n_pages=24, max_ctx=24 * 16, max_tokens=24 * 16, state_slots=4)
    want, toks = {}, {}
    for r, n in enumerate((120, 33, 97, 64, 5, 140, 18)):
        toks[r] = tokens(cfg, n, 10 + r)
        want[r] = Wanted(cfg, W, toks[r], dtype)
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
        close(torch.cat(got[r]), want[r])
    assert be.kv_stats()["pages_free"] == 24 and be.kv_stats()["state_slots_free"] == 4


def test_state_is_neither_shared_nor_cut(tmp_path):
    cfg, W = model("odd", "float32", 6)
    be = open_model(tmp_path, cfg, W)
    toks = tokens(cfg, 60, 2)
    be.begin(1, toks)
    be.forward_at([1], [toks], [[]])
    be.publish(1, toks)
    assert be.begin(2, toks) == 0 and not be.supports_verify
    with pytest.raises(ValueError):
        be.truncate(1, 30)
    be.truncate(1, 0)                                # over again
    close(run(be, 1, toks, [40, 1]), Wanted(cfg, W, toks, "float32"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "usual"])
def test_long_decoding(tmp_path, name, dtype):
    """Every window passes over decoded tokens many times; steps without wanted logits follow one another without waiting."""
    cfg, W = model(name, dtype, 7)
    be = open_model(tmp_path, cfg, W, dtype, max_ctx=700, max_tokens=64)
    toks = tokens(cfg, 500, 4)
    want = Wanted(cfg, W, toks, dtype)
    be.begin(1, None)
    got = [run(be, 1, toks[:30], [30])]
    asked = [i for i in range(30, 500) if i < 60 or i % 16 in (0, 1, 15)]
    got += [be.forward_at([1], [[t]], [[0] if i in asked else []]) for i, t in enumerate(toks) if i >= 30]
    close(torch.cat(got), want, list(range(30)) + asked)


def far_key_model(window, G):
    """One attention layer in which a marked token's key meets a query that only a second kind of marked token has, far above all other scores, so that the answer
    at such a token shows which keys the window holds."""
    H, dim = 2 * G, 64
    cfg = R.config([R.layer_attention(dim, dim, H, G, 16, window, scale=1.0)], width=96, vocab=40)
    W = R.random_weights(cfg, seed=20)
    W["embed"][:, :2] = 0.0
    W["embed"][38, 0], W["embed"][39, 1] = 8.0, 8.0
    for n in ("q", "k"):
        W[f"l0.mix.{n}"][:, :2] = 0.0
    W["l0.mix.k"][40, 0] = 12.0                      # key head 0, a dimension that does not turn: the mark
    W["l0.mix.q"][40, 1] = 12.0                      # query head 0 of whoever asks
    return cfg, {k: v.to(torch.bfloat16).double() for k, v in W.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [17, 64, 100])
def test_far_keys_at_the_edges_of_pages_and_windows(tmp_path, window, dtype):
    """A marked key just inside and just outside the window of the token that asks for it, at page borders, asked for in prompts, in short portions and in decoding."""
    cfg, W = far_key_model(window, 2)
    be = open_model(tmp_path, cfg, W, dtype, max_ctx=400, max_tokens=400)
    seq = 0
    for at in (0, 1, 15, 16, 31, 63, 64, 127, 128):
        for far in (window - 2, window - 1, window):
            toks = [int(t) % 38 for t in tokens(cfg, at + far + 1, 30 + at)]
            toks[at], toks[at + far] = 38, 39
            want = Wanted(cfg, W, toks, dtype)
            plain = R.forward(cfg, W, toks[:at] + [0] + toks[at + 1:], R.Sequence())
            shows = (want.rows[-1] - plain[-1]).abs().max() > 0.5 * want.spread
            assert shows == (far < window)           # the key shows exactly inside the window
            for cuts in ([len(toks)], [len(toks) - 1, 1], [max(1, len(toks) - 2), 2]):
                seq += 1
                be.begin(seq, None)
                close(run(be, seq, toks, cuts)[-1:], want, slice(-1, None))
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
            close(torch.stack([r[b] for r in rows]), Wanted(cfg, W, toks[b] + more[b], "bfloat16"), slice(-3, None))


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
        close(logits[:n], Wanted(cfg, W, prompt + ids, dtype), slice(24, 24 + n))
        be.end(int(graph))
    be.begin(5, None)
    _, nxt = be.engine.forward_tokens([5], [prompt])
    first = int(nxt[0])
    hist = be.engine.decode_steps([5], [first], 9)
    assert [first] + hist[:, 0].tolist() == out


@pytest.mark.parametrize("name", list(CONFIGS))
def test_workspace_canaries(tmp_path, name):
    for dtype in ("float32", "bfloat16"):
        cfg, W = model(name, dtype, 13)
        be = open_model(tmp_path / dtype, cfg, W, dtype, max_num_seqs=3, max_ctx=96, max_tokens=140, canaries=True)
        for b in range(3):
            be.begin(b, None)
        be.forward_at([0, 1, 2], [tokens(cfg, n, n) for n in (70, 1, 69)], [[0], [0], [68]])
        for _ in range(3):
            be.forward_at([0, 1, 2], [[1], [2], [3]], [[0], [0], [0]])
        be.forward_at([0], [[1]], [[0]])
        be.forward_at([2, 0], [[1], [2, 3]], [[0], [1]])
        be.engine.check_status()
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
    save_gguf(path, src.cfg, {k: v.float().reshape(-1) if not v.dim() else v.float() for k, v in W.items()}, PLAN_BF16)
    be2 = CudaBackend.open(path, max_num_seqs=4, max_ctx=128, max_tokens=128, dtype="float32")
    assert be2.cfg.layers == src.cfg.layers
    toks = tokens(cfg, 50, 1)
    for b in (be, be2):
        b.begin(1, None)
    for b in (be, be2):
        close(b.forward_at([1], [toks], [list(range(50))]), Wanted(cfg, W, toks, "float32"))


def test_trace_runner(tmp_path):
    """bin/trace_run as a user starts it."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CONFIGS["odd"]
    ta, tb = tokens(cfg, 40, 1), tokens(cfg, 21, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:20], "want": []}, {"id": "a", "tokens": ta[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ta[31:], "want": [8]}, {"id": "b", "tokens": tb[20:], "want": [0]}], "end": ["a", "b"]}]
    for dtype in ("float32", "bfloat16"):
        cfg, W = model("odd", dtype, 15)
        folder = R.save_model(str(tmp_path / dtype), cfg, W)
        wa, wb = Wanted(cfg, W, ta, dtype), Wanted(cfg, W, tb, dtype)
        want = [[(wa, 0), (wa, 29)], None, [(wa, 39), (wb, 20)]]
        out = tmp_path / ("out-" + dtype)
        out.mkdir()
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        for n, w in enumerate(want):
            f = out / f"{n}.f32"
            assert f.exists() == (w is not None)
            if w is not None:
                for row, (whole, at) in zip(torch.from_numpy(np.fromfile(f, dtype="<f4")).view(len(w), -1), w):
                    close(row[None], whole, [at])
