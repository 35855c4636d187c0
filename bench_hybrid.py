"""Prefill and decode throughput of the hybrid engine (Folirax, Pesorax, Kazolorn, Tekosun) at a real model's layer sizes, beside the closest other engine at equal size:
the Llama engine, or, for a stack with experts, the mixture-of-experts engine.

    python bench.py --workload hybrid [--model folirax-8b-shape | pesorax-8b-shape | kazolorn-8b-shape | kazolorn-moe-shape | tekosun-8b-shape | ...] [--steps K] [--warmup W]

Both engines hold bf16 random weights of the same width, feed-forward, head layout, depth and vocabulary, run the same prompts
and batches, and are timed with CUDA events: a 2048-token prompt, four of them in one call, and decode steps (replayed graphs
with the autoregression on the device) at several batch sizes on a 2048-token context.  ``kernels`` times every kernel of the
hybrid layers alone, L2 flushed before each launch, against its roofline (the slower of its bytes at the measured copy
bandwidth and its FLOPs at the measured bf16 rate), with the like kernel of the Llama layer where there is one.
"""
from __future__ import annotations

import gc
import json
import os

import torch

PROMPT = 2048
BATCHES = (1, 8, 64)


def peaks() -> tuple[float, float, str]:
    try:
        p = json.load(open(os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    except Exception:      # noqa: BLE001
        return 6.65e12, 1.59e15, "fallback"


def like_llama(cfg):
    """The Llama shape with the hybrid's width, depth (a looped layer counts every time), feed-forward, vocabulary and attention heads (Pesorax: heads of
    128, four to a key/value head)."""
    from openagents_b200.models.config import ModelConfig
    m = next(l.mixer for l in cfg.layers if l.mixer.kind == "attention")
    moe = next((l for l in cfg.layers if l.moe), None)
    if moe is not None:              # the same experts, heads and windows, a mixture in every layer
        return ModelConfig(arch="gpt-oss", n_layers=len(cfg.layers), d_model=cfg.d_model, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, ffn=moe.ffn,
                           vocab=cfg.vocab, context=8192, rope_theta=150000.0, rope_style="half", n_experts=moe.moe.experts, top_k=moe.moe.top,
                           sliding_window=m.window, swa_every=1, attn_sinks=True, name="moe-" + cfg.name)
    heads, kv, dim = (cfg.d_model // 128, cfg.d_model // 512, 128) if cfg.arch == "pesorax" else (m.heads, m.kv_heads, m.dim)
    return ModelConfig(arch="llama", n_layers=len(cfg.layer_runs()), d_model=cfg.d_model, n_heads=heads, n_kv_heads=kv, head_dim=dim,
                       ffn=cfg.ffn, vocab=cfg.vocab, context=8192, rope_theta=500000.0, name="llama-" + cfg.name)


def time_engine(cfg, dev, steps: int, warmup: int) -> dict:
    from openagents_b200.models.qweight import RandomSource
    from openagents_b200.models.registry import build_engine
    from openagents_b200.models.weights import PLAN_BF16, PLAN_MOE
    B = max(BATCHES)
    eng = build_engine(RandomSource(cfg, PLAN_MOE if cfg.n_experts else PLAN_BF16, 0, dev), dev, B, PROMPT + 2 * (steps + warmup) * len(BATCHES) + 64, 4 * PROMPT)
    g = torch.Generator().manual_seed(1)
    prompts = torch.randint(0, cfg.vocab, (B, PROMPT), generator=g).tolist()

    def timed(fn):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b)

    def prefill(ids):
        for i in ids:
            eng.begin(i)
        ms = timed(lambda: eng.forward_tokens(ids, [prompts[i] for i in ids]))
        first = eng.out_ids[: len(ids)].tolist()
        return ms, first
    out = {"params": cfg.n_params(), "weight_bytes": eng.weight_bytes()}
    for ids in ([0], [0, 1, 2, 3]):
        ms = []
        for _ in range(4):
            ms.append(prefill(ids)[0])
            for i in ids:
                eng.end(i)
        out[f"prefill_{len(ids)}x{PROMPT}_ms"] = round(min(ms[1:]), 3)
        out[f"prefill_{len(ids)}x{PROMPT}_tok_s"] = round(len(ids) * PROMPT / min(ms[1:]) * 1e3)
    last = []
    for b0 in range(0, B, 4):
        last += prefill(list(range(b0, min(B, b0 + 4))))[1]
    for b in BATCHES:
        ids = list(range(b))
        last[:b] = eng.decode_steps(ids, last[:b], warmup)[warmup - 1].tolist()
        mark = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        h = eng.decode_steps(ids, last[:b], steps, on_replay=lambda i: mark[0].record() if i == 0 else None)
        mark[1].record()
        torch.cuda.synchronize()
        last[:b] = h[steps - 1].tolist()
        ms = mark[0].elapsed_time(mark[1]) / steps
        out[f"decode_bs{b}_ms"], out[f"decode_bs{b}_tok_s"] = round(ms, 4), round(b / ms * 1e3, 1)
        out[f"decode_bs{b}_launches"] = eng.launches_per_decode
    eng.check_status()
    del eng
    gc.collect()
    torch.cuda.empty_cache()
    return out


class _Timer:
    """Median time of a launch with L2 flushed ahead of it, against the slower of its bytes and its FLOPs at the measured rates."""

    def __init__(self, dev, reps: int):
        self.hbm, self.flops, _ = peaks()
        self.reps, self.rows, self.flush = reps, [], torch.empty(1 << 30, dtype=torch.uint8, device=dev)

    def __call__(self, name, fn, nbytes, fl=0.0, like=None):
        ms = []
        for i in range(self.reps + 3):
            torch.cuda.synchronize()
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()                             # queued behind the flush: the launch itself is not in the time
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= 3:
                ms.append(a.elapsed_time(b))
        ms.sort()
        us, roof = ms[len(ms) // 2] * 1e3, max(nbytes / self.hbm, fl / self.flops) * 1e6
        self.rows.append({"kernel": name, "us": round(us, 1), "roofline_us": round(roof, 1), "of_roofline": round(roof / us, 3), "like": like})


def time_pesorax_kernels(cfg, dev, reps: int = 12) -> list[dict]:
    """Every kernel of a differential and a latent layer at 2048 prompt tokens and at decode steps, and its Llama counterpart.  Cached rows are read once, FLOPs
    are those of the visible keys; attention's reading of keys and values counts once per key/value head."""
    from openagents_b200.ops import cuda_ops as ops
    bench = _Timer(dev, reps)
    df, lt = (next(l.mixer for l in cfg.layers if l.mixer.kind == k) for k in ("attention", "latent"))
    ref = like_llama(cfg)
    d, F, T, B, ctx = cfg.d_model, cfg.ffn, PROMPT, 64, PROMPT
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev)                       # noqa: E731
    bf = lambda *s: torch.randn(*s, device=dev).bfloat16()             # noqa: E731
    hf = lambda *s: torch.randn(*s, device=dev).half()                 # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)     # noqa: E731
    pages = (ctx + 15) // 16
    table = lambda s: i32(list(range(s * pages))).view(s, pages)       # noqa: E731
    splits = lambda s, g: max(1, min(64, max(1, pages // 24), max((147 + s * g) // (s * g), (2047 + s * g) // (s * g) if s * g >= 148 else 0)))      # noqa: E731
    H, G, D, V = df.heads, df.kv_heads, df.dim, df.vdim
    Hq, Gq, Dq = ref.n_heads, ref.n_kv_heads, ref.head_dim
    for n in (T, B):
        x, hb, w, al = rnd(n, d), bf(n, d), rnd(d), torch.ones(1, device=dev)
        bench(f"norm_dyt [{n}]", lambda: ops.norm_dyt(x, al, w, w, hb=hb), n * d * 6, like=f"rmsnorm [{n}]")
        bench(f"rmsnorm [{n}]", lambda: ops.rmsnorm(x, w, 1e-6, hb=hb), n * d * 6)
    # ---- differential attention
    nq, nk, nv = 2 * H * D, 2 * G * D, G * V
    for n, seqs in ((T, 1), (B, B), (1, 1)):
        prompt = n == T
        row, bias, lam = rnd(n, nq + nk + nv), rnd(nq + nk + nv), torch.ones(1, device=dev)
        pos, slot = i32([ctx - 1] * n if not prompt else list(range(n))), i32(list(range(n)))
        kc, vc = hf(seqs * pages + 1, G, 16, 2 * D), hf(seqs * pages + 1, G, 16, V)
        q16, q32 = hf(n, nq), rnd(n, 2 * nq)
        q = dict(q16=q16) if prompt else dict(q32=q32, q_wide=True)
        bench(f"qkv_finish two maps [{n}]", lambda: ops.qkv_finish(row, 0, nq, nq + nk, pos, slot, None, 1.0, 2 * H, G, D, V, D, V, 0, 1, False, 1e-6, df.scale, 16, kc=kc,
                                                                   vc=vc, maps=2, bias=bias, **q), n * ((nq + nk + nv) * 4 + nq * (2 if prompt else 8) + (nk + nv) * 2),
              like=f"rope_kv [{n}]")
        ld = (Hq + 2 * Gq) * Dq
        row2, tabf, kl, vl = rnd(n, ld), ops.rope_table(ctx, Dq, 500000.0, dev), hf(seqs * pages + 1, Gq, 16, Dq), hf(seqs * pages + 1, Gq, 16, Dq)
        l16, l32 = hf(n, Hq * Dq), rnd(n, Hq * Dq)
        bench(f"rope_kv [{n}]", lambda: ops.rope_kv(row2, pos, slot, None if prompt else l32, l16 if prompt else None, kl, vl, Hq, Gq, Dq, 16, 500000.0, 0, 0.1, table=tabf),
              n * (ld * 4 + Hq * Dq * (2 if prompt else 4) + 2 * Gq * Dq * 2))
        lens, tb, mo, o = i32([ctx] * seqs), table(seqs), rnd(n, 2 * H * V), bf(n, H * V)
        if prompt:
            z = i32([0])
            bench(f"attn_prefill_tc05 two maps [{T}]", lambda: ops.attn_prefill_tc05(q16, kc, vc, tb, z, lens, lens, 1, T, 2 * H, G, out_f32=mo, status=st, dk=D, dv=V,
                                                                                    chunk=df.chunk, maps=2), T * (nq * 2 + (nk + nv) * 2 + 2 * H * V * 4),
                  2.0 * min(T, df.chunk) * T / 2 * 2 * H * (D + V), like=f"attn_prefill_tc05 [{T}]")
            ol = bf(T, Hq * Dq)
            bench(f"attn_prefill_tc05 [{T}]", lambda: ops.attn_prefill_tc05(l16, kl, vl, tb, z, lens, lens, 1, T, Hq, Gq, out_bf16=ol, status=st, dk=Dq, dv=Dq),
                  T * (Hq + Gq) * Dq * 4, 4.0 * T * T / 2 * Hq * Dq)
        else:
            S = splits(n, G)
            sc, cnt = rnd(ops.attn_decode_scratch_floats(n, 2 * H, G, V, S)), torch.zeros(n * 2 * H, dtype=torch.int32, device=dev)
            bench(f"attn_decode two maps [{n} x {ctx}]", lambda: ops.attn_decode(q32, kc, vc, tb, lens, n, 2 * H, G, 2 * D, dv=V, S=S, out_f32=mo, scratch=sc, counters=cnt,
                                                                                status=st, chunk=df.chunk), n * min(ctx, df.chunk) * (nk + nv) * 2,
                  like=f"attn_decode [{n} x {ctx}]")
            ol, S2 = bf(n, Hq * Dq), splits(n, Gq)
            sc2, cnt2 = rnd(ops.attn_decode_scratch_floats(n, Hq, Gq, Dq, S2)), torch.zeros(n * Hq, dtype=torch.int32, device=dev)
            bench(f"attn_decode [{n} x {ctx}]", lambda: ops.attn_decode(l32, kl, vl, tb, lens, n, Hq, Gq, Dq, S=S2, out_bf16=ol, scratch=sc2, counters=cnt2, status=st),
                  n * ctx * Gq * Dq * 4)
        bench(f"diff_combine [{n}]", lambda: ops.diff_combine(mo, lam, H, G, V, V, 1e-6, 0.5, out_bf16=o), n * H * V * 10, like=f"rmsnorm [{n if n > 1 else B}]")
    # ---- latent attention
    HL, DL, RL, VL, C, Q = lt.heads, lt.dim, lt.rot_dim, lt.vdim, lt.kv_rank, lt.q_rank
    W, hs, n_proj = C + RL, DL + RL, Q + C + RL + HL * VL
    tab = ops.rope_table(ctx, lt.rope_dims, lt.rope_base, dev)
    for n, seqs in ((T, 1), (B, B), (1, 1)):
        prompt = n == T
        row, qw, cw = rnd(n, n_proj), rnd(Q), rnd(C)
        pos, slot = i32([ctx - 1] * n if not prompt else list(range(n))), i32(list(range(n)))
        cache, cq, uq, uq16 = hf(seqs * pages + 1, 16, W), bf(n, Q), rnd(n, HL * hs), bf(n, HL * hs)
        tb, lens, gate, sink = table(seqs), i32([ctx] * seqs), row[:, Q + W:], rnd(HL)
        bench(f"latent_finish [{n}]", lambda: ops.latent_finish(row, 0, Q, Q + C, Q, C, RL, lt.rope_dims, 1, qw, cw, 1e-6, pos, slot, tab, lt.rope_base, cq, cache, C, RL),
              n * ((Q + W) * 4 + Q * 2 + W * 2), like=f"rope_kv [{n}]")
        o = bf(n, HL * VL)
        if prompt:
            q16, z, base, c, kv = hf(n, HL * hs), i32([0]), i32([0]), bf(n, C), hf(n, HL * (DL + VL))
            bench(f"latent_q [{n}]", lambda: ops.latent_q(uq, hs, HL, DL, RL, lt.rope_dims, 1, DL, DL, RL, hs, pos, tab, lt.rope_base, 0.1, q16), n * HL * hs * 6, like=f"rope_kv [{n}]")
            bench(f"latent_gather [{n}]", lambda: ops.latent_gather(cache, C, tb, lens, base, 1, n, c), n * C * 4, like=f"rope_kv [{n}]")
            we = bf(HL * (DL + VL), C)
            bench(f"gemm expand [{n} x {HL * (DL + VL)} x {C}]", lambda: ops.gemm_bf16(c, we, n, HL * (DL + VL), C, out_f16=kv, status=st), n * (C + HL * (DL + VL)) * 2 + we.numel() * 2,
                  2.0 * n * C * HL * (DL + VL), like=f"gemm qkv [{n}]")
            bench(f"attn_prefill_latent [{n}]", lambda: ops.attn_prefill_latent(q16, kv, HL * DL, base, cache, C, tb, z, lens, lens, 1, n, HL, DL, RL, VL, o, sinks=sink, gate=gate,
                                                                               status=st), n * HL * (hs + DL + VL + VL) * 2 + n * HL * VL * 4, 2.0 * n * n / 2 * HL * (hs + VL),
                  like=f"attn_prefill_tc05 [{T}]")
        else:
            ql, ol = rnd(n, HL * W), bf(n, HL * C)
            wa, wv = bf(HL * C, DL), bf(HL * VL, C)
            if n > 1:
                bench(f"gemm_heads absorb [{n}]", lambda: ops.gemm_heads(uq16, wa, HL, C, DL, hs, ql, W, alpha=0.1, status=st), wa.numel() * 2 + n * HL * (DL * 2 + C * 4),
                      2.0 * n * wa.numel(), like=f"gemm qkv [{n}]")
                bench(f"gemm_heads value [{n}]", lambda: ops.gemm_heads(ol, wv, HL, VL, C, C, o, VL, gate=gate, status=st), wv.numel() * 2 + n * HL * (C * 2 + VL * 6),
                      2.0 * n * wv.numel(), like=f"gemm qkv [{n}]")
            bench(f"latent_q [{n}]", lambda: ops.latent_q(uq, hs, HL, DL, RL, lt.rope_dims, 1, 0, C, RL, W, pos, tab, lt.rope_base, 0.1, ql), n * HL * RL * 8, like=f"rope_kv [{n}]")
            ctas, blocks = n * ((HL + 31) // 32), ctx // 128
            S = min(range(1, min(64, blocks, max(1, 592 // ctas)) + 1), key=lambda s: -(-ctas * s // 148) * (-(-blocks // s) + 1))
            sc = rnd(max(1, ops.latent_decode_scratch_floats(n, HL, C, S)))
            bench(f"latent_decode [{n} x {ctx}] ({S} shares)", lambda: ops.latent_decode(ql, cache, tb, None, pos, n, HL, C, RL, S, sc, out_bf16=ol, sinks=sink, status=st),
                  n * (ctx * W * 2 + HL * (W * 4 + C * 2)), 2.0 * n * ctx * HL * (W + C), like=f"attn_decode [{n} x {ctx}]")
    # ---- products
    for n in (T, B):
        a, up, dn, gu, x, act = bf(n, d), bf(F, d), bf(d, F), bf(2 * F, d), rnd(n, d), bf(n, F)
        bench(f"gemm gelu up [{n} x {F} x {d}]", lambda: ops.gemm_bf16(a, up, n, F, d, out_bf16=act, act=ops.ACT_GELU_ERF, status=st), (F * d + n * (d + F)) * 2, 2.0 * n * F * d,
              like=f"gemm swiglu gate/up [{n}]")
        bench(f"gemm swiglu gate/up [{n}]", lambda: ops.gemm_bf16(a, gu, n, 2 * F, d, out_bf16=act, ldc=F, act=ops.ACT_SWIGLU_PAIR, status=st), (2 * F * d + n * (d + F)) * 2, 4.0 * n * F * d)
        bench(f"gemm down, scaled residual [{n}]", lambda: ops.gemm_bf16(act, dn, n, d, F, out_f32=x, accumulate=True, alpha=0.5, status=st), (F * d + n * F) * 2 + n * d * 8,
              2.0 * n * F * d, like=f"gemm down, residual [{n}]")
        bench(f"gemm down, residual [{n}]", lambda: ops.gemm_bf16(act, dn, n, d, F, out_f32=x, resid_f32=x, status=st), (F * d + n * F) * 2 + n * d * 8, 2.0 * n * F * d)
        for nm, N, K in (("gemm differential qkv", nq + nk + nv, d), ("gemm latent down", n_proj, d), ("gemm latent queries", HL * hs, Q), ("gemm qkv", (Hq + 2 * Gq) * Dq, d)):
            wt, ai, o3 = bf(N, K), bf(n, K), torch.zeros(n, N, device=dev)
            bench(f"{nm} [{n}]", lambda: ops.gemm_bf16(ai, wt, n, N, K, out_f32=o3, accumulate=n <= 64 and K == d, status=st), N * K * 2 + n * (K * 2 + N * 4), 2.0 * n * N * K,
                  like=None if nm == "gemm qkv" else f"gemm qkv [{n}]")
    return bench.rows


def time_kazolorn_kernels(cfg, dev, reps: int = 12) -> list[dict]:
    """Every kernel of a Kazolorn layer at 2048 prompt tokens and at decode steps, and its counterpart in the closest engine's layer.  Cached rows are read once; FLOPs
    of the attention are the design's own (raw scores, mixture, output of the visible keys), whatever form the kernel computes them in."""
    from openagents_b200.ops import cuda_ops as ops
    bench = _Timer(dev, reps)
    m = cfg.layers[0].mixer
    H, G, D, win = m.heads, m.kv_heads, m.dim, m.window
    dense, mix = next((l for l in cfg.layers if l.ffn and not l.moe), None), next((l for l in cfg.layers if l.moe), None)
    d, T, B, ctx = cfg.d_model, PROMPT, 64, PROMPT
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev)                       # noqa: E731
    bf = lambda *s: torch.randn(*s, device=dev).bfloat16()             # noqa: E731
    hf = lambda *s: torch.randn(*s, device=dev).half()                 # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)     # noqa: E731
    pages, slabs, ls = (ctx + 15) // 16, (len(cfg.layers) + 2) // 2, rnd(d)
    for n in (T, B, 1):
        xs, w, g, h1, h2 = rnd(slabs + 1, n, d), rnd(slabs), rnd(d), bf(n, d), bf(n, d)
        bench(f"depth_norm of {slabs} [{n}]", lambda: ops.depth_norm(xs[:slabs], d, 1e-6, weights=w, out=xs[slabs], add=g, g1=g, g2=g, h1=h1, h2=h2), n * d * (4 * slabs + 8),
              like=f"rmsnorm [{n}]")
        more, pw = rnd(slabs + 3, n, d), rnd(3, slabs)
        bench(f"depth_norm of {slabs}, three sums more [{n}]", lambda: ops.depth_norm(more[:slabs], d, 1e-6, weights=w, out=xs[slabs], add=g, g1=g, g2=g, h1=h1, h2=h2,
                                                                                     parts=more[slabs:], part_weights=pw), n * d * (4 * slabs + 20), like=f"rmsnorm [{n}]")
        x = rnd(n, d)
        bench(f"rmsnorm [{n}]", lambda: ops.rmsnorm(x, g, 1e-6, hb=h1), n * d * 6)
        del xs, more
    # ---- attention
    nq, nk = H * D, G * D
    for n, seqs in ((T, 1), (B, B), (1, 1)):
        prompt = n == T
        row, bias, mixw, slopes, zero = rnd(n, nq + nk), rnd(nq + nk), rnd(H, H).bfloat16().float(), rnd(H).abs() * 0.01, torch.zeros(H, device=dev)
        pos, slot = i32([ctx - 1] * n if not prompt else list(range(n))), i32(list(range(n)))
        kc = hf(seqs * pages + 1, 1, 16, nk)
        table, lens, o = i32(list(range(seqs * pages))).view(seqs, pages), i32([ctx] * seqs), bf(n, nq)
        ld = (H + 2 * G) * D
        row2, tabf, kl, vl = rnd(n, ld), ops.rope_table(ctx, D, 500000.0, dev), hf(seqs * pages + 1, G, 16, D), hf(seqs * pages + 1, G, 16, D)
        l16, l32 = hf(n, nq), rnd(n, nq)
        seen = min(ctx, win)
        if prompt:
            q16, z = hf(n, H * nk), i32([0])
            bench(f"mixed_finish [{n}]", lambda: ops.mixed_finish(row, nq, bias, mixw, 0.1, slot, H, G, D, D, q16, kc), n * ((nq + nk) * 4 + H * nk * 2 + nk * 2), like=f"rope_kv [{n}]")
            pairs = sum(min(t + 1, win) for t in range(T))
            bench(f"mixed_prefill [{n}]", lambda: ops.mixed_prefill(q16, kc, slopes, table, z, lens, lens, 1, n, H, G, D, window=win, sinks=zero, out_bf16=o, status=st),
                  n * (nq * 4 + nk * 2), 2.0 * pairs * H * (2 * D + H), like=f"attn_prefill_tc05 [{n}]")
            bench(f"attn_prefill_tc05 [{n}]", lambda: ops.attn_prefill_tc05(l16, kl, vl, table, z, lens, lens, 1, n, H, G, window=0 if win >= T else win, out_bf16=o, status=st, dk=D, dv=D),
                  n * (H + G) * D * 4, 4.0 * pairs * H * D)
        else:
            bench(f"qkv_finish keys only [{n}]", lambda: ops.qkv_finish(row, 0, nq, -1, pos, slot, None, 1.0, H, 1, D, D, D, D, 0, 1, False, 0.0, 0.1, 16, q32=l32, kc=kc, maps=G,
                                                                        bias=bias), n * ((nq + nk) * 4 + nq * 4 + nk * 2), like=f"rope_kv [{n}]")
            from openagents_b200.models.hybrid_engine import HybridEngine
            e = HybridEngine.__new__(HybridEngine)
            e.max_splits = 64
            S = e._mixed_splits(n, min(pages, win // 16 + 2))
            sc, prep = rnd(ops.mixed_decode_scratch_floats(n, H, G, D, S)), ops.mixed_decode_prepare(mixw, slopes, H, G, D)
            bench(f"mixed_decode [{n} x {seen}] ({S} shares)", lambda: ops.mixed_decode(l32, kc, prep, table, lens, n, H, G, D, window=win, S=S, sinks=zero, out_bf16=o,
                                                                                     scratch=sc, status=st), n * (seen * nk * 2 + nq * 6),
                  2.0 * n * seen * H * (2 * D + H), like=f"attn_decode [{n} x {seen}]")
            e.attn_target_ctas = 0
            S2 = e._attn_splits(n, G, min(pages, win // 16 + 2))
            sc2, cnt2 = rnd(ops.attn_decode_scratch_floats(n, H, G, D, S2)), torch.zeros(n * H, dtype=torch.int32, device=dev)
            bench(f"attn_decode [{n} x {seen}]", lambda: ops.attn_decode(l32, kl, vl, table, lens, n, H, G, D, window=0 if win >= ctx else win, S=S2, out_bf16=o, scratch=sc2, counters=cnt2,
                                                                      status=st), n * (seen * G * D * 4 + nq * 6))
        bench(f"rope_kv [{n}]", lambda: ops.rope_kv(row2, pos, slot, None if prompt else l32, l16 if prompt else None, kl, vl, H, G, D, 16, 500000.0, 0, 0.1, table=tabf),
              n * (ld * 4 + nq * (2 if prompt else 4) + 2 * nk * 2))
        del kc, kl, vl
    # ---- products
    for n in (T, B):
        a, x = bf(n, d), rnd(n, d)
        for nm, N, like in (("gemm queries and keys", nq + nk, True), ("gemm qkv", nq + 2 * nk, False)):
            wt, o3 = bf(N, d), torch.zeros(n, N, device=dev)
            bench(f"{nm} [{n}]", lambda: ops.gemm_bf16(a, wt, n, N, d, out_f32=o3, accumulate=n <= 64, status=st), N * d * 2 + n * (d * 2 + N * 4), 2.0 * n * N * d,
                  like=f"gemm qkv [{n}]" if like else None)
        wo, ao = bf(d, nq), bf(n, nq)
        bench(f"gemm output, layer scale [{n}]", lambda: ops.gemm_bf16(ao, wo, n, d, nq, out_f32=x, accumulate=True, col_scale=ls, status=st), wo.numel() * 2 + n * (nq * 2 + d * 8),
              2.0 * n * d * nq, like=f"gemm output, residual [{n}]")
        bench(f"gemm output, residual [{n}]", lambda: ops.gemm_bf16(ao, wo, n, d, nq, out_f32=x, resid_f32=x, status=st), wo.numel() * 2 + n * (nq * 2 + d * 8), 2.0 * n * d * nq)
        if dense:
            F = dense.ffn
            zb = 4 if n <= 64 else 2                        # bytes of an activation on its way to PolyNorm
            up, dn, gu, z, act, coef = bf(F, d), bf(d, F), bf(2 * F, d), rnd(n, F) if zb == 4 else bf(n, F), bf(n, F), rnd(4)
            bench(f"gemm up [{n}]", lambda: ops.gemm_bf16(a, up, n, F, d, out_f32=z if zb == 4 else None, out_bf16=z if zb == 2 else None, status=st), (F * d + n * d) * 2 + n * F * zb, 2.0 * n * F * d, like=f"gemm swiglu gate/up [{n}]")
            bench(f"gemm swiglu gate/up [{n}]", lambda: ops.gemm_bf16(a, gu, n, 2 * F, d, out_bf16=act, ldc=F, act=ops.ACT_SWIGLU_PAIR, status=st), (2 * F * d + n * (d + F)) * 2,
                  4.0 * n * F * d)
            bench(f"poly_norm [{n}]", lambda: ops.poly_norm(z, F, coef, 1e-6, act), n * F * (zb + 2), like=f"rmsnorm [{n}]")
            bench(f"gemm down, layer scale [{n}]", lambda: ops.gemm_bf16(act, dn, n, d, F, out_f32=x, accumulate=True, col_scale=ls, status=st), (F * d + n * F) * 2 + n * d * 8,
                  2.0 * n * F * d, like=f"gemm down, residual [{n}]")
            bench(f"gemm down, residual [{n}]", lambda: ops.gemm_bf16(act, dn, n, d, F, out_f32=x, resid_f32=x, status=st), (F * d + n * F) * 2 + n * d * 8, 2.0 * n * F * d)
            del up, dn, gu, z, act
    # ---- experts
    if mix:
        E, top, F = mix.moe.experts, mix.moe.top, mix.ffn
        w13, w2, router = bf(E * 2 * F, d) * 0.02, bf(E * d, F) * 0.02, rnd(E, d) * 0.02
        for n in (T, B):
            cap = (n + 127) // 128 * 128
            rx, mid, meta, rw = bf(E * cap, d), bf(E * cap, F), torch.zeros(E * cap, 2, dtype=torch.int32, device=dev), rnd(E * cap)
            h, x, ids, w = bf(n, d), rnd(n, d), torch.zeros(n, top, dtype=torch.int32, device=dev), rnd(n, top)
            cnt = torch.zeros(64, E, dtype=torch.int32, device=dev)
            used = min(E, n * top)
            for nm, score, like in (("route and dispatch, sigmoid", ops.SCORE_SIGMOID, "route and dispatch, softmax"), ("route and dispatch, softmax", ops.SCORE_SOFTMAX, None)):
                cnt.zero_()
                turn = iter(range(64))
                bench(f"{nm} [{n}]", lambda: ops.moe_route_dispatch(h, None, router, None, top, E, cap, rx.data_ptr(), meta.data_ptr(), rw.data_ptr(), cnt[next(turn)].data_ptr(), None,
                                                                    topk_ids=ids, topk_w=w, status=st, score=score), n * d * 2 * (1 + top) + E * d * 4, like=like and f"{like} [{n}]")
            for nm, gw, like in (("experts gate/up, weight on the input", rw, "experts gate/up"), ("experts gate/up", None, None)):
                bench(f"{nm} [{n}]", lambda: ops.moe_gemm(rx, w13, E, cap, 2 * F, d, cnt[0], 1, out_bf16=mid, ldc=F, gate_w=gw, status=st, live_rows=n * top),
                      used * 2 * F * d * 2 + n * top * (d + F) * 2, 4.0 * n * top * F * d, like=like and f"{like} [{n}]")
            for nm, gw, sc, like in (("experts down, layer scale", None, ls, "experts down"), ("experts down", rw, None, None)):
                bench(f"{nm} [{n}]", lambda: ops.moe_gemm(mid, w2, E, cap, d, F, cnt[0], 2, ldc=d, meta=meta, gate_w=gw, sym_off=x.data_ptr(), col_scale=sc, status=st, live_rows=n * top),
                      used * F * d * 2 + n * top * (F * 2 + d * 4), 2.0 * n * top * F * d, like=like and f"{like} [{n}]")
        h, x, ids, w, mid = rnd(1, d), rnd(1, d), i32([list(range(top))]), rnd(1, top), rnd(1, top, F)
        bench("expert_gate_up [1]", lambda: ops.expert_gate_up(h, w13, F, ids, w, mid), top * 2 * F * d * 2, like="matvec swiglu [1]")
        bench("expert_down [1]", lambda: ops.expert_down(mid, w2, d, ids, x, scale=ls), top * F * d * 2, like="matvec down [1]")
        F4 = top * F
        gu, dn, act = bf(2 * F4, d), bf(d, F4), rnd(1, F4)
        bench("matvec swiglu [1]", lambda: ops.matvec(ops.WT_BF16, gu, None, F4, d, 1, xf=h, epi=ops.EPI_SWIGLU_F32, y=act, ldy=F4), 2 * F4 * d * 2)
        bench("matvec down [1]", lambda: ops.matvec(ops.WT_BF16, dn, None, d, F4, 1, xf=act, epi=ops.EPI_RESID, resid=x, y=x, ldy=d), F4 * d * 2)
    return bench.rows


def time_tekosun_kernels(cfg, dev, reps: int = 12) -> list[dict]:
    """Every kernel that a Tekosun layer has and another engine's layer has not, at 2048 prompt tokens and at decode steps, and its counterpart: gated linear attention
    of the same width (heads of 128 x 256) for the recurrences, the mixture-of-experts engine's kernels for the rest.  A recurrence's bytes are its projection
    rows and outputs, and for decoding its state, read and written."""
    from openagents_b200.ops import cuda_ops as ops
    bench = _Timer(dev, reps)
    dl, sd, at = (next(l.mixer for l in cfg.layers if l.mixer.kind == k) for k in ("delta", "ssd", "attention"))
    mix = next(l for l in cfg.layers if l.moe)
    d, T, B, ctx, eps = cfg.d_model, PROMPT, 64, PROMPT, 1e-6
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev)                       # noqa: E731
    bf = lambda *s: torch.randn(*s, device=dev).bfloat16()             # noqa: E731
    hf = lambda *s: torch.randn(*s, device=dev).half()                 # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)     # noqa: E731
    for n in (T, B, 1):
        x, y, hb, gn = rnd(n, d), rnd(n, d), bf(n, d), rnd(d)
        bench(f"norm_residual behind only [{n}]", lambda: ops.norm_residual(x, eps, y=y, gy=gn, hb=hb), n * d * 14, like=f"rmsnorm [{n}]")
        bench(f"rmsnorm [{n}]", lambda: ops.rmsnorm(x, gn, eps, hb=hb), n * d * 6)
    # ---- recurrences
    H, D, r = dl.heads, dl.dim, dl.rank
    hd, ld = H * D, (5 * H * D + r + 7) // 8 * 8
    w2, w0, ab, gain = bf(hd, (r + 7) // 8 * 8), rnd(hd) - 3, rnd(hd), rnd(hd)
    Hg, dk, dv, rg = d // 256, 128, 256, 16
    qk, vv = Hg * dk, Hg * dv
    lg = (2 * qk + 2 * vv + rg + 7) // 8 * 8
    go = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
    a2, b2, wg = rnd(rg, qk), rnd(qk), rnd(dv)
    Hs, P, N, G = sd.heads, sd.vdim, sd.dim, sd.groups
    inner, ls = Hs * P, (sd.heads * sd.vdim + sd.channels + sd.heads + 7) // 8 * 8
    conv, cb, dtb, A, skip, sn = rnd(sd.channels, sd.conv), rnd(sd.channels), rnd(Hs) - 3, rnd(Hs), rnd(Hs), rnd(inner)
    offs = tuple(i * hd for i in range(6))
    s1, s2, s3, ring = rnd(B, H, D, D), rnd(B, Hs, N, P), rnd(B, Hg, dk, dv), rnd(B, sd.conv, sd.channels)
    for seqs in (1, 4):
        n = seqs * T
        qs, ql, sl = i32([T * b for b in range(seqs)]), i32([T] * seqs), i32(list(range(seqs)))
        row, out = rnd(n, ld), bf(n, hd)
        ws = torch.empty(ops.delta_chunk_bytes(n, seqs, H, D, D, dl.log_decay), dtype=torch.uint8, device=dev)
        bench(f"delta_chunked [{seqs} x {T}] (3 kernels)", lambda: ops.delta_chunked(row, offs, r, w2, w0, ab, gain, s1, qs, ql, ql, sl, seqs, H, D, D, D, dl.log_decay, eps, out,
                                                                                     max_q=T, ws=ws), n * (ld * 4 + hd * 2), like=f"gla_chunked [{seqs} x {T}] (3 kernels)")
        row, y = rnd(n, ls), rnd(n, inner)
        ws = torch.empty(ops.ssd_prefill_bytes(n, seqs, Hs, P, N, G), dtype=torch.uint8, device=dev)
        bench(f"ssd_prefill [{seqs} x {T}] (3 kernels)", lambda: ops.ssd_prefill(row, inner, inner + sd.channels, conv, cb, dtb, A, skip, s2, ring, qs, ql, ql, sl, seqs, Hs, P, N, G, P, y,
                                                                                 max_q=T, ws=ws), n * ((sd.channels + Hs) * 4 + inner * 4), like=f"gla_chunked [{seqs} x {T}] (3 kernels)")
        row, out = rnd(n, lg), bf(n, vv)
        ws = torch.empty(ops.gla_chunk_bytes(n, seqs, Hg, dk, dv, rg), dtype=torch.uint8, device=dev)
        bench(f"gla_chunked [{seqs} x {T}] (3 kernels)", lambda: ops.gla_chunked(row, go, rg, a2, b2, wg, s3, qs, ql, ql, sl, seqs, Hg, dk, dv, dv, 16.0, dk ** -0.5, eps, T, ws, out_bf16=out),
              n * (lg * 4 + vv * 2))
    for n in (B, 1):
        sl, one, held = i32(list(range(n))), i32([1] * n), i32([ctx] * n)
        row, out = rnd(n, ld), bf(n, hd)
        bench(f"delta_recurrent [{n}]", lambda: ops.delta_recurrent(row, offs, r, w2, w0, ab, gain, s1, sl, one, held, sl, n, H, D, D, D, dl.log_decay, eps, out),
              n * (8 * H * D * D + ld * 4 + hd * 2) + w2.numel() * 2, like=f"gla_recurrent [{n}]")
        row2, y, ws = rnd(n, ls), rnd(n, inner), torch.empty(ops.ssd_decode_bytes(n, Hs, P, N, G), dtype=torch.uint8, device=dev)
        bench(f"ssd_decode [{n}]", lambda: ops.ssd_decode(row2, inner, inner + sd.channels, conv, cb, dtb, A, skip, s2, ring, sl, one, held, sl, n, Hs, P, N, G, P, y, ws=ws),
              n * (8 * Hs * N * P + (1 + sd.conv) * sd.channels * 4 + inner * 4), like=f"gla_recurrent [{n}]")
        row3, out3 = rnd(n, lg), bf(n, vv)
        bench(f"gla_recurrent [{n}]", lambda: ops.gla_recurrent(row3, go, rg, a2, b2, wg, s3, sl, one, held, sl, n, Hg, dk, dv, dv, 16.0, dk ** -0.5, eps, out_bf16=out3),
              n * (8 * Hg * dk * dv + lg * 4))
    for n in (T, B, 1):
        y, z, o = rnd(n, inner), rnd(n, ls), bf(n, inner)
        bench(f"group_norm gated [{n} x {inner}]", lambda: ops.group_norm(y, inner, sd.norm_groups, sn, eps, o, gate=z[:, :inner]), n * inner * 10, like=f"rmsnorm [{n}]")
    # ---- attention's projections
    Hq, G, D = at.heads, at.kv_heads, at.dim
    nq, nk, pages = Hq * D, G * D, (ctx + 15) // 16
    wq, wk, lam = rnd(nq), rnd(nk), torch.full((1,), 0.3, device=dev)
    for n, seqs in ((T, 1), (B, B), (1, 1)):
        row, first = rnd(n, nq + 2 * nk), rnd(n, nk)
        pos, slot = i32([ctx - 1] * n if n != T else list(range(n))), i32(list(range(n)))
        kc, vc = hf(seqs * pages + 1, G, 16, D), hf(seqs * pages + 1, G, 16, D)
        q16, q32, tab = hf(n, nq), rnd(n, nq), ops.rope_table(ctx, at.rope_dims, at.rope_base, dev, at.rope_frequencies())
        tabf = ops.rope_table(ctx, D, at.rope_base, dev)
        q = dict(q16=q16) if n == T else dict(q32=q32)
        nb = n * ((nq + 2 * nk) * 4 + nq * (2 if n == T else 4) + 2 * nk * 2)
        bench(f"row_qkv_finish mixing [{n}]", lambda: ops.row_qkv_finish(row, 0, nq, nq + nk, wq, wk, pos, slot, tab, Hq, G, D, D, D, D, at.rope_dims, 1, True, eps, at.scale, 16, kc, vc,
                                                                         lam=lam, v_first=first, **q), nb + n * nk * 4, like=f"rope_kv [{n}]")
        bench(f"rope_kv [{n}]", lambda: ops.rope_kv(row, pos, slot, None if n == T else q32, q16 if n == T else None, kc, vc, Hq, G, D, 16, at.rope_base, 0, at.scale, table=tabf), nb)
        del kc, vc
    # ---- products
    for n in (T, B):
        a = bf(n, d)
        for nm, cols in (("gemm delta projection", ld), ("gemm mamba projection", ls), ("gemm qkv", nq + 2 * nk)):
            wt, o3 = bf(cols, d), torch.zeros(n, cols, device=dev)
            bench(f"{nm} [{n}]", lambda: ops.gemm_bf16(a, wt, n, cols, d, out_f32=o3, accumulate=n <= 64, status=st), cols * d * 2 + n * (d * 2 + cols * 4), 2.0 * n * cols * d,
                  like=None if nm == "gemm qkv" else f"gemm qkv [{n}]")
    # ---- experts
    E, top, F, scale = mix.moe.experts, mix.moe.top, mix.ffn, mix.moe.scale
    w13, w1, w2e, router = bf(E * 2 * F, d) * 0.02, bf(E * F, d) * 0.02, bf(E * d, F) * 0.02, rnd(E, d) * 0.02
    for n in (T, B):
        cap = (n + 127) // 128 * 128
        rx, mid, meta, rw = bf(E * cap, d), bf(E * cap, F), torch.zeros(E * cap, 2, dtype=torch.int32, device=dev), rnd(E * cap)
        h, x, ids, w = bf(n, d), rnd(n, d), torch.zeros(n, top, dtype=torch.int32, device=dev), rnd(n, top)
        cnt = torch.zeros(64, E, dtype=torch.int32, device=dev)
        used = min(E, n * top)
        for nm, sc, like in (("route and dispatch, scaled", scale, "route and dispatch"), ("route and dispatch", 1.0, None)):
            cnt.zero_()
            turn = iter(range(64))
            bench(f"{nm} [{n}]", lambda: ops.moe_route_dispatch(h, None, router, None, top, E, cap, rx.data_ptr(), meta.data_ptr(), rw.data_ptr(), cnt[next(turn)].data_ptr(), None,
                                                                topk_ids=ids, topk_w=w, status=st, scale=sc), n * d * 2 * (1 + top) + E * d * 4, like=like and f"{like} [{n}]")
        bench(f"experts up, relu2 [{n}]", lambda: ops.moe_gemm(rx, w1, E, cap, F, d, cnt[0], 3, out_bf16=mid, ldc=F, status=st, live_rows=n * top),
              used * F * d * 2 + n * top * (d + F) * 2, 2.0 * n * top * F * d, like=f"experts gate/up [{n}]")
        bench(f"experts gate/up [{n}]", lambda: ops.moe_gemm(rx, w13, E, cap, 2 * F, d, cnt[0], 1, out_bf16=mid, ldc=F, status=st, live_rows=n * top),
              used * 2 * F * d * 2 + n * top * (d + F) * 2, 4.0 * n * top * F * d)
        bench(f"experts down [{n}]", lambda: ops.moe_gemm(mid, w2e, E, cap, d, F, cnt[0], 2, ldc=d, meta=meta, gate_w=rw, sym_off=x.data_ptr(), status=st, live_rows=n * top),
              used * F * d * 2 + n * top * (F * 2 + d * 4), 2.0 * n * top * F * d)
        Fs = mix.moe.shared
        if Fs:
            up, dn, act, y = bf(Fs, d), bf(d, Fs), bf(n, Fs), torch.zeros(n, d, device=dev)
            bench(f"gemm shared up [{n}]", lambda: ops.gemm_bf16(h, up, n, Fs, d, out_bf16=act, act=ops.ACT_RELU2, status=st), (Fs * d + n * (d + Fs)) * 2, 2.0 * n * Fs * d, like=f"gemm qkv [{n}]")
            bench(f"gemm shared down [{n}]", lambda: ops.gemm_bf16(act, dn, n, d, Fs, out_f32=y, accumulate=n <= 64, status=st), (Fs * d + n * Fs) * 2 + n * d * 4, 2.0 * n * Fs * d, like=f"gemm qkv [{n}]")
    h, x, ids, w, mid = rnd(1, d), rnd(1, d), i32([list(range(top))]), rnd(1, top), rnd(1, top, F)
    bench("expert_up [1]", lambda: ops.expert_up(h, w1, F, ids, w, mid), top * F * d * 2, like="expert_gate_up [1]")
    bench("expert_gate_up [1]", lambda: ops.expert_gate_up(h, w13, F, ids, w, mid), top * 2 * F * d * 2)
    bench("expert_down [1]", lambda: ops.expert_down(mid, w2e, d, ids, x), top * F * d * 2)
    return bench.rows


def time_kernels(cfg, dev, reps: int = 12) -> list[dict]:
    """Every kernel of one hybrid layer pair at 2048 prompt tokens and at a 64-sequence decode step, and its Llama counterpart."""
    from openagents_b200.ops import cuda_ops as ops
    bench = _Timer(dev, reps)
    at = next(l.mixer for l in cfg.layers if l.mixer.kind == "attention")
    gl = next(l.mixer for l in cfg.layers if l.mixer.kind == "gla")
    d, F, T, B, ctx = cfg.d_model, cfg.ffn, PROMPT, 64, PROMPT
    H, G, D = at.heads, at.kv_heads, at.dim
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev)                       # noqa: E731
    bf = lambda *s: torch.randn(*s, device=dev).bfloat16()             # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)     # noqa: E731
    # ---- norms and residual
    for n in (T, B):
        x, y, hb, gn = rnd(n, d), rnd(n, d), bf(n, d), rnd(d)
        bench(f"norm_residual [{n}]", lambda: ops.norm_residual(x, 1e-6, y=y, gy=gn, gh=gn, hb=hb), n * d * 14, like=f"rmsnorm [{n}]")
        bench(f"rmsnorm [{n}]", lambda: ops.rmsnorm(x, gn, 1e-6, hb=hb), n * d * 6)
    # ---- attention: projection finish, prompt, decode
    pages = (ctx + 15) // 16
    for n, seqs in ((T, 1), (B, B), (1, 1)):
        N = (H + 2 * G) * D + (H + 7) // 8 * 8
        row, pos, slot = rnd(n, N), i32([ctx - 1] * n if n != T else list(range(n))), i32(list(range(n)))
        q16, q32 = bf(n, H * D).half(), rnd(n, H * D)
        kc, vc = rnd(seqs * pages + 1, G, 16, D).half(), rnd(seqs * pages + 1, G, 16, D).half()
        tab, tabf = ops.rope_table(ctx, at.rope_dims, at.rope_base, dev), ops.rope_table(ctx, D, at.rope_base, dev)
        nb = n * ((H + 2 * G) * D * 4 + H * D * (2 if n == T else 4) + 2 * G * D * 2)
        q = dict(q16=q16) if n == T else dict(q32=q32)
        bench(f"qkv_finish [{n}]", lambda: ops.qkv_finish(row, 0, H * D, (H + G) * D, pos, slot, tab, at.rope_base, H, G, D, D, D, D,
                                                         at.rope_dims, 0, True, 1e-6, at.scale, 16, kc=kc, vc=vc, **q), nb, like=f"rope_kv [{n}]")
        row2 = row[:, : (H + 2 * G) * D].contiguous()
        bench(f"rope_kv [{n}]", lambda: ops.rope_kv(row2, pos, slot, None if n == T else q32, q16 if n == T else None, kc, vc, H, G, D, 16, at.rope_base,
                                                    0, at.scale, table=tabf), nb)
        table, gate = i32(list(range(seqs * pages))).view(seqs, pages), row[:, (H + 2 * G) * D:]
        lens = i32([ctx] * seqs)
        if n == T:
            o, z = bf(T, H * D), i32([0])
            fl = 4.0 * T * T / 2 * H * D
            for nm, gt, lk in (("attn_prefill_tc05 gated", gate, "attn_prefill_tc05"), ("attn_prefill_tc05", None, None)):
                bench(f"{nm} [{T}]", lambda: ops.attn_prefill_tc05(q16, kc, vc, table, z, lens, lens, 1, T, H, G, out_bf16=o, status=st, dk=D, dv=D, gate=gt),
                      T * (H + G) * D * 4, fl, like=lk and f"{lk} [{T}]")
        else:
            o, S = bf(n, H * D), 4
            sc, cnt = rnd(ops.attn_decode_scratch_floats(n, H, G, D, S)), torch.zeros(n * H, dtype=torch.int32, device=dev)
            for nm, gt, lk in (("attn_decode gated", gate, "attn_decode"), ("attn_decode", None, None)):
                bench(f"{nm} [{n} x {ctx}]", lambda: ops.attn_decode(q32, kc, vc, table, lens, n, H, G, D, S=S, gate=gt, out_bf16=o, scratch=sc, counters=cnt,
                                                                     status=st), n * ctx * G * D * 4, like=lk and f"{lk} [{n} x {ctx}]")
    # ---- gated linear attention
    Hg, dk, dv, r = gl.heads, gl.dim, gl.vdim, gl.rank
    qk, vv = Hg * dk, Hg * dv
    ld = (2 * qk + 2 * vv + r + 7) // 8 * 8
    offs = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
    a2, b2, w = rnd(r, qk), rnd(qk), rnd(dv)
    state = torch.zeros(B, Hg, dk, dv, device=dev)
    for seqs in (1, 4):
        n = seqs * T
        row, out = rnd(n, ld), bf(n, vv)
        ws = torch.empty(ops.gla_chunk_bytes(n, seqs, Hg, dk, dv, r), dtype=torch.uint8, device=dev)
        qs, ql, sl = i32([T * b for b in range(seqs)]), i32([T] * seqs), i32(list(range(seqs)))
        fl = n * Hg * (4.0 * dk * dv + 64 * (dk + dv))
        bench(f"gla_chunked [{seqs} x {T}] (3 kernels)", lambda: ops.gla_chunked(row, offs, r, a2, b2, w, state, qs, ql, ql, sl, seqs, Hg, dk, dv, dv, 16.0, dk ** -0.5,
                                                                                   1e-6, T, ws, out_bf16=out), n * (ld * 4 + vv * 2), fl, like=f"attn_prefill_tc05 [{T}]")
    for n in (1, B):
        row, out, sl, one, held = rnd(n, ld), bf(n, vv), i32(list(range(n))), i32([1] * n), i32([ctx] * n)
        bench(f"gla_recurrent [{n}]", lambda: ops.gla_recurrent(row, offs, r, a2, b2, w, state, sl, one, held, sl, n, Hg, dk, dv, dv, 16.0, dk ** -0.5, 1e-6,
                                                                out_bf16=out), n * (8 * Hg * dk * dv + ld * 4), like=f"attn_decode [{n} x {ctx}]")
    # ---- products
    for n in (T, B):
        a, up, gu = bf(n, d), bf(F, d), bf(2 * F, d)
        o1, o2 = bf(n, F), bf(n, F)
        bench(f"gemm relu2 up [{n} x {F} x {d}]", lambda: ops.gemm_bf16(a, up, n, F, d, out_bf16=o1, act=ops.ACT_RELU2, status=st), (F * d + n * (d + F)) * 2, 2.0 * n * F * d,
              like=f"gemm swiglu gate/up [{n} x {2 * F} x {d}]")
        bench(f"gemm swiglu gate/up [{n} x {2 * F} x {d}]", lambda: ops.gemm_bf16(a, gu, n, 2 * F, d, out_bf16=o2, ldc=F, act=ops.ACT_SWIGLU_PAIR, status=st),
              (2 * F * d + n * (d + F)) * 2, 4.0 * n * F * d)
        for nm, N in (("gemm gla projection", ld), ("gemm qkv projection", (H + 2 * G) * D)):
            wt, o3 = bf(N, d), torch.zeros(n, N, device=dev)
            bench(f"{nm} [{n} x {N} x {d}]", lambda: ops.gemm_bf16(a, wt, n, N, d, out_f32=o3, accumulate=n <= 64, status=st), N * d * 2 + n * (d * 2 + N * 4), 2.0 * n * N * d)
    lg = rnd(B, cfg.vocab)
    bench(f"logits_finish [{B} x {cfg.vocab}]", lambda: ops.logits_finish(lg, 0.5, 30.0), 8 * B * cfg.vocab)
    return bench.rows


def run(args) -> dict:
    from openagents_b200.models.config import PRESETS
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    cfg = PRESETS[args.model]
    llama_cfg = like_llama(cfg)
    ours, llama = time_engine(cfg, dev, args.steps, max(3, args.warmup)), time_engine(llama_cfg, dev, args.steps, max(3, args.warmup))
    return {"workload": "hybrid", "model": cfg.name, "dtype": "bf16", "data": "synthetic", "prompt": PROMPT, "peaks": peaks()[2], "hybrid": ours,
            "moe_equal_size" if llama_cfg.n_experts else "llama_equal_size": llama,
            "kernels": {"pesorax": time_pesorax_kernels, "kazolorn": time_kazolorn_kernels, "tekosun": time_tekosun_kernels}.get(cfg.arch, time_kernels)(cfg, dev)}
