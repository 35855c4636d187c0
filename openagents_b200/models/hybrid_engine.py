"""Engine for hybrid stacks: softmax attention over the paged cache and gated linear attention with a state slot per sequence,
layer by layer in the order the configuration gives, a norm on both sides of every sublayer.

Batching, pages, state slots, CUDA graphs and the public operations are ``PagedEngine``'s.  A step runs, per sublayer:
``norm_residual`` (the previous sublayer's norm, the residual sum, this one's norm, in one pass), one fused projection
(queries, keys, values, gates in one matrix), the mixer, and the output projection into an fp32 row that the next
``norm_residual`` takes.  The residual stream, norms, rotations, scores, decays and states are fp32 in both modes.

``dtype`` "bfloat16": projections and activations in bf16 on the tensor cores (up to ``small_path_tokens`` decoded tokens: the
bf16 mat-vec on fp32 activations), fp16 keys and values.  "float32": fp32 activations, keys and values throughout, products on
the CUDA cores (the weights are bf16 numbers, whose expansion is exact).
"""
from __future__ import annotations

import os
from dataclasses import dataclass

import torch

from ..ops import cuda_ops as ops
from .config import LayerSpec, MixerSpec, ModelConfig
from .engine import MATVEC_MAX_TOKENS, QGEMM_MAX_TOKENS
from .paged import PAGE, PagedEngine
from .qweight import WeightSource


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass
class _Lin:
    """A bf16 [N][K] matrix with both sizes padded to multiples of 8 (zeros)."""
    w: torch.Tensor

    @property
    def N(self):
        return self.w.shape[0]

    @property
    def K(self):
        return self.w.shape[1]


@dataclass
class _Block:
    spec: LayerSpec
    norm1: torch.Tensor
    norm1b: torch.Tensor
    proj: _Lin
    out: _Lin
    DK: int = 0                  # attention: padded head sizes of queries / keys and values;  gla: DV is the padded value size
    DV: int = 0
    tc: bool = False             # attention: the tensor-core kernels take these head sizes
    kv: int = -1                 # index of the key / value cache this layer reads
    table: torch.Tensor | None = None
    a2: torch.Tensor | None = None
    b2: torch.Tensor | None = None
    o_norm: torch.Tensor | None = None
    state: torch.Tensor | None = None
    norm2: torch.Tensor | None = None
    norm2b: torch.Tensor | None = None
    up: _Lin | None = None
    down: _Lin | None = None


class HybridEngine(PagedEngine):
    ARCHS = ("folirax",)
    world = 1                    # one GPU; the serving layer asks
    vocab_sharded = False

    def __init__(self, cfg: ModelConfig, src: WeightSource, device="cuda", max_batch: int = 64, max_ctx: int = 4096,
                 n_pages: int | None = None, max_tokens: int = 4096, dtype: str = "bfloat16", state_slots: int | None = None,
                 canaries: bool | None = None):
        if cfg.arch not in self.ARCHS or not cfg.layers:
            raise ValueError(f"{type(self).__name__} serves {self.ARCHS} models, not {cfg.arch!r}")
        self.cfg, self.d = cfg, cfg.d_model
        self.exact = dtype == "float32"
        # one state slot per sequence that is open: the running ones, and some for idle sessions and scoring
        slots = 0 if not cfg.has_state else (state_slots if state_slots is not None else max_batch + max(4, max_batch // 4))
        self._init_paged(device, max_batch, max_ctx, n_pages, max_tokens, canaries, state_slots=slots)
        self.dp = _up(self.d, 8)
        # Decode batches up to this size take the mat-vec kernels.  Measured (ms per step, one token, mat-vec / GEMM): width 2048
        # 1.04 / 1.30, width 4096 4.41 / 4.19; the GEMM costs the same at eight tokens, the mat-vec grows with each.
        self.small_path_tokens = min(MATVEC_MAX_TOKENS, int(os.environ.get("B200_SMALL_PATH_TOKENS", 1)))
        self._load(src)
        self._alloc()

    # ------------------------------------------------------------------ weights
    def _lin(self, w: torch.Tensor) -> _Lin:
        N, K = w.shape
        out = torch.zeros((_up(N, 8), _up(K, 8)), dtype=torch.bfloat16, device=self.device)
        out[:N, :K] = w.to(self.device)
        return _Lin(out)

    def _matrix(self, src: WeightSource, name: str) -> torch.Tensor:
        return src.get(name).to_float().to(torch.bfloat16)

    def _vector(self, src: WeightSource, name: str, centred: bool = False) -> torch.Tensor:
        v = src.get(name).to_float().to(self.device).contiguous()
        return v + 1.0 if centred else v

    def _out_proj(self, src: WeightSource, name: str, heads: int, vdim: int, pad: int) -> _Lin:
        """The output projection with every head's columns padded to the mixer's output row."""
        w = self._matrix(src, name).view(self.d, heads, vdim)
        return self._lin(torch.nn.functional.pad(w, (0, pad - vdim)).reshape(self.d, heads * pad))

    def _load(self, src: WeightSource):
        cfg = self.cfg
        self.emb = self._matrix(src, "embed").to(self.device).contiguous()
        self.blocks: list[_Block] = []
        tables: dict[tuple, torch.Tensor] = {}
        n_kv = 0
        for i, spec in enumerate(cfg.layers):
            m, p = spec.mixer, f"l{i}."
            names = ["q", "k", "v", "g", "a1"] if m.kind == "gla" else ["q"] + (["k", "v"] if m.kv_from is None else []) + (["g"] if m.head_gate else [])
            proj = self._lin(torch.cat([self._matrix(src, f"{p}mix.{n}") for n in names]))
            b = _Block(spec, self._vector(src, p + "norm1", True), self._vector(src, p + "norm1b", True), proj, None)
            if m.kind == "gla":
                b.DV = _up(m.vdim, 8)
                b.a2 = src.get(p + "mix.a2").to_float().to(self.device).t().contiguous()
                b.b2, b.o_norm = self._vector(src, p + "mix.a2.b"), self._vector(src, p + "mix.norm")
                b.state = torch.zeros((self.state_slots, m.heads, m.dim, b.DV), dtype=torch.float32, device=self.device)
            else:
                b.DK, b.DV, b.tc = self._head_pad(m)
                if m.kv_from is None:
                    b.kv, n_kv = n_kv, n_kv + 1
                else:
                    b.kv = self.blocks[m.kv_from].kv
                if m.rope_dims:
                    key = (m.rope_base, m.rope_dims)
                    if key not in tables:
                        tables[key] = ops.rope_table(self.max_pages * PAGE, m.rope_dims, m.rope_base, self.device)
                    b.table = tables[key]
            b.out = self._out_proj(src, p + "mix.o", m.heads, m.vdim, b.DV)
            if spec.ffn:
                b.norm2, b.norm2b = self._vector(src, p + "norm2", True), self._vector(src, p + "norm2b", True)
                b.up, b.down = self._lin(self._matrix(src, p + "mlp.up")), self._lin(self._matrix(src, p + "mlp.down"))
            self.blocks.append(b)
        self.final_norm = self._vector(src, "final.norm", True)
        self.head = self._lin(self._matrix(src, "head"))
        torch.cuda.synchronize(self.device)

    def _head_pad(self, m: MixerSpec) -> tuple[int, int, bool]:
        """Padded head sizes in the cache, and whether the tensor-core attention kernels take them (else, and always in the 32-bit
        mode, the any-size kernel runs)."""
        dk, dv = _up(m.dim, 64), _up(m.vdim, 64)
        if self.exact or dk > 256 or dv > 128:
            return _up(m.dim, 8), _up(m.vdim, 8), False
        return dk, dv, True

    def weight_bytes(self) -> int:
        n = self.head.w.numel()
        for b in self.blocks:
            n += b.proj.w.numel() + b.out.w.numel() + (b.up.w.numel() + b.down.w.numel() if b.up is not None else 0)
        return 2 * n

    def scratch_bytes(self) -> int:
        return 0

    # ------------------------------------------------------------------ workspaces
    def _alloc(self):
        T, d, dev = self.max_tokens, self.dp, self.device
        f32, bf = torch.float32, torch.bfloat16
        self._alloc_batch()
        own = [b for b in self.blocks if b.spec.mixer.kind == "attention" and b.spec.mixer.kv_from is None]
        ct = f32 if self.exact else torch.float16
        self.kc = [torch.zeros((self.n_pages, b.spec.mixer.kv_heads, PAGE, b.DK), dtype=ct, device=dev) for b in own]
        self.vc = [torch.zeros((self.n_pages, b.spec.mixer.kv_heads, PAGE, b.DV), dtype=ct, device=dev) for b in own]
        ws = self._ws
        n_proj = max(b.proj.N for b in self.blocks)
        n_mix = max(b.out.K for b in self.blocks)
        n_ffn = max((b.up.N for b in self.blocks if b.up is not None), default=8)
        attn = [b for b in self.blocks if b.spec.mixer.kind == "attention"]
        n_q = max((b.spec.mixer.heads * b.DK for b in attn), default=8)
        n_q32 = max((b.spec.mixer.heads * b.DK for b in attn if not b.tc), default=0)      # rows of a prompt in fp32
        self.x = ws("x", (T, self.d), f32)
        self.y = ws("y", (T, d), f32, zero=True)
        self.proj = ws("proj", (T * n_proj,), f32, zero=True)
        self.q32 = ws("q32", (max(T * n_q32, self.max_batch * n_q),), f32)
        self.q16 = ws("q16", (T * n_q if any(b.tc for b in attn) else 8,), torch.float16)
        tc = [(b.spec.mixer, b.DV) for b in attn if b.tc]
        self.attn_scratch = ws("attn_scratch", (max((ops.attn_decode_scratch_floats(self.max_batch, m.heads, m.kv_heads, dv, self.max_splits)
                                                     for m, dv in tc), default=4),), f32)
        self.attn_counters = ws("attn_counters", (self.max_batch * max((m.heads for m, _ in tc), default=1),), torch.int32, zero=True)
        gla = [b for b in self.blocks if b.spec.mixer.kind == "gla"]
        self.gla_ws = ws("gla_ws", (max((ops.gla_chunk_bytes(T, self.max_batch, m.heads, m.dim, dv, m.rank)
                                         for m, dv in ((b.spec.mixer, b.DV) for b in gla)), default=0) if not self.exact else 0,), torch.uint8)
        small = self.max_batch if not self.exact else T            # rows of the fp32 activations
        self.hf = ws("hf", (small * d,), f32)
        self.mf = ws("mf", (small * n_mix,), f32)
        self.ff = ws("ff", (small * n_ffn,), f32)
        big = 1 if self.exact else T
        self.hb = ws("hb", (big * d,), bf)
        self.mb = ws("mb", (big * n_mix,), bf)
        self.fb = ws("fb", (big * n_ffn,), bf)
        self.V = self.cfg.vocab
        self.logits = ws("logits", (self.max_batch, self.V), f32)
        self.argmax_scratch = ops.argmax_scratch(self.max_batch, dev)
        self.iota = torch.arange(self.max_batch, dtype=torch.int32, device=dev)
        self.ones = torch.ones(self.max_batch, dtype=torch.int32, device=dev)
        k_max = max(d, n_mix, n_ffn)
        # the bf16 mat-vec keeps its fp32 activations in shared memory
        self.matvec_rows = max((n for n in (1, 2, 4, 8) if n * (k_max * 4 + 256) <= 200 * 1024), default=0)

    # ------------------------------------------------------------------ building blocks
    def _mm(self, a: torch.Tensor, L: _Lin, out: torch.Tensor, act: int = 0, add: bool = False):
        """out = act(a W^T).  fp32 activations: mat-vec for a few rows, else the 32-bit product; bf16: the tensor-core GEMM (``add``:
        the output was zeroed ahead, K may be split)."""
        T = a.shape[0]
        if a.dtype == torch.float32:
            if T <= self.matvec_rows:
                ops.matvec(ops.WT_BF16, L.w, None, L.N, L.K, T, xf=a, epi=ops.EPI_RELU2 if act else ops.EPI_STORE, y=out, ldy=out.stride(0))
            else:
                ops.gemm_f32(a, L.w, out, act)
        else:
            f32 = out.dtype == torch.float32
            ops.gemm_bf16(a, L.w, T, L.N, L.K, lda=a.stride(0), ldb=L.K, out_f32=out if f32 else None, out_bf16=None if f32 else out,
                          ldc=out.stride(0), act=ops.ACT_RELU2 if act else ops.ACT_NONE, accumulate=add and f32 and not act, status=self.status)

    def _attention(self, b: _Block, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        cfg, m = self.cfg, b.spec.mixer
        own = m.kv_from is None
        k_off = m.heads * m.dim if own else -1
        v_off = k_off + m.kv_heads * m.dim
        g_off = v_off + m.kv_heads * m.vdim if own else m.heads * m.dim
        kc, vc = self.kc[b.kv], self.vc[b.kv]
        tc_prompt = b.tc and not decode
        q = (self.q16 if tc_prompt else self.q32)[: T * m.heads * b.DK].view(T, -1)
        ops.qkv_finish(proj, 0, k_off, v_off, self.pos, self.slot, b.table, m.rope_base, m.heads, m.kv_heads, m.dim, m.vdim, b.DK, b.DV,
                       m.rope_dims, 0 if m.rope_style == "pairs" else 1, m.qk_norm, cfg.norm_eps, m.scale, PAGE, q32=None if tc_prompt else q,
                       q16=q if tc_prompt else None, kc=kc, vc=vc)
        gate = proj[:, g_off:] if m.head_gate else None
        if tc_prompt:
            ops.attn_prefill_tc05(q, kc, vc, self.page_table, self.q_start, self.q_len, self.seq_lens, n_seqs, max_q, m.heads, m.kv_heads,
                                  out_bf16=o16, status=self.status, dk=b.DK, dv=b.DV, gate=gate)
            return 2
        if b.tc:
            ops.attn_decode(q, kc, vc, self.page_table, self.seq_lens, n_seqs, m.heads, m.kv_heads, b.DK, dv=b.DV,
                            S=self._attn_splits(n_seqs, m.kv_heads, pages), gate=gate, out_f32=o32, out_bf16=o16,
                            scratch=self.attn_scratch, counters=self.attn_counters, status=self.status)
            return 2
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        ops.attn_exact(q, kc, vc, self.page_table, qs, ql, self.seq_lens, n_seqs, max_q, m.heads, m.kv_heads, b.DK, b.DV, gate=gate,
                       out_f32=o32, out_bf16=o16)
        return 2

    def _gla(self, b: _Block, proj, T: int, decode: bool, n_seqs: int, max_q: int, o32, o16) -> int:
        m = b.spec.mixer
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        offs = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        args = (proj, offs, m.rank, b.a2, b.b2, b.o_norm, b.state, qs, ql, self.seq_lens, self.state_slot, n_seqs, m.heads, m.dim, m.vdim, b.DV,
                m.tau, m.dim ** -0.5, self.cfg.norm_eps)
        if decode or self.exact or not ops.gla_chunk_bytes(T, n_seqs, m.heads, m.dim, b.DV, m.rank):
            ops.gla_recurrent(*args, out_f32=o32, out_bf16=o16)
            return 1
        ops.gla_chunked(*args, max_q, self.gla_ws, out_f32=o32, out_bf16=o16)
        return 3

    def _run_layers(self, T: int, decode: bool, n_seqs: int, max_q: int, pages: int) -> int:
        eps, x, y = self.cfg.norm_eps, self.x[:T], self.y[:T]
        f32 = self.exact or (decode and T <= min(self.small_path_tokens, self.matvec_rows))
        h = (self.hf if f32 else self.hb)[: T * self.dp].view(T, self.dp)
        hk = dict(hf=h) if f32 else dict(hb=h)
        add = not f32 and T <= QGEMM_MAX_TOKENS          # one row tile: the projections may split K and add into zeroed outputs
        gy, n = None, 0
        for b in self.blocks:
            proj = self.proj[: T * b.proj.N].view(T, b.proj.N)
            mix = (self.mf if f32 else self.mb)[: T * b.out.K].view(T, b.out.K)
            ops.norm_residual(x, eps, y=y if gy is not None else None, gy=gy, gh=b.norm1, y_clear=add, zero=proj if add else None,
                              zero2=y if add and gy is None else None, **hk)
            self._mm(h, b.proj, proj, add=add)
            o = (mix, None) if f32 else (None, mix)
            if b.spec.mixer.kind == "gla":
                n += self._gla(b, proj, T, decode, n_seqs, max_q, *o)
            else:
                n += self._attention(b, proj, T, decode, n_seqs, max_q, pages, *o)
            self._mm(mix, b.out, y, add=add)
            gy, n = b.norm1b, n + 3
            if b.up is not None:
                act = (self.ff if f32 else self.fb)[: T * b.up.N].view(T, b.up.N)
                ops.norm_residual(x, eps, y=y, gy=gy, gh=b.norm2, y_clear=add, **hk)
                self._mm(h, b.up, act, act=1)
                self._mm(act, b.down, y, add=add)
                gy, n = b.norm2b, n + 3
        if decode:
            self._tail = gy                              # the last residual step is folded into the final norm
        else:
            self._tail = None
            ops.norm_residual(x, eps, y=y, gy=gy)
            n += 1
        return n

    def _head(self, rows: torch.Tensor, nb: int, greedy: bool = True):
        eps = self.cfg.norm_eps
        gy, self._tail = self._tail, None
        f32 = self.exact or nb <= min(MATVEC_MAX_TOKENS, self.matvec_rows) or self.V % 4 != 0
        y = self.y[:nb] if gy is not None else None
        h = (self.hf if f32 else self.hb)[: nb * self.dp].view(nb, self.dp)
        ops.norm_residual(rows, eps, y=y, gy=gy, gh=self.final_norm, **(dict(hf=h) if f32 else dict(hb=h)))
        w = _Lin(self.head.w[: self.V])
        out = self.logits[:nb]
        step = max(1, self.matvec_rows) if f32 and not self.exact else nb
        for lo in range(0, nb, step):
            self._mm(h[lo: lo + step], w, out[lo: lo + step])
        n = 2
        if self.cfg.logit_scale != 1.0 or self.cfg.logit_softcap > 0:
            ops.logits_finish(out, self.cfg.logit_scale, self.cfg.logit_softcap)
            n += 1
        if greedy:
            ops.argmax(out, self.out_ids, self.out_val, scratch=self.argmax_scratch)
            n += 1
        return n

    def _embed(self, T: int):
        ops.embedding(self.ids, self.x[:T], ops.EMB_BF16, self.emb, vocab_n=self.V)
