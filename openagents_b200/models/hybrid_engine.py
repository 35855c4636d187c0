"""Engine for hybrid stacks: softmax attention over the paged cache (plain, windowed, chunked, differential, with mixed heads, or in a latent space) and
recurrent layers with a state slot per sequence (gated linear attention, the generalized delta rule, Mamba-2's state-space duality), layer by layer in
the order the configuration gives.

Batching, pages, state slots, CUDA graphs and the public operations are ``PagedEngine``'s.  Three kinds of residual step: with a norm behind
every sublayer, and possibly one ahead, ``norm_residual`` (the previous sublayer's norm, the residual sum, this one's norm, in one pass) takes the fp32 row an
output projection left; with a norm ahead only (Dynamic Tanh), the output projection adds its scaled product into the residual itself and
``norm_dyt`` reads it; with parallel sublayers and a depth average, both output projections add their products, scaled per channel, into the layer's
row of a history, and ``depth_norm`` makes the next layer's row and its two norms out of that history.  Per sublayer one fused projection (queries, keys, values, gates, latents in one matrix), the mixer, and the output
projection.  A looped span of layers runs several times with the same weights; every run has a cache (or state) of its own.  The residual
stream, norms, rotations, scores, decays and states are fp32 in both modes.

Latent attention: a step's short entries (single decoded tokens, portions of a few) come first in the batch and work in the latent space,
straight on the cache; the others expand the latents of their context into keys and values and take the prompt kernel.

Mixed heads: prompts take the mixture on the queries (wide ones, on a cache row of all heads' keys), decoding takes it on the scores.

``dtype`` "bfloat16": projections and activations in bf16 on the tensor cores (up to ``small_path_tokens`` decoded tokens: the
bf16 mat-vec on fp32 activations), fp16 keys, values and latents.  "float32": fp32 activations and caches throughout, products on
the CUDA cores (the weights are bf16 numbers, whose expansion is exact).
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field

import torch

from ..ops import cuda_ops as ops
from .config import LayerSpec, MixerSpec, ModelConfig
from .engine import MATVEC_MAX_TOKENS, QGEMM_MAX_TOKENS
from .paged import PAGE, PagedEngine
from .qweight import WeightSource

MIXED_CTAS = 592             # most CTAs of a mixed-head decode launch that splits the keys
LATENT_CTAS = 592            # most CTAs of a latent decode launch that splits the keys
DEPTH_GROUP = 4              # depth averages that share one reading of the results so far
MOE_EXPERTS, MOE_TOP = 256, 32   # most experts of a layer, and of a token
DELTA_DIM, DELTA_RANK = 256, 1024    # largest heads of the delta rule, and rank of its decay
SSD_DIM = 256                # largest state and value sizes of a state-space head
SHORT_TOKENS = 16            # latent attention: entries of up to this many new tokens work in the latent space
ALONE = ("polynorm", "swiglu")   # activations that are no epilogue of the up projection
ACTS = {None: (ops.EPI_STORE, ops.ACT_NONE, 0), "relu2": (ops.EPI_RELU2, ops.ACT_RELU2, 1), "gelu": (ops.EPI_GELU_ERF, ops.ACT_GELU_ERF, 2)}


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def _state_pad(vdim: int) -> int:
    """Columns of a state row: multiples of 8; wide ones divide among the CTAs of a cluster."""
    return _up(vdim, 8 if vdim <= 128 else 32)


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
class _Norm:
    """An RMS norm's weight, or Dynamic Tanh's weight, shift and scalar."""
    w: torch.Tensor
    b: torch.Tensor | None = None
    alpha: torch.Tensor | None = None


@dataclass
class _Latent:
    """A latent mixer's own weights and padded sizes.  CR / RR: columns of the latent and of the rotated key part in the cache; KN: of a head's own key
    part once expanded; QH: of a head in the query projection; offs: columns of the query latent, the latent, the rotated part and the gate."""
    CR: int
    RR: int
    KN: int
    QH: int
    offs: tuple[int, int, int, int]
    uq: _Lin
    absorb: torch.Tensor         # [heads * CR][dim]: a head's queries into the latent space
    value: torch.Tensor          # [heads * DV][CR]: a head's values out of it
    expand: _Lin | None          # [heads * (KN + DV)][CR]: every head's keys and values of a latent
    q_norm: torch.Tensor
    c_norm: torch.Tensor


@dataclass
class _Experts:
    """A mixture's weights; F: the experts' width, padded."""
    F: int
    router: torch.Tensor         # fp32 [E][dp]
    w13: torch.Tensor            # bf16 [E * 2 F][dp], rows interleaved (gate, up); experts without a gate: [E * F][dp]
    w2: torch.Tensor             # bf16 [E * dp][F]


@dataclass
class _Delta:
    """A delta-rule mixer's own weights; offs: columns of r, k, v, the output gate, the removal rate and the low-rank decay input."""
    offs: tuple[int, ...]
    w2: torch.Tensor             # bf16 [heads * dim][rank padded to 8]
    w0: torch.Tensor
    rate: torch.Tensor


@dataclass
class _Ssd:
    """A Mamba-2 mixer's own weights."""
    conv: torch.Tensor           # fp32 [channels][taps]
    conv_b: torch.Tensor
    dt_bias: torch.Tensor
    A_log: torch.Tensor
    D: torch.Tensor


@dataclass
class _Block:
    spec: LayerSpec
    norm1: _Norm | None
    norm1b: _Norm | None
    proj: _Lin
    out: _Lin
    DK: int = 0                  # attention: padded head sizes of queries / keys and values;  gla, latent: DV is the padded value size
    DV: int = 0
    tc: bool = False             # attention, latent: the tensor-core kernels take these head sizes
    dec: bool = False            # mixed heads: the decode kernel takes them (``tc``: the prompt kernel does)
    bias: torch.Tensor | None = None
    lam: torch.Tensor | None = None
    sink: torch.Tensor | None = None
    lat: _Latent | None = None
    delta: _Delta | None = None
    ssd: _Ssd | None = None
    q_norm: torch.Tensor | None = None           # norms of whole projections
    k_norm: torch.Tensor | None = None
    v_mix: torch.Tensor | None = None            # the share of the first mixing layer's values (that layer itself: None)
    table: torch.Tensor | None = None
    a2: torch.Tensor | None = None
    b2: torch.Tensor | None = None
    o_norm: torch.Tensor | None = None
    norm2: _Norm | None = None
    norm2b: _Norm | None = None
    up: _Lin | None = None
    down: _Lin | None = None
    act: torch.Tensor | None = None              # PolyNorm's four numbers
    moe: _Experts | None = None
    mix: torch.Tensor | None = None              # fp32 [heads][heads]
    mix_dec: torch.Tensor | None = None          # mixture and slopes as the decode kernel reads them
    slopes: torch.Tensor | None = None           # what a step of distance takes off a score, per head (behind the mixture)
    silent: torch.Tensor | None = None           # zeros: the scores of the silent sinks
    out_bias: torch.Tensor | None = None         # times the layer scale: joins the residual ahead of the layer
    ls1: torch.Tensor | None = None
    ls2: torch.Tensor | None = None
    average: torch.Tensor | None = None


@dataclass
class _Run:
    """One pass of a layer: which cache it reads, its state, and whether the embedding joins the residual ahead of it."""
    block: _Block
    joins: bool
    kv: int = -1                 # index among the key / value caches (latent mixers: among the latent caches)
    state: torch.Tensor | None = None
    ring: torch.Tensor | None = None             # ssd: the latest inputs of the filter, by position


@dataclass
class _Plan:
    """Layout of a step that is not a decode step: its first ``n_short`` entries (``t_short`` tokens) work in the latent space, the others expand
    their context, in groups [first, last, longest portion, longest context, rows] that fit the workspace."""
    n_short: int = 0
    t_short: int = 0
    short_pages: int = 1
    groups: list = field(default_factory=list)


def plan_latent_batch(q_len: list[int], ctx: list[int], short_rows: int, ctx_rows: int) -> tuple[_Plan, list[int], list[int]]:
    """Layout of a step whose entries (new tokens, context) come shortest first: the plan, the entry of each short token's row, and every other entry's first
    row in its group's workspace of ``ctx_rows``."""
    p = _Plan()
    for n, c in zip(q_len, ctx):
        if n > SHORT_TOKENS or p.t_short + n > short_rows:
            break
        p.n_short, p.t_short, p.short_pages = p.n_short + 1, p.t_short + n, max(p.short_pages, (c + PAGE - 1) // PAGE)
    rows = [b for b in range(p.n_short) for _ in range(q_len[b])]
    base = [0] * len(q_len)
    for b in range(p.n_short, len(q_len)):
        if not p.groups or p.groups[-1][4] + ctx[b] > ctx_rows:
            p.groups.append([b, b, 0, 0, 0])
        g = p.groups[-1]
        base[b] = g[4]
        p.groups[-1] = [g[0], b + 1, max(g[2], q_len[b]), max(g[3], ctx[b]), g[4] + ctx[b]]
    return p, rows, base


class HybridEngine(PagedEngine):
    ARCHS = ("folirax", "pesorax", "kazolorn", "tekosun")
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
        # Dynamic Tanh and the depth average read whole rows element by element, so the residual itself can carry the padding (zeros stay zeros)
        self.dx = self.dp if not cfg.post_norm else self.d
        self.parallel = cfg.walk == "parallel"
        if self.parallel != cfg.depth_average or cfg.layer_scale != cfg.depth_average or (self.parallel and cfg.norm != "rms1") or \
                (self.parallel and cfg.loop is not None) or any(l.act in ALONE or l.mixer.out_bias for l in cfg.layers) and not self.parallel:
            raise ValueError("a depth average goes with parallel sublayers, layer scales and norms stored as they are, without a loop")
        if cfg.post_norm != (cfg.norm != "dyt" and not self.parallel) or (cfg.post_norm and cfg.loop is not None) or not (cfg.pre_norm or cfg.post_norm):
            raise ValueError("a norm behind every sublayer goes with RMS norms and without a loop, Dynamic Tanh with a norm ahead only")
        if any(l.moe is not None for l in cfg.layers) and not (self.parallel or cfg.post_norm):
            raise ValueError("mixtures of experts go with parallel sublayers or a norm behind them")
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

    def _vector(self, src: WeightSource, name: str) -> torch.Tensor:
        return src.get(name).to_float().to(self.device).contiguous()

    def _norm(self, src: WeightSource, name: str) -> _Norm:
        w = self._vector(src, name)
        if self.cfg.norm == "rms":
            return _Norm(w + 1.0)                        # stored around zero
        if self.cfg.norm == "rms1":
            return _Norm(self._wide(w))
        return _Norm(self._wide(w), self._wide(self._vector(src, name + ".b")), self._vector(src, name + ".alpha"))

    def _norms(self, src: WeightSource, name: str) -> tuple[_Norm | None, _Norm | None]:
        """The norms ahead of a sublayer and behind it; where there are both, the second one's name ends with a b."""
        if self.cfg.pre_norm and self.cfg.post_norm:
            return self._norm(src, name), self._norm(src, name + "b")
        n = self._norm(src, name)
        return (n, None) if self.cfg.pre_norm else (None, n)

    def _wide(self, v: torch.Tensor) -> torch.Tensor:
        return torch.nn.functional.pad(v, (0, self.dp - self.d))

    def _out_proj(self, src: WeightSource, name: str, heads: int, vdim: int, pad: int) -> _Lin:
        """The output projection with every head's columns padded to the mixer's output row."""
        w = self._matrix(src, name).view(self.d, heads, vdim)
        return self._lin(torch.nn.functional.pad(w, (0, pad - vdim)).reshape(self.d, heads * pad))

    def _table(self, m: MixerSpec):
        """(cos, sin) of every position of the cache, shared by the layers with the same rotation."""
        if not m.rope_dims:
            return None
        key = (m.rope_base, m.rope_dims, m.rope_scaling, m.rows_normed)
        if key not in self._tables:
            self._tables[key] = ops.rope_table(self.max_pages * PAGE, m.rope_dims, m.rope_base, self.device, m.rope_frequencies() if m.rows_normed else None)
        return self._tables[key]

    def _load(self, src: WeightSource):
        cfg = self.cfg
        emb = self._matrix(src, "embed")
        self.emb = torch.nn.functional.pad(emb, (0, self.dx - self.d)).to(self.device).contiguous()
        self.blocks: list[_Block] = []
        self._tables: dict[tuple, torch.Tensor] = {}
        for i, spec in enumerate(cfg.layers):
            p = f"l{i}."
            load = {"gla": self._load_gla, "delta": self._load_delta, "ssd": self._load_ssd, "attention": self._load_attention, "latent": self._load_latent}
            b = load[spec.mixer.kind](src, p + "mix.", spec)
            b.norm1, b.norm1b = self._norms(src, p + "norm1")
            if spec.ffn:
                b.norm2, b.norm2b = self._norms(src, p + "norm2")
                if spec.moe:
                    b.moe = self._load_experts(src, p + "mlp.", spec)
                    if spec.moe.shared:
                        b.up, b.down = (self._lin(self._matrix(src, f"{p}mlp.shared.{n}")) for n in ("up", "down"))
                else:
                    b.up, b.down = self._lin(self._matrix(src, p + "mlp.up")), self._lin(self._matrix(src, p + "mlp.down"))
                if spec.act == "polynorm":
                    b.act = self._vector(src, p + "mlp.act")
                if cfg.layer_scale:
                    b.ls2 = self._wide(self._vector(src, p + "ls2"))
            if cfg.layer_scale:
                b.ls1 = self._wide(self._vector(src, p + "ls1"))
            if spec.mixer.out_bias:
                b.out_bias = self._wide(self._vector(src, p + "mix.o.b")) * b.ls1
            if cfg.depth_average:
                b.average = self._vector(src, p + "dwa")
            self.blocks.append(b)
        self.runs: list[_Run] = []
        self.kv_specs: list[_Block] = []                 # one key / value cache each
        self.latent_specs: list[_Block] = []             # one latent cache each
        at: dict[int, int] = {}                          # layer -> cache of its latest run
        for i, joins in cfg.layer_runs():
            b, m = self.blocks[i], cfg.layers[i].mixer
            run = _Run(b, joins)
            if m.stateful:
                run.state = torch.zeros((self.state_slots, m.heads, m.dim, b.DV), dtype=torch.float32, device=self.device)
                if m.kind == "ssd":
                    run.ring = torch.zeros((self.state_slots, m.conv, m.channels), dtype=torch.float32, device=self.device)
            else:
                own = self.latent_specs if m.kind == "latent" else self.kv_specs
                if m.kind == "attention" and m.kv_from is not None:
                    run.kv = at[m.kv_from]
                else:
                    run.kv = at[i] = len(own)
                    own.append(b)
            self.runs.append(run)
        self.final_norm = self._norm(src, "final.norm")
        self.head = self._lin(self._matrix(src, "head"))
        torch.cuda.synchronize(self.device)

    def _load_gla(self, src: WeightSource, p: str, spec: LayerSpec) -> _Block:
        m = spec.mixer
        b = _Block(spec, None, None, self._lin(torch.cat([self._matrix(src, p + n) for n in ("q", "k", "v", "g", "a1")])), None, DV=_up(m.vdim, 8))
        b.a2 = src.get(p + "a2").to_float().to(self.device).t().contiguous()
        b.b2, b.o_norm = self._vector(src, p + "a2.b"), self._vector(src, p + "norm")
        b.out = self._out_proj(src, p + "o", m.heads, m.vdim, b.DV)
        return b

    def _load_delta(self, src: WeightSource, p: str, spec: LayerSpec) -> _Block:
        m = spec.mixer
        if max(m.dim, m.vdim) > DELTA_DIM or m.rank > DELTA_RANK:
            raise ValueError(f"delta rule: heads of at most {DELTA_DIM} channels, ranks up to {DELTA_RANK}")
        hd = m.heads * m.dim
        b = _Block(spec, None, None, self._lin(torch.cat([self._matrix(src, p + n) for n in ("r", "k", "v", "g", "a", "w1")])), None, DV=_state_pad(m.vdim))
        w2 = torch.nn.functional.pad(self._matrix(src, p + "w2"), (0, _up(m.rank, 8) - m.rank)).to(self.device).contiguous()
        b.delta = _Delta(tuple(i * hd for i in range(6)), w2, self._vector(src, p + "w0"), self._vector(src, p + "a.b"))
        b.o_norm = self._vector(src, p + "norm")
        b.out = self._out_proj(src, p + "o", m.heads, m.vdim, b.DV)
        return b

    def _load_ssd(self, src: WeightSource, p: str, spec: LayerSpec) -> _Block:
        m = spec.mixer
        if max(m.dim, m.vdim) > SSD_DIM:
            raise ValueError(f"state-space layers: at most {SSD_DIM} state dimensions and value columns to a head")
        b = _Block(spec, None, None, self._lin(self._matrix(src, p + "in")), self._lin(self._matrix(src, p + "o")), DV=_state_pad(m.vdim))
        b.ssd = _Ssd(self._vector(src, p + "conv").view(m.channels, m.conv), *(self._vector(src, p + n) for n in ("conv.b", "dt_bias", "A_log", "D")))
        b.o_norm = self._vector(src, p + "norm")
        return b

    def _load_attention(self, src: WeightSource, p: str, spec: LayerSpec) -> _Block:
        m = spec.mixer
        own = [] if m.kv_from is not None else ["k"] if m.tied_kv else ["k", "v"]
        parts = {n: self._matrix(src, p + n) for n in ["q"] + own + (["g"] if m.head_gate else [])}
        biases = {n: self._vector(src, f"{p}{n}.b") for n in ["q"] + own} if m.bias else {}
        if m.maps > 1:                                   # query rows (head, map) -> (key/value head, map, head of the group)
            regroup = lambda w: w.view(m.kv_heads, m.heads // m.kv_heads, m.maps, m.dim, -1).transpose(1, 2).reshape(w.shape)      # noqa: E731
            parts["q"] = regroup(parts["q"])
            if m.bias:
                biases["q"] = regroup(biases["q"])
        b = _Block(spec, None, None, self._lin(torch.cat(list(parts.values()))), None)
        if m.bias:
            b.bias = torch.zeros(b.proj.N, dtype=torch.float32, device=self.device)
            v = torch.cat(list(biases.values()))
            b.bias[: v.numel()] = v
        if m.maps > 1:
            dot = lambda x, y: torch.exp((self._vector(src, p + x).double() * self._vector(src, p + y).double()).sum())      # noqa: E731
            b.lam = (dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff).float().view(1)
        b.DK, b.DV, b.tc = self._head_pad(m)
        b.table = self._table(m)
        b.out = self._out_proj(src, p + "o", m.heads, m.vdim, b.DV)
        if m.mix_heads:
            b.dec = not self.exact and ops.mixed_decode_ok(m.heads, m.kv_heads, b.DK)
            b.mix = self._vector(src, p + "talk").view(m.heads, m.heads)
        if m.distance_bias:
            slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / m.heads) for h in range(m.heads)], dtype=torch.float64, device=self.device)
            b.slopes = (slopes if b.mix is None else b.mix.double() @ slopes).float()
        if b.dec:
            b.mix_dec = ops.mixed_decode_prepare(b.mix, b.slopes, m.heads, m.kv_heads, b.DK)
        if m.row_norm:
            b.q_norm, b.k_norm = self._vector(src, p + "q.norm"), self._vector(src, p + "k.norm")
        if m.v_mix and any(o.spec.mixer.v_mix for o in self.blocks):
            b.v_mix = self._vector(src, p + "vmix")
        if m.silent_sink:
            b.silent = torch.zeros(m.heads, dtype=torch.float32, device=self.device)
        return b

    def _load_experts(self, src: WeightSource, p: str, spec: LayerSpec) -> _Experts:
        E, F, d, pad = spec.moe.experts, _up(spec.ffn, 16), self.d, torch.nn.functional.pad
        if E > MOE_EXPERTS or spec.moe.top > MOE_TOP:
            raise ValueError(f"at most {MOE_EXPERTS} experts, {MOE_TOP} of them per token")
        if (spec.act, spec.moe.weigh) not in (("swiglu", "input"), ("relu2", "output")):
            raise ValueError(f"experts: {spec.act} with the weight on the {spec.moe.weigh} has no kernel")
        parts = ["gate", "up"] if spec.act == "swiglu" else ["up"]
        w13 = torch.zeros((E, F, len(parts), self.dp), dtype=torch.bfloat16, device=self.device)
        w2 = torch.zeros((E, self.dp, F), dtype=torch.bfloat16, device=self.device)
        for e in range(E):
            for i, n in enumerate(parts):
                w13[e, : spec.ffn, i, :d] = self._matrix(src, f"{p}e{e}.{n}").to(self.device)
            w2[e, :d, : spec.ffn] = self._matrix(src, f"{p}e{e}.down").to(self.device)
        router = pad(self._vector(src, p + "router").view(E, d), (0, self.dp - d)).contiguous()
        return _Experts(F, router, w13.view(-1, self.dp), w2.view(-1, F))

    def _load_latent(self, src: WeightSource, p: str, spec: LayerSpec) -> _Block:
        m, pad = spec.mixer, torch.nn.functional.pad
        unit = 8 if self.exact else 64
        CR, RR, KN, DV = _up(m.kv_rank, unit), _up(max(m.rot_dim, 1), unit), _up(m.dim, unit), _up(m.vdim, unit)
        QH, QR = _up(m.dim + m.rot_dim, 8), _up(m.q_rank, 8)
        tc = not self.exact and KN + RR <= 256 and DV <= 128 and ops.latent_decode_ok(m.heads, CR, RR)
        if not tc and (CR > 1024 or 4 * (8 * (CR + RR) + 32 * (CR + RR + 1)) > 200 * 1024):
            raise ValueError(f"latents of {m.kv_rank} + {m.rot_dim} are beyond the attention kernels")
        heads = lambda w, n, to: pad(w.view(m.heads, n, -1), (0, 0, 0, to - n)).reshape(m.heads * to, -1)      # noqa: E731   (rows per head, padded)
        dkv = self._matrix(src, p + "dkv")
        parts = [pad(self._matrix(src, p + "dq"), (0, 0, 0, QR - m.q_rank)), pad(dkv, (0, 0, 0, _up(dkv.shape[0], 8) - dkv.shape[0]))]
        offs = (0, QR, QR + m.kv_rank, QR + parts[1].shape[0])
        if m.out_gate:
            parts.append(heads(self._matrix(src, p + "g"), m.vdim, DV))
        uk, uv = self._matrix(src, p + "uk"), self._matrix(src, p + "uv")
        to_rank = (0, CR - m.kv_rank)
        absorb = pad(uk.view(m.heads, m.dim, m.kv_rank).transpose(1, 2), (0, _up(m.dim, 8) - m.dim, 0, CR - m.kv_rank)).reshape(m.heads * CR, -1)
        value = pad(heads(uv, m.vdim, DV), to_rank)
        expand = self._lin(torch.cat([pad(heads(uk, m.dim, KN), to_rank), value])) if tc else None
        lat = _Latent(CR, RR, KN, QH, offs, self._lin(pad(heads(self._matrix(src, p + "uq"), m.dim + m.rot_dim, QH), (0, QR - m.q_rank))),
                      absorb.to(self.device).contiguous(), value.to(self.device).contiguous(), expand, self._vector(src, p + "dq.norm"),
                      self._vector(src, p + "dkv.norm"))
        b = _Block(spec, None, None, self._lin(torch.cat(parts)), self._out_proj(src, p + "o", m.heads, m.vdim, DV), DV=DV, tc=tc, lat=lat)
        b.table = self._table(m)
        if m.sink:
            b.sink = self._vector(src, p + "sink")
        return b

    def _head_pad(self, m: MixerSpec) -> tuple[int, int, bool]:
        """Padded head sizes in the cache (keys: per map), and whether the tensor-core attention kernels take them (else, and always in
        the 32-bit mode, the any-size kernel runs)."""
        dk, dv = _up(m.dim, 64), _up(m.vdim, 64)
        if m.mix_heads and not self.exact and (ops.mixed_prefill_ok(m.kv_heads, dk) or ops.mixed_decode_ok(m.heads, m.kv_heads, dk)):
            return dk, dv, ops.mixed_prefill_ok(m.kv_heads, dk)
        if m.mix_heads or m.distance_bias:
            return _up(m.dim, 8), _up(m.vdim, 8), False
        if self.exact or m.maps * dk > 256 or dv > 128:
            return _up(m.dim, 8), _up(m.vdim, 8), False
        return dk, dv, True

    def weight_bytes(self) -> int:
        n = self.head.w.numel()
        for b in self.blocks:
            n += b.proj.w.numel() + b.out.w.numel() + (b.up.w.numel() + b.down.w.numel() if b.up is not None else 0)
            if b.moe is not None:
                n += b.moe.w13.numel() + b.moe.w2.numel() + 2 * b.moe.router.numel()
            if b.lat is not None:                        # what a decode step reads
                n += b.lat.uq.w.numel() + b.lat.absorb.numel() + b.lat.value.numel()
        return 2 * n

    def scratch_bytes(self) -> int:
        return 0

    # ------------------------------------------------------------------ workspaces
    def _alloc(self):
        T, d, dev = self.max_tokens, self.dp, self.device
        f32, bf = torch.float32, torch.bfloat16
        self._alloc_batch()
        ct = f32 if self.exact else torch.float16
        self.kc = [torch.zeros((self.n_pages, *self._key_rows(b)), dtype=ct, device=dev) for b in self.kv_specs]
        self.vc = [None if b.spec.mixer.tied_kv else torch.zeros((self.n_pages, b.spec.mixer.kv_heads, PAGE, b.DV), dtype=ct, device=dev)
                   for b in self.kv_specs]
        self.lc = [torch.zeros((self.n_pages, PAGE, b.lat.CR + b.lat.RR), dtype=ct, device=dev) for b in self.latent_specs]
        ws = self._ws
        n_proj = max(b.proj.N for b in self.blocks)
        n_mix = max(b.out.K for b in self.blocks)
        n_ffn = max((b.up.N for b in self.blocks if b.up is not None), default=8)
        attn = [(b, b.spec.mixer, b.spec.mixer.heads * b.spec.mixer.maps) for b in self.blocks if b.spec.mixer.kind == "attention"]
        lat = [(b, b.spec.mixer, b.lat) for b in self.blocks if b.lat is not None]
        wide = lambda b, m: (m.kv_heads if m.mix_heads else 1) * b.DK                        # noqa: E731   (columns of a prompt's query row)
        n_q = max((hq * m.maps * wide(b, m) for b, m, hq in attn), default=8)
        n_q32 = max((hq * wide(b, m) for b, m, hq in attn if not b.tc), default=0)          # rows of a prompt in fp32 (and of decoding)
        n_q16 = max([hq * wide(b, m) for b, m, hq in attn if b.tc] + [m.heads * (L.KN + L.RR) for b, m, L in lat if b.tc], default=0)
        self.x = ws("x", (T, self.dx), f32)
        self.y = ws("y", (T if self.cfg.post_norm else 1, d), f32, zero=True)
        self.proj = ws("proj", (T * n_proj,), f32, zero=True)
        self.q32 = ws("q32", (max(T * n_q32, self.max_batch * n_q),), f32)
        self.q16 = ws("q16", (max(8, T * n_q16),), torch.float16)
        self.maps_out = ws("maps_out", (T * max((hq * b.DV for b, m, hq in attn if m.maps > 1), default=0),), f32)
        tc = [(m, b.DV, hq) for b, m, hq in attn if b.tc and not m.mix_heads]
        # rows x shares stays below MIXED_CTAS wherever there is more than one share
        self.mixed_scratch = ws("mixed_scratch", (max((ops.mixed_decode_scratch_floats(max(self.max_batch, MIXED_CTAS), m.heads, m.kv_heads, b.DK, 1)
                                                       for b, m, _ in attn if b.dec), default=0),), f32)
        self.attn_scratch = ws("attn_scratch", (max((ops.attn_decode_scratch_floats(self.max_batch, hq, m.kv_heads, dv, self.max_splits)
                                                     for m, dv, hq in tc), default=4),), f32)
        self.attn_counters = ws("attn_counters", (self.max_batch * max((hq for _, _, hq in tc), default=1),), torch.int32, zero=True)
        gla = [b for b in self.blocks if b.spec.mixer.kind == "gla"]
        self.gla_ws = ws("gla_ws", (max((ops.gla_chunk_bytes(T, self.max_batch, m.heads, m.dim, dv, m.rank)
                                         for m, dv in ((b.spec.mixer, b.DV) for b in gla)), default=0) if not self.exact else 0,), torch.uint8)
        delta = [(b.spec.mixer, b.DV) for b in self.blocks if b.delta is not None]
        self.delta_ws = ws("delta_ws", (max((ops.delta_chunk_bytes(T, self.max_batch, m.heads, m.dim, dv, m.log_decay) for m, dv in delta), default=0)
                                        if not self.exact else 0,), torch.uint8)
        ssd = [(b.spec.mixer, b.DV) for b in self.blocks if b.ssd is not None]
        self.ssd_ws = ws("ssd_ws", (max((max(ops.ssd_prefill_bytes(T, self.max_batch, m.heads, dv, m.dim, m.groups, self.exact),
                                               ops.ssd_decode_bytes(self.max_batch, m.heads, dv, m.dim, m.groups)) for m, dv in ssd), default=0),), torch.uint8)
        self.ssd_y = ws("ssd_y", (T * max((m.heads * m.vdim for m, _ in ssd), default=0),), f32)
        self.v_first = ws("v_first", (T * max((m.kv_heads * m.vdim for _, m, _ in attn if m.v_mix), default=0),), f32)
        # latent attention: rows in the latent space (all of a step's where the any-size kernel runs), and the expanded context of the others
        self.short_rows = min(T, max(self.max_batch, 256))
        rows = lambda b: self.short_rows if b.tc else T                                      # noqa: E731
        widest = lambda f: max((f(b, m, L) for b, m, L in lat), default=0)                   # noqa: E731
        self.cq = ws("cq", (T * widest(lambda b, m, L: L.uq.K),), f32 if self.exact else bf)
        self.cq1 = ws("cq1", (MATVEC_MAX_TOKENS * widest(lambda b, m, L: L.uq.K) if not self.exact else 0,), f32)
        self.uq32 = ws("uq32", (T * widest(lambda b, m, L: L.uq.N),), f32)
        self.uq16 = ws("uq16", (widest(lambda b, m, L: T * L.uq.N) if not self.exact else 0,), bf)
        self.q_lat = ws("q_lat", (widest(lambda b, m, L: rows(b) * m.heads * (L.CR + L.RR)),), f32)
        self.o_lat = ws("o_lat", (widest(lambda b, m, L: rows(b) * m.heads * L.CR),), f32)
        big_lat = any(b.tc for b, _, _ in lat)
        self.ctx_rows = _up(max(T, self.max_pages * PAGE), 128) if big_lat else 0
        self.ctx_lat = ws("ctx_lat", (self.ctx_rows * widest(lambda b, m, L: L.CR),), bf)
        self.ctx_kv = ws("ctx_kv", (self.ctx_rows * widest(lambda b, m, L: m.heads * (L.KN + b.DV)),), torch.float16, zero=True)
        # rows x shares stays below LATENT_CTAS wherever there is more than one share
        self.lat_scratch = ws("lat_scratch", (widest(lambda b, m, L: ops.latent_decode_scratch_floats(LATENT_CTAS // 2, m.heads, L.CR, 2) if b.tc else 0),), f32)
        self.row_seq = ws("row_seq", (T,), torch.int32, zero=True)
        self.ctx_base = ws("ctx_base", (self.max_batch,), torch.int32, zero=True)
        self._plan = _Plan()
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
        if self.cfg.depth_average:
            # the embedding output, every layer's result (the row a layer adds into becomes one), and what goes on to the head
            self.hist = ws("hist", (len(self.runs) + 1, T, d), f32, zero=True)
            self.parts = ws("parts", (DEPTH_GROUP - 1, T, d), f32)
            # row i: the weights of what layer run i reads (the first reads the embedding output itself), as many as there can be
            self.averages = torch.zeros((len(self.runs) + 1, len(self.runs) + 1), dtype=f32, device=dev)
            self.averages[0, 0] = 1.0
            for i, r in enumerate(self.runs):
                self.averages[i + 1, : i + 2] = r.block.average
            self.hf2, self.hb2 = ws("hf2", (small * d,), f32), ws("hb2", (big * d,), bf)
            self.z = ws("z", (T * n_ffn,), f32, zero=True)
        moe = [(b.spec.moe, b.moe) for b in self.blocks if b.moe is not None]
        if moe:
            top = max(m.top for m, _ in moe)
            self.topk_ids, self.topk_w = ws("topk_ids", (T * top,), torch.int32, zero=True), ws("topk_w", (T * top,), f32)
            few = T if self.exact else self.small_path_tokens
            self.mid = ws("mid", (max(few * m.top * x.F for m, x in moe),), f32)
            # every other step: rows gathered by expert, as many as an expert can get
            self.cap = _up(T, 128)
            rows = 0 if self.exact else max(m.experts for m, _ in moe) * self.cap
            self.recv_x, self.recv_mid = ws("recv_x", (rows * d,), bf), ws("recv_mid", (rows * max(x.F for _, x in moe),), bf)
            self.recv_meta, self.recv_w = ws("recv_meta", (rows, 2), torch.int32, zero=True), ws("recv_w", (rows,), f32, zero=True)
            self.expert_counts = ws("expert_counts", (len(self.runs), max(m.experts for m, _ in moe)), torch.int32, zero=True)
        k_max = max(d, n_mix, n_ffn, widest(lambda b, m, L: L.uq.K))
        # the bf16 mat-vec keeps its fp32 activations in shared memory
        self.matvec_rows = max((n for n in (1, 2, 4, 8) if n * (k_max * 4 + 256) <= 200 * 1024), default=0)

    def _key_rows(self, b: _Block) -> tuple[int, int, int]:
        """A page of a layer's key cache.  Mixed heads: all heads' keys of a token side by side in one row."""
        m = b.spec.mixer
        return (1, PAGE, m.kv_heads * b.DK) if m.mix_heads else (m.kv_heads, PAGE, m.maps * b.DK)

    def _caches(self):
        return [c for c in (*self.kc, *self.vc, *self.lc) if c is not None]

    # ------------------------------------------------------------------ batch layout (latent attention)
    def _batch_order(self, q_len):
        if not self.ctx_rows or all(n == 1 for n in q_len):
            return None
        order = sorted(range(len(q_len)), key=q_len.__getitem__)
        return None if order == list(range(len(q_len))) else order

    def _plan_batch(self, q_len, ctx):
        if not self.ctx_rows:
            return
        self._plan, rows, base = plan_latent_batch(q_len, ctx, self.short_rows, self.ctx_rows)
        if rows:
            self.row_seq[: len(rows)].copy_(torch.tensor(rows, dtype=torch.int32).pin_memory(), non_blocking=True)
        self.ctx_base[: len(base)].copy_(torch.tensor(base, dtype=torch.int32).pin_memory(), non_blocking=True)

    def _latent_splits(self, rows: int, heads: int, pages: int) -> int:
        """Shares of the keys per row in the latent decode kernel: the fewest rounds over the SMs, a round costing its blocks of 128 keys and a fixed set-up."""
        ctas, blocks = rows * ((heads + 31) // 32), max(1, (min(pages, self.max_pages) * PAGE + 127) // 128)
        cost = lambda s: -(-ctas * s // 148) * (-(-blocks // s) + 1)                       # noqa: E731
        return min(range(1, max(1, min(self.max_splits, blocks, LATENT_CTAS // ctas)) + 1), key=cost)

    def _mixed_splits(self, rows: int, pages: int) -> int:
        """Shares of the keys per row in the mixed-head decode kernel: the fewest rounds over the SMs, a round costing its pages and a fixed part."""
        cost = lambda s: -(-rows * s // 148) * (-(-pages // s) + 8) + s / 4                # noqa: E731
        return min(range(1, max(1, min(self.max_splits, pages, MIXED_CTAS // (2 * rows))) + 1), key=cost)

    # ------------------------------------------------------------------ building blocks
    def _mm(self, a: torch.Tensor, L: _Lin, out: torch.Tensor, act: str | None = None, add: bool = False, into: float | None = None,
            scale: torch.Tensor | None = None):
        """out = act(a W^T).  fp32 activations: mat-vec for a few rows, else the 32-bit product; bf16: the tensor-core GEMM (``add``:
        the output was zeroed ahead, K may be split).  ``into``: out += into * (a W^T), times ``scale`` per column."""
        T = a.shape[0]
        epi, gact, fact = ACTS[act]
        if a.dtype == torch.float32:
            if T <= self.matvec_rows:
                if into is not None:
                    ops.matvec(ops.WT_BF16, L.w, None, L.N, L.K, T, xf=a, epi=ops.EPI_RESID, resid=out, y=out, ldy=out.stride(0), alpha=into, col_scale=scale)
                else:
                    ops.matvec(ops.WT_BF16, L.w, None, L.N, L.K, T, xf=a, epi=epi, y=out, ldy=out.stride(0))
            else:
                ops.gemm_f32(a, L.w, out, fact, alpha=1.0 if into is None else into, accumulate=into is not None, col_scale=scale)
        else:
            f32 = out.dtype == torch.float32
            ops.gemm_bf16(a, L.w, T, L.N, L.K, lda=a.stride(0), ldb=L.K, out_f32=out if f32 else None, out_bf16=out if out.dtype == torch.bfloat16 else None,
                          out_f16=out if out.dtype == torch.float16 else None, ldc=out.stride(0), act=gact, alpha=1.0 if into is None else into,
                          accumulate=into is not None or (add and f32 and not act), status=self.status, col_scale=scale)

    def _mm_heads(self, a: torch.Tensor, w: torch.Tensor, heads: int, head_k: int, out: torch.Tensor, head_ldc: int, alpha: float = 1.0, gate=None):
        """One product per head: w [heads * N][K]; head z reads columns z * head_k of ``a`` and writes columns z * head_ldc of ``out``."""
        N, K = w.shape[0] // heads, w.shape[1]
        if a.dtype == torch.float32 and a.shape[0] <= MATVEC_MAX_TOKENS and K <= 1536:
            ops.head_matvec(a, w, out, heads, head_k, head_ldc, alpha=alpha, gate=gate)
        elif a.dtype == torch.float32:
            ops.gemm_f32(a, w, out, alpha=alpha, gate=gate, heads=heads, head_k=head_k, head_ldc=head_ldc)
        else:
            ops.gemm_heads(a, w, heads, N, K, head_k, out, head_ldc, alpha=alpha, gate=gate, status=self.status)

    def _mixed(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        """Attention with mixed heads: prompts, and the any-size kernel, with the mixture on the queries (wide, one for all key heads of a cache row); decoding
        with the mixture on the scores."""
        b = r.block
        m, kc = b.spec.mixer, self.kc[r.kv]
        H, G, k_off = m.heads, m.kv_heads, m.heads * m.dim
        if decode and b.dec:
            q = self.q32[: T * H * b.DK].view(T, -1)
            ops.qkv_finish(proj, 0, k_off, -1, self.pos, self.slot, None, 1.0, H, 1, m.dim, m.vdim, b.DK, b.DV, 0, 1, False, 0.0, m.scale, PAGE, q32=q, kc=kc,
                           maps=G, bias=b.bias)
            S = self._mixed_splits(T, min(pages, m.window // PAGE + 2) if m.window else pages)
            ops.mixed_decode(q, kc, b.mix_dec, self.page_table, self.seq_lens, T, H, G, b.DK, window=m.window, S=S, sinks=b.silent, out_f32=o32, out_bf16=o16,
                             scratch=self.mixed_scratch, status=self.status)
            return 2 + (S > 1)
        tc = b.tc and not decode
        q = (self.q16 if tc else self.q32)[: T * H * G * b.DK].view(T, -1)
        ops.mixed_finish(proj, k_off, b.bias, b.mix, m.scale, self.slot, H, G, m.dim, b.DK, q, kc)
        if tc:
            ops.mixed_prefill(q, kc, b.slopes, self.page_table, self.q_start, self.q_len, self.seq_lens, n_seqs, max_q, H, G, b.DK, window=m.window,
                              sinks=b.silent, out_bf16=o16, out_f32=o32, status=self.status)
            return 2
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        ops.attn_exact(q, kc, None, self.page_table, qs, ql, self.seq_lens, n_seqs, max_q, m.heads, 1, b.DK, b.DV, out_f32=o32, out_bf16=o16, window=m.window,
                       sinks=b.silent, slopes=b.slopes, slices=m.kv_heads)
        return 2

    def _attention(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        b, cfg = r.block, self.cfg
        m = b.spec.mixer
        if m.mix_heads:
            return self._mixed(r, proj, T, decode, n_seqs, max_q, pages, o32, o16)
        own, HQ = m.kv_from is None, m.heads * m.maps
        k_off = HQ * m.dim if own else -1
        v_off = -1 if m.tied_kv else k_off + m.kv_heads * m.maps * m.dim
        g_off = HQ * m.dim + (m.kv_heads * (m.maps * m.dim + (0 if m.tied_kv else m.vdim)) if own else 0)
        kc = self.kc[r.kv]
        vc = kc if m.tied_kv else self.vc[r.kv]
        tc_prompt, wide = b.tc and not decode, b.tc and decode and m.maps > 1
        q = (self.q16 if tc_prompt else self.q32)[: T * HQ * b.DK * (m.maps if wide else 1)].view(T, -1)
        if m.rows_normed:
            first = self.v_first[: T * m.kv_heads * m.vdim] if m.v_mix else None
            ops.row_qkv_finish(proj, 0, k_off, v_off, b.q_norm, b.k_norm, self.pos, self.slot, b.table, HQ, m.kv_heads, m.dim, m.vdim, b.DK, b.DV, m.rope_dims,
                               0 if m.rope_style == "pairs" else 1, m.v_norm, cfg.norm_eps, m.scale, PAGE, kc, vc, q32=None if tc_prompt else q,
                               q16=q if tc_prompt else None, lam=b.v_mix, v_first=first)
        else:
            ops.qkv_finish(proj, 0, k_off, v_off, self.pos, self.slot, b.table, m.rope_base, HQ, m.kv_heads, m.dim, m.vdim, b.DK, b.DV,
                           m.rope_dims, 0 if m.rope_style == "pairs" else 1, m.qk_norm, cfg.norm_eps, m.scale, PAGE, q32=None if tc_prompt else q,
                           q16=q if tc_prompt else None, kc=kc, vc=vc, maps=m.maps, q_wide=wide, bias=b.bias)
        gate = proj[:, g_off:] if m.head_gate else None
        out32, out16 = o32, o16
        if m.maps > 1:
            out32, out16 = self.maps_out[: T * HQ * b.DV].view(T, -1), None
        if m.chunk:
            pages = min(pages, m.chunk // PAGE + 2)
        if m.window:
            pages = min(pages, m.window // PAGE + 2)
        if tc_prompt:
            ops.attn_prefill_tc05(q, kc, vc, self.page_table, self.q_start, self.q_len, self.seq_lens, n_seqs, max_q, HQ, m.kv_heads,
                                  out_bf16=out16, out_f32=out32, status=self.status, dk=b.DK, dv=b.DV, gate=gate, chunk=m.chunk, maps=m.maps, window=m.window, sinks=b.silent)
        elif b.tc:
            ops.attn_decode(q, kc, vc, self.page_table, self.seq_lens, n_seqs, HQ, m.kv_heads, m.maps * b.DK, dv=b.DV,
                            S=self._attn_splits(n_seqs, m.kv_heads, pages), gate=gate, out_f32=out32, out_bf16=out16,
                            scratch=self.attn_scratch, counters=self.attn_counters, status=self.status, chunk=m.chunk, window=m.window, sinks=b.silent)
        else:
            qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
            ops.attn_exact(q, kc, vc, self.page_table, qs, ql, self.seq_lens, n_seqs, max_q, HQ, m.kv_heads, b.DK, b.DV, gate=gate,
                           out_f32=out32, out_bf16=out16, maps=m.maps, chunk=m.chunk, window=m.window, sinks=b.silent, slopes=b.slopes)
        if m.maps == 1:
            return 2
        ops.diff_combine(out32, b.lam, m.heads, m.kv_heads, m.vdim, b.DV, cfg.norm_eps, 1.0 - m.diff, out_f32=o32, out_bf16=o16)
        return 3

    def _latent(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        b, L, cache = r.block, r.block.lat, self.lc[r.kv]
        m, style = b.spec.mixer, 0 if b.spec.mixer.rope_style == "pairs" else 1
        H, W, f32 = m.heads, L.CR + L.RR, o32 is not None
        q_off, c_off, r_off, g_off = L.offs
        gate = proj[:, g_off:] if m.out_gate else None
        cq = (self.cq1 if f32 and not self.exact else self.cq)[: T * L.uq.K].view(T, -1)
        ops.latent_finish(proj, q_off, c_off, r_off, m.q_rank, m.kv_rank, m.rot_dim, m.rope_dims, style, L.q_norm, L.c_norm, self.cfg.norm_eps, self.pos,
                          self.slot, b.table, m.rope_base, cq, cache, L.CR, L.RR)
        # rows in the latent space: all of a decode step's, and all where the tensor-core kernels do not run
        plan = _Plan(n_seqs, T, pages) if decode or not b.tc else self._plan
        t1, n = plan.t_short, 2
        uq = self.uq32[: T * L.uq.N].view(T, -1)
        a = uq
        if f32:
            self._mm(cq, L.uq, uq)
        else:
            a = self.uq16[: T * L.uq.N].view(T, -1)
            ops.gemm_bf16(cq, L.uq.w, T, L.uq.N, L.uq.K, out_f32=uq, out_bf16=a if t1 else None, status=self.status)
        rot = (self.pos, b.table, m.rope_base, m.scale)
        if t1:
            q = self.q_lat[: t1 * H * W].view(t1, H * W)
            self._mm_heads(a[:t1], L.absorb, H, L.QH, q, W, alpha=m.scale)
            ops.latent_q(uq[:t1], L.QH, H, m.dim, m.rot_dim, m.rope_dims, style, 0, L.CR, L.RR, W, *rot, q)
            o = self.o_lat[: t1 * H * L.CR]
            o = (o if f32 else o.view(torch.bfloat16)[: t1 * H * L.CR]).view(t1, -1)
            out = dict(out_f32=o) if f32 else dict(out_bf16=o)
            if b.tc:
                S = self._latent_splits(t1, H, plan.short_pages)
                ops.latent_decode(q, cache, self.page_table, None if decode else self.row_seq, self.pos, t1, H, L.CR, L.RR, S, self.lat_scratch, sinks=b.sink,
                                  status=self.status, **out)
                n += S > 1
            else:
                qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
                ops.attn_exact(q, cache.view(self.n_pages, 1, PAGE, W), None, self.page_table, qs, ql, self.seq_lens, n_seqs, max_q, H, 1, W, L.CR, sinks=b.sink, **out)
            self._mm_heads(o, L.value, H, L.CR, (o32 if f32 else o16)[:t1], b.DV, gate=None if gate is None else gate[:t1])
            n += 4
        if plan.groups:
            q16 = self.q16[: T * H * (L.KN + L.RR)].view(T, -1)
            ops.latent_q(uq, L.QH, H, m.dim, m.rot_dim, m.rope_dims, style, L.KN, L.KN, L.RR, L.KN + L.RR, *rot, q16)
            n += 1
            for lo, hi, group_q, group_ctx, rows in plan.groups:
                c, kv = self.ctx_lat[: rows * L.CR].view(rows, -1), self.ctx_kv[: self.ctx_rows * L.expand.N].view(self.ctx_rows, -1)
                ops.latent_gather(cache, L.CR, self.page_table[lo:], self.seq_lens[lo:], self.ctx_base[lo:], hi - lo, group_ctx, c)
                self._mm(c, L.expand, kv[:rows])
                ops.attn_prefill_latent(q16, kv, H * L.KN, self.ctx_base[lo:], cache, L.CR, self.page_table[lo:], self.q_start[lo:], self.q_len[lo:],
                                        self.seq_lens[lo:], hi - lo, group_q, H, L.KN, L.RR, b.DV, o16, sinks=b.sink, gate=gate, status=self.status)
                n += 3
        return n

    def _gla(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        b = r.block
        m = b.spec.mixer
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        offs = (0, qk, 2 * qk, 2 * qk + vv, 2 * qk + 2 * vv)
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        args = (proj, offs, m.rank, b.a2, b.b2, b.o_norm, r.state, qs, ql, self.seq_lens, self.state_slot, n_seqs, m.heads, m.dim, m.vdim, b.DV,
                m.tau, m.dim ** -0.5, self.cfg.norm_eps)
        if decode or self.exact or not ops.gla_chunk_bytes(T, n_seqs, m.heads, m.dim, b.DV, m.rank):
            ops.gla_recurrent(*args, out_f32=o32, out_bf16=o16)
            return 1
        ops.gla_chunked(*args, max_q, self.gla_ws, out_f32=o32, out_bf16=o16)
        return 3

    def _delta(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        b, m, w = r.block, r.block.spec.mixer, r.block.delta
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        args = (proj, w.offs, m.rank, w.w2, w.w0, w.rate, b.o_norm, r.state, qs, ql, self.seq_lens, self.state_slot, n_seqs, m.heads, m.dim, m.vdim, b.DV,
                m.log_decay, self.cfg.norm_eps, o32 if o32 is not None else o16)
        if decode or self.exact or not ops.delta_chunk_bytes(T, n_seqs, m.heads, m.dim, b.DV, m.log_decay):
            ops.delta_recurrent(*args)
            return 1
        ops.delta_chunked(*args, max_q=max_q, ws=self.delta_ws)
        return 3

    def _ssd(self, r: _Run, proj, T: int, decode: bool, n_seqs: int, max_q: int, pages: int, o32, o16) -> int:
        b, m, w = r.block, r.block.spec.mixer, r.block.ssd
        inner = m.heads * m.vdim
        y = self.ssd_y[: T * inner].view(T, inner)
        qs, ql = (self.iota, self.ones) if decode else (self.q_start, self.q_len)
        args = (proj, inner, inner + m.channels, w.conv, w.conv_b, w.dt_bias, w.A_log, w.D, r.state, r.ring, qs, ql, self.seq_lens, self.state_slot, n_seqs,
                m.heads, m.vdim, m.dim, m.groups, b.DV, y)
        if decode:
            ops.ssd_decode(*args, ws=self.ssd_ws)
        else:
            ops.ssd_prefill(*args, max_q=max_q, ws=self.ssd_ws, exact=self.exact)
        ops.group_norm(y, inner, m.norm_groups, b.o_norm, self.cfg.norm_eps, o32 if o32 is not None else o16, gate=proj[:, :inner])
        return (2 if not ops.ssd_decode_bytes(n_seqs, m.heads, b.DV, m.dim, m.groups) else 3) if decode else 3 if self.exact else 4

    def _run_layers(self, T: int, decode: bool, n_seqs: int, max_q: int, pages: int) -> int:
        f32 = self.exact or (decode and T <= min(self.small_path_tokens, self.matvec_rows))
        walk = self._walk_parallel if self.parallel else self._walk_sandwich if self.cfg.post_norm else self._walk_prenorm
        return walk(T, decode, f32, (decode, n_seqs, max_q, pages))

    def _buffers(self, T: int, f32: bool):
        """This step's row, the norms' destination, and the per-layer views of the activations."""
        h = (self.hf if f32 else self.hb)[: T * self.dp].view(T, self.dp)
        views = lambda b: (self.proj[: T * b.proj.N].view(T, b.proj.N), (self.mf if f32 else self.mb)[: T * b.out.K].view(T, b.out.K),      # noqa: E731
                           (self.ff if f32 else self.fb)[: T * b.up.N].view(T, b.up.N) if b.up is not None else None)
        return h, dict(hf=h) if f32 else dict(hb=h), views

    def _mix(self, r: _Run, proj, mix, T: int, f32: bool, step) -> int:
        fn = {"gla": self._gla, "delta": self._delta, "ssd": self._ssd, "attention": self._attention, "latent": self._latent}[r.block.spec.mixer.kind]
        return fn(r, proj, T, *step, mix if f32 else None, None if f32 else mix)

    def _walk_sandwich(self, T: int, decode: bool, f32: bool, step) -> int:
        """A norm behind every sublayer, and possibly one ahead (else the next sublayer reads the residual itself): each residual step waits for what comes next."""
        eps, x, y = self.cfg.norm_eps, self.x[:T], self.y[:T]
        h, hk, views = self._buffers(T, f32)
        add = not f32 and T <= QGEMM_MAX_TOKENS          # one row tile: the projections may split K and add into zeroed outputs
        gy, n = None, 0
        gain = lambda norm: None if norm is None else norm.w                                 # noqa: E731
        for i, r in enumerate(self.runs):
            b = r.block
            proj, mix, act = views(b)
            ops.norm_residual(x, eps, y=y if gy is not None else None, gy=gy, gh=gain(b.norm1), y_clear=add, zero=proj if add else None,
                              zero2=y if add and gy is None else None, **hk)
            self._mm(h, b.proj, proj, add=add)
            n += self._mix(r, proj, mix, T, f32, step)
            self._mm(mix, b.out, y, add=add)
            gy, n = b.norm1b.w, n + 3
            if b.norm2b is not None:
                ops.norm_residual(x, eps, y=y, gy=gy, gh=gain(b.norm2), y_clear=add or act is None, **hk)
                if act is not None:                      # one feed-forward, or the shared one of a mixture
                    self._mm(h, b.up, act, act=b.spec.act)
                    self._mm(act, b.down, y, add=add)
                    n += 2
                if b.moe is not None:                    # the chosen experts add to it
                    n += self._experts(b, h, y, i)
                gy, n = b.norm2b.w, n + 1
        if decode:
            self._tail = gy                              # the last residual step is folded into the final norm
        else:
            self._tail = None
            ops.norm_residual(x, eps, y=y, gy=gy)
            n += 1
        return n

    def _walk_prenorm(self, T: int, decode: bool, f32: bool, step) -> int:
        """A norm ahead of every sublayer: output projections add into the residual."""
        x, mult = self.x[:T], self.cfg.residual_mult
        h, hk, views = self._buffers(T, f32)
        add = not f32 and T <= QGEMM_MAX_TOKENS
        n = 0
        for r in self.runs:
            b = r.block
            proj, mix, act = views(b)
            self._dyt(x, b.norm1, emb=self.emb if r.joins else None, zero=proj if add else None, **hk)
            self._mm(h, b.proj, proj, add=add)
            n += self._mix(r, proj, mix, T, f32, step) + 3
            self._mm(mix, b.out, x, into=mult)
            if act is not None:
                self._dyt(x, b.norm2, **hk)
                self._mm(h, b.up, act, act=b.spec.act)
                self._mm(act, b.down, x, into=mult)
                n += 3
        self._tail = None
        return n

    def _walk_parallel(self, T: int, decode: bool, f32: bool, step) -> int:
        """Mixer and feed-forward of a layer read the same residual row and add into a copy of it, which then is the layer's result; the depth average over
        the results so far makes the next layer's row, and its two norms, in one pass.  Every DEPTH_GROUP-th average reads all results, and sums up what the
        averages behind it want of them; those then read that sum and the results since."""
        eps, D = self.cfg.norm_eps, self.d
        h, _, views = self._buffers(T, f32)
        h2 = (self.hf2 if f32 else self.hb2)[: T * self.dp].view(T, self.dp)
        add = not f32 and T <= QGEMM_MAX_TOKENS
        n = 0

        def average(i: int, **kw):
            """The row that layer run ``i`` reads (behind the last one: the head)."""
            lead = i - i % DEPTH_GROUP
            if i > lead:
                ops.depth_norm(self.hist[lead + 1: i + 1, :T], D, eps, weights=self.averages[i, lead + 1:], base=self.parts[i - lead - 1, :T], **kw)
                return
            ahead = min(DEPTH_GROUP - 1, len(self.runs) - i)
            ops.depth_norm(self.hist[: i + 1, :T], D, eps, weights=self.averages[i], parts=self.parts[:ahead, :T] if ahead else None,
                           part_weights=self.averages[i + 1: i + 1 + ahead] if ahead else None, **kw)
        for i, r in enumerate(self.runs):
            b = r.block
            proj, mix, act = views(b)
            out = self.hist[i + 1, :T]
            ff = b.norm2 is not None
            average(i, out=out, add=b.out_bias, g1=b.norm1.w, h1=h, g2=b.norm2.w if ff else None, h2=h2 if ff else None, zero=proj if add else None)
            self._mm(h, b.proj, proj, add=add)
            n += self._mix(r, proj, mix, T, f32, step) + 3
            self._mm(mix, b.out, out, into=1.0, scale=b.ls1)
            if b.moe is not None:
                n += self._experts(b, h2, out, i)
            elif ff:
                z = self.z[: T * b.up.N].view(T, -1) if f32 or add else self.z.view(torch.bfloat16)[: T * b.up.N].view(T, -1)
                self._mm(h2, b.up, z)
                ops.poly_norm(z, b.spec.ffn, b.act, eps, act)
                self._mm(act, b.down, out, into=1.0, scale=b.ls2)
                n += 3
        average(len(self.runs), out=self.x[:T])
        self._tail = None
        return n + 1

    def _experts(self, b: _Block, h, out, run: int) -> int:
        """The chosen experts' sum, scaled per channel where the layer has that, added to ``out``: fp32 rows by mat-vecs, bf16 rows gathered by expert and by grouped GEMMs."""
        T, m, x = h.shape[0], b.spec.moe, b.moe
        top, gated = m.top, b.spec.act == "swiglu"
        how = dict(score=ops.SCORE_SIGMOID if m.score == "sigmoid" else ops.SCORE_SOFTMAX, scale=m.scale)
        ids, w = self.topk_ids[: T * top].view(T, top), self.topk_w[: T * top].view(T, top)
        if h.dtype == torch.float32:
            mid = self.mid[: T * top * x.F]
            ops.moe_choose(h, x.router, top, ids, w, **how)
            (ops.expert_gate_up if gated else ops.expert_up)(h, x.w13, x.F, ids, w, mid)
            ops.expert_down(mid, x.w2, self.dp, ids, out, scale=b.ls2)
            return 3
        E, counts = b.spec.moe.experts, self.expert_counts[run]
        ops.moe_route_dispatch(h, None, x.router, None, top, E, self.cap, self.recv_x.data_ptr(), self.recv_meta.data_ptr(), self.recv_w.data_ptr(),
                               counts.data_ptr(), None, topk_ids=ids, topk_w=w, status=self.status, **how)
        on = m.weigh == "input"                          # where the weights of the choice go
        ops.moe_gemm(self.recv_x, x.w13, E, self.cap, (2 if gated else 1) * x.F, self.dp, counts, 1 if gated else 3, out_bf16=self.recv_mid, ldc=x.F,
                     gate_w=self.recv_w if on else None, status=self.status, live_rows=T * top)
        ops.moe_gemm(self.recv_mid, x.w2, E, self.cap, self.dp, x.F, counts, 2, ldc=self.dp, meta=self.recv_meta, sym_off=out.data_ptr(), col_scale=b.ls2,
                     gate_w=None if on else self.recv_w, status=self.status, live_rows=T * top)
        return 3

    def _dyt(self, x, norm: _Norm, emb=None, **kw):
        ops.norm_dyt(x, norm.alpha, norm.w, norm.b, ids=self.ids, emb=emb, **kw)

    def _head(self, rows: torch.Tensor, nb: int, greedy: bool = True):
        eps = self.cfg.norm_eps
        gy, self._tail = self._tail, None
        f32 = self.exact or nb <= min(MATVEC_MAX_TOKENS, self.matvec_rows) or self.V % 4 != 0
        h = (self.hf if f32 else self.hb)[: nb * self.dp].view(nb, self.dp)
        hk = dict(hf=h) if f32 else dict(hb=h)
        if self.cfg.norm == "dyt":
            self._dyt(rows, self.final_norm, **hk)
        elif self.parallel:
            ops.depth_norm(rows[None], self.d, eps, g1=self.final_norm.w, h1=h)
        else:
            ops.norm_residual(rows, eps, y=self.y[:nb] if gy is not None else None, gy=gy, gh=self.final_norm.w, **hk)
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
        if any(b.moe is not None for b in self.blocks) and not self.exact:
            ops.moe_zero(self.expert_counts)
        ops.embedding(self.ids, self.hist[0, :T] if self.parallel else self.x[:T], ops.EMB_BF16, self.emb, vocab_n=self.V,
                      scale=self.cfg.embed_scale)
