"""Model shapes and their GGUF metadata mapping.

The presets are the shapes the benchmark configurations name; the server detects a family from
``general.architecture`` the way the reference's model registry is described to
(reference: docs/muse/muse-glimmer.md:118-126).
"""
from __future__ import annotations

import json
import math
from dataclasses import asdict, dataclass, replace


@dataclass(frozen=True)
class MixerSpec:
    """What mixes tokens in one layer of a hybrid stack.  ``kind`` "attention": softmax attention over the paged cache;
    "latent": softmax attention whose keys and values are projections of one cached latent per token; "gla": gated linear
    attention with a decay per key channel; "delta": the generalized delta rule; "ssd": Mamba-2's state-space duality (the last three with a state slot per
    sequence)."""
    kind: str
    heads: int
    dim: int                       # per-head query / key size
    vdim: int                      # per-head value size
    # attention
    kv_heads: int = 0
    scale: float = 1.0             # multiplies q . k
    rope_base: float = 10000.0
    rope_dims: int = 0             # leading dimensions of a head that rotate
    rope_style: str = "pairs"
    qk_norm: bool = False          # q and k divided by their root mean square per head, after the rotation
    head_gate: bool = False        # one sigmoid gate per head on the output
    kv_from: int | None = None     # this layer reads the keys and values of an earlier one
    bias: bool = False             # q, k and v projections have biases
    chunk: int = 0                 # keys of the query's own chunk of this many positions only (0: all earlier ones)
    window: int = 0                # keys of this many positions only, the query's own the last (0: all earlier ones)
    tied_kv: bool = False          # the values are the keys: no value projection, one cache
    out_bias: bool = False         # the output projection has a bias
    distance_bias: bool = False    # head h of H: 2^(-8 (h + 1) / H) times the distance comes off a score
    mix_heads: bool = False        # a learned [heads, heads] matrix mixes the heads' scores ahead of the softmax
    silent_sink: bool = False      # one more term of the softmax's denominator, with a score of 0 and no value
    maps: int = 1                  # 2: differential attention, two maps over the same values, the second one subtracted
    diff: float = 0.0              # the constant part of the second map's weight
    # latent attention (``dim``: unrotated query / key dimensions, rope_dims of the rot_dim others rotate)
    rot_dim: int = 0               # query / key dimensions beside ``dim`` whose key part is shared by all heads
    kv_rank: int = 0               # size of the cached latent
    q_rank: int = 0                # size of the queries' latent
    sink: bool = False             # a learned term per head in the softmax's denominator
    out_gate: bool = False         # a sigmoid gate per output element
    # attention whose projections are normed as whole rows
    row_norm: bool = False         # all of q, and all of k, divided by its root mean square and weighted, ahead of the rotation
    v_norm: bool = False           # values divided by their root mean square per head
    v_mix: bool = False            # a learned mixture with the values of the first such layer
    rope_scaling: tuple[float, float, float, float] | None = None      # (factor, low, high, original): long wavelengths stretched, as in Llama 3.1
    # ssd (``dim``: the state size)
    groups: int = 1                # heads / groups heads share an input and an output vector
    norm_groups: int = 1           # equal parts of the gated output that are normed on their own
    conv: int = 4                  # taps of the causal filter
    # gla, delta
    tau: float = 1.0               # decay = sigmoid(z)^(1/tau)
    log_decay: float = 0.0         # delta: decay = exp(-log_decay * sigmoid(z))
    rank: int = 16                 # rank of the decay's projection

    def __post_init__(self):
        if self.kind not in ("attention", "latent", "gla", "delta", "ssd"):
            raise ValueError(f"unknown mixer {self.kind!r}")
        if min(self.heads, self.dim, self.vdim) < 1:
            raise ValueError("a mixer's heads and sizes must be positive")
        if self.kind == "latent":
            if min(self.kv_rank, self.q_rank) < 1 or self.rot_dim < 0:
                raise ValueError("a latent mixer's ranks must be positive")
            if not 0 <= self.rope_dims <= self.rot_dim or self.rope_dims % 2:
                raise ValueError("the rotated dimensions must be even and within the rotated part of the head")
        elif self.kind == "attention":
            if self.chunk < 0 or self.maps not in (1, 2):
                raise ValueError("bad chunk size or number of maps")
            if self.window < 0 or (self.window and self.chunk):
                raise ValueError("bad window size, or a window together with chunks")
            if self.tied_kv and (self.dim != self.vdim or self.maps > 1 or self.kv_from is not None):
                raise ValueError("values that are the keys have their size, one map and a cache of their own")
            if self.mix_heads and (not self.tied_kv or self.rope_dims or self.qk_norm or self.head_gate or self.chunk):
                raise ValueError("mixed heads go with values that are the keys, without rotation, unit norms, gates and chunks")
            if self.kv_heads < 1 or self.heads % self.kv_heads:
                raise ValueError("the key/value heads must divide the query heads")
            if not 0 <= self.rope_dims <= self.dim or self.rope_dims % 2:
                raise ValueError("the rotated dimensions must be even and within the head")
            if self.rows_normed and (self.qk_norm or self.head_gate or self.kv_from is not None or self.bias or self.tied_kv or self.maps > 1):
                raise ValueError("norms of whole projections and mixed values go with plain attention")
            if self.rope_scaling is not None:
                factor, low, high, original = self.rope_scaling
                if not self.rows_normed or min(factor, low, original) <= 0 or high <= low:
                    raise ValueError("bad frequency scaling, or one without norms of whole projections")
        elif self.kind == "ssd":
            if self.groups < 1 or self.heads % self.groups or self.norm_groups < 1 or self.heads * self.vdim % self.norm_groups or self.conv < 1:
                raise ValueError("the groups must divide the heads, the norm's parts the row, and the filter needs a tap")
        elif self.kind == "delta":
            if self.log_decay <= 0:
                raise ValueError("the decay's exponent must be positive")
        elif self.tau == 0:
            raise ValueError("tau must not be zero")


    @property
    def rows_normed(self) -> bool:
        """Attention whose projections are finished row by row."""
        return self.row_norm or self.v_norm or self.v_mix

    @property
    def stateful(self) -> bool:
        return self.kind in ("gla", "delta", "ssd")

    @property
    def channels(self) -> int:
        """ssd: what passes the filter."""
        return self.heads * self.vdim + 2 * self.groups * self.dim

    def rope_frequencies(self) -> list[float]:
        """Angle per position of every rotated pair: base^(-2i/dims); with ``rope_scaling``, wavelengths longer than original / low are divided by the factor,
        shorter than original / high kept, and those between mixed."""
        out = []
        for i in range(self.rope_dims // 2):
            f = self.rope_base ** (-2.0 * i / self.rope_dims)
            if self.rope_scaling is not None:
                factor, low, high, original = self.rope_scaling
                turns = original * f / (2.0 * math.pi)               # original over the wavelength
                keep = min(1.0, max(0.0, (turns - low) / (high - low)))
                f = (1.0 - keep) * f / factor + keep * f
            out.append(f)
        return out


@dataclass(frozen=True)
class ExpertSpec:
    """A mixture of feed-forwards in place of one: each token uses the ``top`` experts with the largest scores.  ``score`` "sigmoid": weights are the sigmoids
    of the chosen router logits, as they are; "softmax": the softmax of all logits, renormalised over the chosen; times ``scale``.  ``weigh`` "input": the weight
    multiplies what goes into an expert; "output": what comes out.  ``shared``: width of one more feed-forward that every token uses (0: none)."""
    experts: int
    top: int
    score: str = "sigmoid"
    scale: float = 1.0
    weigh: str = "input"
    shared: int = 0

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError("a token's experts must be at least one and no more than there are")
        if self.score not in ("sigmoid", "softmax") or self.weigh not in ("input", "output") or self.shared < 0:
            raise ValueError("bad router score, place of the weight or shared width")


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a hybrid stack: a mixer and, unless ``ffn`` is 0, a feed-forward of that width (with ``moe``: experts of that width each); a norm
    before each and, where the model has them (``ModelConfig.post_norm``), behind each."""
    mixer: MixerSpec
    ffn: int = 0
    act: str = "relu2"             # "relu2": the square of relu; "gelu": the exact (erf) gelu; "polynorm": unit-RMS powers 1 to 3, mixed; "swiglu"
    moe: ExpertSpec | None = None


@dataclass(frozen=True)
class ModelConfig:
    arch: str = "llama"            # llama | gpt2 | gpt-oss | folirax | pesorax | kazolorn | tekosun
    n_layers: int = 2
    d_model: int = 256
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 64
    ffn: int = 688
    vocab: int = 32000
    context: int = 2048
    rope_theta: float = 10000.0
    rope_style: str = "pairs"      # "pairs": (2i, 2i+1) rotate together; "half": (i, i + hd/2)
    norm_eps: float = 1e-5
    tied_embeddings: bool = False
    # mixture of experts (gpt-oss)
    n_experts: int = 0
    top_k: int = 0
    sliding_window: int = 0        # 0 = every layer attends to the full context
    swa_every: int = 2             # layer i uses the window when sliding_window > 0 and i % swa_every == 0
    attn_sinks: bool = False
    qkv_bias: bool = False
    # hybrid stacks: the layers one by one (the flat head and width fields above then hold the largest of each)
    layers: tuple[LayerSpec, ...] = ()
    norm: str = "rms"              # "rms": root-mean-square, weights stored around zero; "rms1": the same, stored as they are; "dyt": w * tanh(alpha x) + b
    walk: str = "serial"           # "parallel": mixer and feed-forward of a layer read the same residual (a norm each) and are added together
    layer_scale: bool = False      # a learned factor per channel on what either adds
    depth_average: bool = False    # what a layer hands on is a learned mixture of the embedding output and every layer's result so far
    pre_norm: bool = True          # a norm ahead of every sublayer
    post_norm: bool = True         # a norm behind every sublayer
    embed_scale: float = 1.0       # multiplies the embedding
    residual_mult: float = 1.0     # multiplies what a sublayer adds to the residual (stacks without post_norm)
    loop: tuple[int, int, int] | None = None     # (start, stop, times): these layers run ``times`` times in a row, the embedding added ahead of every pass but the first
    logit_scale: float = 1.0
    logit_softcap: float = 0.0     # 0 = none
    name: str = "tiny-llama"

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    def layer_uses_window(self, i: int) -> bool:
        return self.sliding_window > 0 and i % self.swa_every == 0

    def layer_runs(self) -> list[tuple[int, bool]]:
        """Hybrid stacks: the layers in the order they run, and whether the embedding is added to the residual ahead of each."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop
        body = [(i, p > 0 and i == a) for p in range(times) for i in range(a, b)]
        return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]

    @property
    def has_state(self) -> bool:
        """Whether some layer carries a recurrent state from token to token."""
        return any(l.mixer.stateful for l in self.layers)

    def n_params(self) -> int:
        d, f, v = self.d_model, self.ffn, self.vocab
        if self.layers:
            from .weights import tensor_specs
            n = 0
            for s in tensor_specs(self):
                k = 1
                for e in s.shape:
                    k *= e
                n += k
            return n
        if self.arch == "gpt2":
            per = 4 * d * d + 2 * d * f + 9 * d + f
            return self.n_layers * per + v * d + self.context * d + 2 * d
        attn = d * self.q_dim * 2 + d * self.kv_dim * 2
        mlp = 3 * d * f * max(1, self.n_experts)
        emb = v * d * (1 if self.tied_embeddings else 2)
        return self.n_layers * (attn + mlp + 2 * d) + emb + d

    def to_gguf_metadata(self) -> dict:
        a = self.arch
        if self.layers:
            return {"general.architecture": a, "general.name": self.name, f"{a}.context_length": self.context,
                    "b200.model_json": json.dumps(hybrid_to_json(self))}
        md = {
            "general.architecture": a,
            "general.name": self.name,
            f"{a}.block_count": self.n_layers,
            f"{a}.embedding_length": self.d_model,
            f"{a}.feed_forward_length": self.ffn,
            f"{a}.attention.head_count": self.n_heads,
            f"{a}.attention.head_count_kv": self.n_kv_heads,
            f"{a}.attention.key_length": self.head_dim,
            f"{a}.attention.layer_norm_rms_epsilon": float(self.norm_eps),
            f"{a}.rope.freq_base": float(self.rope_theta),
            f"{a}.context_length": self.context,
            f"{a}.vocab_size": self.vocab,
            "b200.rope_style": self.rope_style,
            "b200.tied_embeddings": self.tied_embeddings,
        }
        if self.n_experts:
            md[f"{a}.expert_count"] = self.n_experts
            md[f"{a}.expert_used_count"] = self.top_k
        if self.sliding_window:
            md[f"{a}.attention.sliding_window"] = self.sliding_window
            md["b200.swa_every"] = self.swa_every
        md["b200.attn_sinks"] = self.attn_sinks
        md["b200.qkv_bias"] = self.qkv_bias
        return md

    @staticmethod
    def from_gguf_metadata(md: dict) -> "ModelConfig":
        a = md.get("general.architecture")
        own = md.get("b200.model_json")
        if own:
            return config_from_json(json.loads(own if isinstance(own, str) else bytes(own).decode()), name=md.get("general.name", a),
                                    context=int(md.get(f"{a}.context_length", HYBRID_CONTEXT)))
        if a not in ("llama", "gpt2", "gpt-oss"):
            raise ValueError(f"unsupported architecture {a!r}")
        g = lambda k, dflt=None: md.get(f"{a}.{k}", dflt)
        n_heads = int(g("attention.head_count"))
        d = int(g("embedding_length"))
        hd = int(g("attention.key_length", d // n_heads))
        return ModelConfig(
            arch=a, n_layers=int(g("block_count")), d_model=d, n_heads=n_heads,
            n_kv_heads=int(g("attention.head_count_kv", n_heads)), head_dim=hd,
            ffn=int(g("feed_forward_length")), vocab=int(g("vocab_size", 0)),
            context=int(g("context_length", 2048)), rope_theta=float(g("rope.freq_base", 10000.0)),
            rope_style=md.get("b200.rope_style", "half" if a == "gpt-oss" else "pairs"),
            norm_eps=float(g("attention.layer_norm_rms_epsilon", g("attention.layer_norm_epsilon", 1e-5))),
            tied_embeddings=bool(md.get("b200.tied_embeddings", a == "gpt2")),
            n_experts=int(g("expert_count", 0)), top_k=int(g("expert_used_count", 0)),
            sliding_window=int(g("attention.sliding_window", 0)), swa_every=int(md.get("b200.swa_every", 2)),
            attn_sinks=bool(md.get("b200.attn_sinks", a == "gpt-oss")),
            qkv_bias=bool(md.get("b200.qkv_bias", a == "gpt2")),
            name=md.get("general.name", a))

    def with_(self, **kw) -> "ModelConfig":
        return replace(self, **kw)

    def as_dict(self) -> dict:
        return asdict(self)


# ------------------------------------------------------------------ configurations given as JSON
HYBRID_CONTEXT = 1 << 20           # such a file names no limit; the engine's cache sets it


def _need(d: dict, key: str, kind, where: str):
    v = d.get(key) if isinstance(d, dict) else None
    if kind is float:
        ok = isinstance(v, (int, float)) and not isinstance(v, bool)
    else:
        ok = isinstance(v, kind) and not isinstance(v, bool)
    if not ok:
        raise ValueError(f"config: {where}{key} must be {'a number' if kind is float else kind.__name__}")
    return float(v) if kind is float else v


def _folirax(c: dict, ranks: dict[int, int], name: str, context: int) -> ModelConfig:
    """Folirax: attention (rotated, then unit-RMS queries and keys, a sigmoid gate per head, keys and values optionally those of an
    earlier layer) and gated linear attention in any order, a norm on both sides of every sublayer, squared-relu
    feed-forwards, scaled and soft-capped logits."""
    layers = []
    for i, e in enumerate(_need(c, "layers", list, "")):
        w = f"layers[{i}]."
        mx, kind = _need(e, "mixer", dict, w), _need(e, "type", str, w)
        w2 = w + "mixer."
        common = dict(heads=_need(mx, "heads", int, w2), dim=_need(mx, "dim", int, w2), vdim=_need(mx, "vdim", int, w2))
        if kind == "gla":
            m = MixerSpec("gla", **common, tau=_need(mx, "tau", float, w2), rank=ranks.get(i, MixerSpec.rank))
        elif kind == "attention":
            src = mx.get("kv_from")
            rot = {"base": 1.0, "dims": 0} if "rot" in mx and mx["rot"] is None else _need(mx, "rot", dict, w2)      # null: no rotation
            m = MixerSpec("attention", **common, kv_heads=_need(mx, "kv_heads", int, w2), scale=_need(mx, "scale", float, w2),
                          rope_base=_need(rot, "base", float, w2 + "rot."), rope_dims=_need(rot, "dims", int, w2 + "rot."),
                          qk_norm=True, head_gate=True, kv_from=None if src is None else _need(mx, "kv_from", int, w2))
            if src is not None:
                if not 0 <= src < i or layers[src].mixer.kind != "attention" or layers[src].mixer.kv_from is not None:
                    raise ValueError(f"config: {w2}kv_from must name an earlier attention layer with keys and values of its own")
                o = layers[src].mixer
                if (o.kv_heads, o.dim, o.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"config: {w2}kv_from names a layer with other key/value sizes")
        else:
            raise ValueError(f"config: {w}type {kind!r} is not a mixer of this design")
        mlp = e.get("mlp")
        if mlp is not None and _need(mlp, "kind", str, w + "mlp.") != "dense":
            raise ValueError(f"config: {w}mlp.kind {mlp['kind']!r} is not known")
        layers.append(LayerSpec(m, 0 if mlp is None else _need(mlp, "ff", int, w + "mlp.")))
    if not layers:
        raise ValueError("config: layers is empty")
    mx = [l.mixer for l in layers]
    cap = c.get("logit_softcap")
    return ModelConfig(arch="folirax", n_layers=len(layers), d_model=_need(c, "width", int, ""), vocab=_need(c, "vocab", int, ""),
                       n_heads=max(m.heads for m in mx), n_kv_heads=max(1, *(m.kv_heads for m in mx)), head_dim=max(m.dim for m in mx),
                       ffn=max(l.ffn for l in layers), context=context, norm_eps=_need(_need(c, "norm", dict, ""), "eps", float, "norm."),
                       layers=tuple(layers), logit_scale=1.0 if c.get("logit_scale") is None else _need(c, "logit_scale", float, ""),
                       logit_softcap=0.0 if cap is None else _need(c, "logit_softcap", float, ""), name=name)


def _pesorax(c: dict, ranks: dict[int, int], name: str, context: int) -> ModelConfig:
    """Pesorax: chunked differential attention (biased projections, no positions in the scores) and latent attention (a query latent, half-split
    rotation of a shared key part, sinks, a gate per output element) in any order, Dynamic Tanh ahead of every sublayer, scaled
    residual branches, erf-gelu feed-forwards, and a span of layers that runs several times."""
    layers = []
    for i, e in enumerate(_need(c, "layers", list, "")):
        w = f"layers[{i}]."
        mx, kind = _need(e, "mixer", dict, w), _need(e, "type", str, w)
        w2 = w + "mixer."
        common = dict(heads=_need(mx, "heads", int, w2), dim=_need(mx, "dim", int, w2), vdim=_need(mx, "vdim", int, w2), scale=_need(mx, "scale", float, w2))
        if kind == "attention":
            chunk = 0 if mx.get("mask") is None else _need(_need(mx, "mask", dict, w2), "size", int, w2 + "mask.")
            if mx.get("mask") is not None and chunk < 1:
                raise ValueError(f"config: {w2}mask.size must be positive")
            m = MixerSpec("attention", **common, kv_heads=_need(mx, "kv_heads", int, w2), bias=True, chunk=chunk, maps=2, diff=_need(mx, "diff", float, w2))
        elif kind == "latent_attention":
            rot = _need(mx, "rot", dict, w2)
            rank = _need(mx, "q_rank", int, w2) if mx.get("q_rank") is not None or i not in ranks else ranks[i]
            m = MixerSpec("latent", **common, rot_dim=_need(mx, "rot_dim", int, w2), kv_rank=_need(mx, "kv_rank", int, w2), q_rank=rank,
                          rope_base=_need(rot, "base", float, w2 + "rot."), rope_dims=_need(rot, "dims", int, w2 + "rot."), rope_style="half",
                          sink=True, out_gate=True)
        else:
            raise ValueError(f"config: {w}type {kind!r} is not a mixer of this design")
        mlp = e.get("mlp")
        if mlp is not None and _need(mlp, "kind", str, w + "mlp.") != "dense":
            raise ValueError(f"config: {w}mlp.kind {mlp['kind']!r} is not known")
        layers.append(LayerSpec(m, 0 if mlp is None else _need(mlp, "ff", int, w + "mlp."), "gelu"))
    if not layers:
        raise ValueError("config: layers is empty")
    loop = None
    if c.get("loop") is not None:
        lp = _need(c, "loop", dict, "")
        loop = tuple(_need(lp, k, int, "loop.") for k in ("start", "stop", "times"))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError("config: loop must name a span of layers and a positive number of passes")
    mx = [l.mixer for l in layers]
    return ModelConfig(arch="pesorax", n_layers=len(layers), d_model=_need(c, "width", int, ""), vocab=_need(c, "vocab", int, ""),
                       n_heads=max(m.heads for m in mx), n_kv_heads=max(1, *(m.kv_heads for m in mx)), head_dim=max(m.dim for m in mx),
                       ffn=max(l.ffn for l in layers), context=context, norm_eps=_need(_need(c, "norm", dict, ""), "eps", float, "norm."),
                       layers=tuple(layers), norm="dyt", post_norm=False, loop=loop,
                       residual_mult=1.0 if c.get("residual_mult") is None else _need(c, "residual_mult", float, ""), name=name)


def _pesorax_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for l in cfg.layers:
        m = l.mixer
        mx = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
        if m.kind == "latent":
            mx.update(rot_dim=m.rot_dim, kv_rank=m.kv_rank, q_rank=m.q_rank, rot={"base": m.rope_base, "dims": m.rope_dims})
        else:
            mx.update(kv_heads=m.kv_heads, diff=m.diff, mask={"size": m.chunk} if m.chunk else None)
        layers.append({"type": "latent_attention" if m.kind == "latent" else "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": l.ffn} if l.ffn else None})
    return {"architecture": "Pesorax", "layers": layers, "width": cfg.d_model, "vocab": cfg.vocab, "norm": {"eps": cfg.norm_eps},
            "loop": None if cfg.loop is None else dict(zip(("start", "stop", "times"), cfg.loop)), "residual_mult": cfg.residual_mult}


def _kazolorn(c: dict, ranks: dict[int, int], name: str, context: int) -> ModelConfig:
    """Kazolorn: sliding-window attention whose keys are its values, with a distance bias, mixed heads and a silent sink; the feed-forward (PolyNorm, or
    experts whose weights scale their input) in parallel, both scaled per channel; a depth average behind every layer."""
    layers = []
    for i, e in enumerate(_need(c, "layers", list, "")):
        w = f"layers[{i}]."
        mx, kind = _need(e, "mixer", dict, w), _need(e, "type", str, w)
        w2 = w + "mixer."
        if kind != "attention":
            raise ValueError(f"config: {w}type {kind!r} is not a mixer of this design")
        window = _need(_need(mx, "mask", dict, w2), "size", int, w2 + "mask.")
        if window < 1:
            raise ValueError(f"config: {w2}mask.size must be positive")
        dim = _need(mx, "dim", int, w2)
        m = MixerSpec("attention", _need(mx, "heads", int, w2), dim, dim if mx.get("vdim") is None else _need(mx, "vdim", int, w2),
                      kv_heads=_need(mx, "kv_heads", int, w2), scale=_need(mx, "scale", float, w2), bias=True, out_bias=True, window=window, tied_kv=True,
                      distance_bias=True, mix_heads=True, silent_sink=True)
        mlp, ff, moe = e.get("mlp"), 0, None
        if mlp is not None:
            kind = _need(mlp, "kind", str, w + "mlp.")
            if kind == "dense":
                ff = _need(mlp, "ff", int, w + "mlp.")
            elif kind == "moe":
                ff = _need(_need(mlp, "expert", dict, w + "mlp."), "ff", int, w + "mlp.expert.")
                router = _need(mlp, "router", dict, w + "mlp.")
                moe = ExpertSpec(_need(router, "experts", int, w + "mlp.router."), _need(router, "top", int, w + "mlp.router."))
            else:
                raise ValueError(f"config: {w}mlp.kind {kind!r} is not known")
            if ff < 1:
                raise ValueError(f"config: {w}mlp: the width must be positive")
        layers.append(LayerSpec(m, ff, "swiglu" if moe else "polynorm", moe))
    if not layers:
        raise ValueError("config: layers is empty")
    mx = [l.mixer for l in layers]
    return ModelConfig(arch="kazolorn", n_layers=len(layers), d_model=_need(c, "width", int, ""), vocab=_need(c, "vocab", int, ""),
                       n_heads=max(m.heads for m in mx), n_kv_heads=max(m.kv_heads for m in mx), head_dim=max(m.dim for m in mx),
                       ffn=max(l.ffn for l in layers), context=context, norm_eps=_need(_need(c, "norm", dict, ""), "eps", float, "norm."),
                       layers=tuple(layers), norm="rms1", post_norm=False, walk="parallel", layer_scale=True, depth_average=True, name=name)


def _kazolorn_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for l in cfg.layers:
        m, mlp = l.mixer, None
        if l.moe:
            mlp = {"kind": "moe", "expert": {"ff": l.ffn}, "router": {"experts": l.moe.experts, "top": l.moe.top}}
        elif l.ffn:
            mlp = {"kind": "dense", "ff": l.ffn}
        layers.append({"type": "attention", "mlp": mlp, "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                                                  "mask": {"size": m.window}}})
    return {"architecture": "Kazolorn", "layers": layers, "width": cfg.d_model, "vocab": cfg.vocab, "norm": {"eps": cfg.norm_eps}}


DELTA_LOG_DECAY = math.exp(-0.5)   # Tekosun: log decays lie between this, negated, and 0


def _tekosun(c: dict, ranks: dict[int, int], name: str, context: int) -> ModelConfig:
    """Tekosun: generalized delta rule, Mamba-2 and windowed attention (whole-row query and key norms, normed and mixed values, scaled rotation) in any order; a norm
    behind every sublayer only; mixtures of squared-relu experts with a shared one; a scaled embedding."""
    layers = []
    for i, e in enumerate(_need(c, "layers", list, "")):
        w = f"layers[{i}]."
        mx, kind = _need(e, "mixer", dict, w), _need(e, "type", str, w)
        w2 = w + "mixer."
        heads = _need(mx, "heads", int, w2)
        if kind == "general_delta":
            dim = _need(mx, "dim", int, w2)
            m = MixerSpec("delta", heads, dim, dim, log_decay=DELTA_LOG_DECAY, rank=ranks.get(i, MixerSpec.rank))
        elif kind == "mamba2":
            m = MixerSpec("ssd", heads, _need(mx, "state", int, w2), _need(mx, "vdim", int, w2), groups=_need(mx, "groups", int, w2),
                          norm_groups=_need(mx, "norm_groups", int, w2), conv=_need(mx, "conv", int, w2))
        elif kind == "attention":
            window = 0 if mx.get("mask") is None else _need(_need(mx, "mask", dict, w2), "size", int, w2 + "mask.")
            if mx.get("mask") is not None and window < 1:
                raise ValueError(f"config: {w2}mask.size must be positive")
            rot = {"base": 1.0, "dims": 0} if "rot" in mx and mx["rot"] is None else _need(mx, "rot", dict, w2)      # null: no rotation
            scaling = None
            if rot.get("scaling") is not None:
                sc = _need(rot, "scaling", dict, w2 + "rot.")
                scaling = tuple(_need(sc, k, float, w2 + "rot.scaling.") for k in ("factor", "low", "high", "original"))
            if not isinstance(mx.get("v_mix", False), bool):
                raise ValueError(f"config: {w2}v_mix must be true or false")
            dim = _need(mx, "dim", int, w2)
            m = MixerSpec("attention", heads, dim, dim if mx.get("vdim") is None else _need(mx, "vdim", int, w2), kv_heads=_need(mx, "kv_heads", int, w2),
                          scale=_need(mx, "scale", float, w2), rope_base=_need(rot, "base", float, w2 + "rot."), rope_dims=_need(rot, "dims", int, w2 + "rot."),
                          rope_style="half", rope_scaling=scaling, row_norm=True, v_norm=True, v_mix=mx.get("v_mix", False), window=window)
            first = next((l.mixer for l in layers if l.mixer.v_mix), m)
            if m.v_mix and (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                raise ValueError(f"config: {w2}v_mix: the values have another size than the first such layer's")
        else:
            raise ValueError(f"config: {w}type {kind!r} is not a mixer of this design")
        mlp, ff, moe = e.get("mlp"), 0, None
        if mlp is not None:
            if _need(mlp, "kind", str, w + "mlp.") != "moe":
                raise ValueError(f"config: {w}mlp.kind {mlp['kind']!r} is not known")
            ff = _need(_need(mlp, "expert", dict, w + "mlp."), "ff", int, w + "mlp.expert.")
            router = _need(mlp, "router", dict, w + "mlp.")
            shared = 0 if mlp.get("shared") is None else _need(_need(mlp, "shared", dict, w + "mlp."), "ff", int, w + "mlp.shared.")
            if ff < 1 or (mlp.get("shared") is not None and shared < 1):
                raise ValueError(f"config: {w}mlp: the widths must be positive")
            w3 = w + "mlp.router."
            moe = ExpertSpec(_need(router, "experts", int, w3), _need(router, "top", int, w3), "softmax",
                             1.0 if router.get("scale") is None else _need(router, "scale", float, w3), "output", shared)
        layers.append(LayerSpec(m, ff, "relu2", moe))
    if not layers:
        raise ValueError("config: layers is empty")
    mx = [l.mixer for l in layers]
    scale = 1.0 if c.get("embedding") is None or c["embedding"].get("scale") is None else _need(c["embedding"], "scale", float, "embedding.")
    return ModelConfig(arch="tekosun", n_layers=len(layers), d_model=_need(c, "width", int, ""), vocab=_need(c, "vocab", int, ""),
                       n_heads=max(m.heads for m in mx), n_kv_heads=max(1, *(m.kv_heads for m in mx)), head_dim=max(m.dim for m in mx),
                       ffn=max(l.ffn for l in layers), context=context, norm_eps=_need(_need(c, "norm", dict, ""), "eps", float, "norm."),
                       layers=tuple(layers), norm="rms1", pre_norm=False, embed_scale=scale, name=name)


def _tekosun_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for l in cfg.layers:
        m, mlp = l.mixer, None
        if m.kind == "delta":
            kind, mx = "general_delta", {"heads": m.heads, "dim": m.dim}
        elif m.kind == "ssd":
            kind, mx = "mamba2", {"heads": m.heads, "vdim": m.vdim, "state": m.dim, "groups": m.groups, "norm_groups": m.norm_groups, "conv": m.conv}
        else:
            rot = {"base": m.rope_base, "dims": m.rope_dims}
            if m.rope_scaling is not None:
                rot["scaling"] = dict(zip(("factor", "low", "high", "original"), m.rope_scaling))
            kind, mx = "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot, "v_mix": m.v_mix,
                                     "mask": {"size": m.window} if m.window else None}
        if l.moe:
            mlp = {"kind": "moe", "expert": {"ff": l.ffn}, "router": {"experts": l.moe.experts, "top": l.moe.top, "scale": l.moe.scale},
                   "shared": {"ff": l.moe.shared} if l.moe.shared else None}
        layers.append({"type": kind, "mixer": mx, "mlp": mlp})
    return {"architecture": "Tekosun", "layers": layers, "width": cfg.d_model, "vocab": cfg.vocab, "norm": {"eps": cfg.norm_eps},
            "embedding": {"scale": cfg.embed_scale}, "ranks": {str(i): l.mixer.rank for i, l in enumerate(cfg.layers) if l.mixer.kind == "delta"}}


def hybrid_to_json(cfg: ModelConfig) -> dict:
    """The inverse of ``config_from_json``."""
    if cfg.arch == "tekosun":
        return _tekosun_to_json(cfg)
    if cfg.arch == "pesorax":
        return _pesorax_to_json(cfg)
    if cfg.arch == "kazolorn":
        return _kazolorn_to_json(cfg)
    layers = []
    for l in cfg.layers:
        m = l.mixer
        mx = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if m.kind == "gla":
            mx.update(tau=m.tau)
        else:
            mx.update(kv_heads=m.kv_heads, scale=m.scale, rot={"base": m.rope_base, "dims": m.rope_dims})
            if m.kv_from is not None:
                mx["kv_from"] = m.kv_from
        layers.append({"type": m.kind, "mixer": mx, "mlp": {"kind": "dense", "ff": l.ffn} if l.ffn else None})
    return {"architecture": "Folirax", "layers": layers, "width": cfg.d_model, "vocab": cfg.vocab, "norm": {"eps": cfg.norm_eps},
            "logit_scale": cfg.logit_scale, "logit_softcap": cfg.logit_softcap,
            "ranks": {str(i): l.mixer.rank for i, l in enumerate(cfg.layers) if l.mixer.kind == "gla"}}


JSON_ARCHITECTURES = {"Folirax": _folirax, "Pesorax": _pesorax, "Kazolorn": _kazolorn, "Tekosun": _tekosun}
HYBRID_ARCHS = tuple(a.lower() for a in JSON_ARCHITECTURES)


def config_from_json(c: dict, ranks: dict[int, int] | None = None, name: str | None = None, context: int = HYBRID_CONTEXT) -> ModelConfig:
    """A model configuration from a checkpoint folder's config.json.  ``ranks``: sizes the file may leave to the tensors' shapes, by layer
    (rank of the decay projection, size of the queries' latent)."""
    arch = _need(c, "architecture", str, "")
    reader = JSON_ARCHITECTURES.get(arch)
    if reader is None:
        raise ValueError(f"unsupported architecture {arch!r}")
    if ranks is None:
        ranks = {int(k): int(v) for k, v in c.get("ranks", {}).items()}
    return reader(c, ranks, name or arch.lower(), context)


TINY_LLAMA = ModelConfig()
LLAMA3_8B = ModelConfig(arch="llama", n_layers=32, d_model=4096, n_heads=32, n_kv_heads=8, head_dim=128,
                        ffn=14336, vocab=128256, context=8192, rope_theta=500000.0, name="llama-3-8b-shape")
LLAMA3_70B = ModelConfig(arch="llama", n_layers=80, d_model=8192, n_heads=64, n_kv_heads=8, head_dim=128,
                         ffn=28672, vocab=128256, context=16384, rope_theta=500000.0, name="llama-3-70b-shape")
GPT2_SMALL = ModelConfig(arch="gpt2", n_layers=12, d_model=768, n_heads=12, n_kv_heads=12, head_dim=64,
                         ffn=3072, vocab=50257, context=1024, tied_embeddings=True, qkv_bias=True,
                         name="gpt2-small-shape")
GPT_OSS_20B = ModelConfig(arch="gpt-oss", n_layers=24, d_model=2880, n_heads=64, n_kv_heads=8, head_dim=64,
                          ffn=2880, vocab=201088, context=8192, rope_theta=150000.0, rope_style="half",
                          n_experts=32, top_k=4, sliding_window=128, swa_every=2, attn_sinks=True,
                          name="gpt-oss-20b-shape")



def folirax_stack(width: int, ffn: int, vocab: int, groups: int, heads: int, kv_heads: int, head_dim: int, gla_heads: int, gla_dim: int,
                  gla_vdim: int, name: str, ratio: int = 2) -> ModelConfig:
    """A regular stack: ``groups`` times (``ratio`` recurrent layers, then an attention layer with keys and values of its own and one
    that shares them)."""
    gla = LayerSpec(MixerSpec("gla", gla_heads, gla_dim, gla_vdim, tau=16.0), ffn)
    own = MixerSpec("attention", heads, head_dim, head_dim, kv_heads=kv_heads, scale=head_dim ** -0.5, rope_dims=head_dim // 2, qk_norm=True,
                    head_gate=True)
    layers: list[LayerSpec] = []
    for _ in range(groups):
        layers += [gla] * ratio
        layers += [LayerSpec(own, ffn), LayerSpec(replace(own, kv_from=len(layers)), ffn)]
    return ModelConfig(arch="folirax", n_layers=len(layers), d_model=width, n_heads=max(heads, gla_heads), n_kv_heads=kv_heads,
                       head_dim=max(head_dim, gla_dim), ffn=ffn, vocab=vocab, context=HYBRID_CONTEXT, norm_eps=1e-6, layers=tuple(layers),
                       logit_scale=0.5, logit_softcap=30.0, name=name)


# layers of the size of the 8B preset's (width, heads, feed-forward), and a smaller stack
FOLIRAX_8B = folirax_stack(4096, 14336, 128256, 8, 32, 8, 128, 16, 128, 256, "folirax-8b-shape")
FOLIRAX_1B = folirax_stack(2048, 8192, 32000, 4, 16, 4, 128, 8, 128, 256, "folirax-1b-shape")



def pesorax_stack(width: int, ffn: int, vocab: int, groups: int, heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, latent_heads: int,
                  latent_dim: int, rot_dim: int, latent_vdim: int, kv_rank: int, q_rank: int, name: str, loop: tuple[int, int, int] | None = None) -> ModelConfig:
    """A regular stack: ``groups`` times (three chunked differential attention layers, then a latent attention layer)."""
    local = LayerSpec(MixerSpec("attention", heads, dim, vdim, kv_heads=kv_heads, scale=dim ** -0.5, bias=True, chunk=chunk, maps=2, diff=0.5), ffn, "gelu")
    latent = LayerSpec(MixerSpec("latent", latent_heads, latent_dim, latent_vdim, scale=(latent_dim + rot_dim) ** -0.5, rope_base=500000.0, rope_dims=rot_dim,
                                 rope_style="half", rot_dim=rot_dim, kv_rank=kv_rank, q_rank=q_rank, sink=True, out_gate=True), ffn, "gelu")
    layers = (local, local, local, latent) * groups
    return ModelConfig(arch="pesorax", n_layers=len(layers), d_model=width, n_heads=max(heads, latent_heads), n_kv_heads=kv_heads, head_dim=max(dim, latent_dim),
                       ffn=ffn, vocab=vocab, context=HYBRID_CONTEXT, norm_eps=1e-5, layers=layers, norm="dyt", post_norm=False, loop=loop, residual_mult=0.5,
                       name=name)


# the same two sizes with differential and latent attention; the smaller one runs its middle layers twice
PESORAX_8B = pesorax_stack(4096, 14336, 128256, 8, 16, 4, 64, 128, 2048, 32, 128, 64, 128, 512, 1536, "pesorax-8b-shape")
PESORAX_1B = pesorax_stack(2048, 8192, 32000, 3, 8, 2, 64, 128, 1024, 16, 128, 64, 128, 512, 768, "pesorax-1b-shape", loop=(4, 8, 2))


def kazolorn_stack(width: int, ffn: int, vocab: int, layers: int, heads: int, kv_heads: int, dim: int, window: int, name: str, experts: int = 0, top: int = 0,
                   expert_ffn: int = 0, dense: int = 1) -> ModelConfig:
    """A regular stack: ``dense`` layers with one feed-forward, the others (all of them without ``experts``) with a mixture."""
    m = MixerSpec("attention", heads, dim, dim, kv_heads=kv_heads, scale=dim ** -0.5, bias=True, out_bias=True, window=window, tied_kv=True, distance_bias=True,
                  mix_heads=True, silent_sink=True)
    own, mixture = LayerSpec(m, ffn, "polynorm"), LayerSpec(m, expert_ffn, "swiglu", ExpertSpec(experts, top)) if experts else None
    stack = tuple(mixture if experts and i >= dense else own for i in range(layers))
    return ModelConfig(arch="kazolorn", n_layers=layers, d_model=width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim, ffn=max(ffn, expert_ffn), vocab=vocab,
                       context=HYBRID_CONTEXT, norm_eps=1e-5, layers=stack, norm="rms1", post_norm=False, walk="parallel", layer_scale=True,
                       depth_average=True, name=name)


# layers of the 8B preset's size with one feed-forward each, and a smaller stack whose layers (but the first) have 32 experts of which a token uses four
KAZOLORN_8B = kazolorn_stack(4096, 14336, 128256, 32, 32, 8, 128, 4096, "kazolorn-8b-shape")
KAZOLORN_MOE = kazolorn_stack(2048, 8192, 32000, 16, 16, 4, 128, 1024, "kazolorn-moe-shape", experts=32, top=4, expert_ffn=2048)

def tekosun_stack(width: int, vocab: int, groups: int, heads: int, kv_heads: int, dim: int, window: int, delta_heads: int, delta_dim: int, rank: int, ssd_heads: int,
                  ssd_vdim: int, state: int, experts: int, top: int, expert_ffn: int, shared: int, name: str) -> ModelConfig:
    """A regular stack: ``groups`` times (delta rule, attention, delta rule, state-space duality), a mixture of experts behind each."""
    moe = ExpertSpec(experts, top, "softmax", 1.5, "output", shared)
    delta = LayerSpec(MixerSpec("delta", delta_heads, delta_dim, delta_dim, log_decay=DELTA_LOG_DECAY, rank=rank), expert_ffn, "relu2", moe)
    attn = LayerSpec(MixerSpec("attention", heads, dim, dim, kv_heads=kv_heads, scale=dim ** -0.5, rope_base=500000.0, rope_dims=dim, rope_style="half",
                               rope_scaling=(8.0, 1.0, 4.0, 8192.0), row_norm=True, v_norm=True, v_mix=True, window=window), expert_ffn, "relu2", moe)
    ssd = LayerSpec(MixerSpec("ssd", ssd_heads, state, ssd_vdim, groups=1, norm_groups=1, conv=4), expert_ffn, "relu2", moe)
    layers = (delta, attn, delta, ssd) * groups
    return ModelConfig(arch="tekosun", n_layers=len(layers), d_model=width, n_heads=max(heads, delta_heads, ssd_heads), n_kv_heads=kv_heads,
                       head_dim=max(dim, delta_dim, state), ffn=expert_ffn, vocab=vocab, context=HYBRID_CONTEXT, norm_eps=1e-6, layers=layers, norm="rms1",
                       pre_norm=False, embed_scale=4.0, name=name)


# layers of the 8B preset's width, and a smaller stack; 32 experts of which a token uses four, and a shared one of the size of two
TEKOSUN_8B = tekosun_stack(4096, 128256, 8, 32, 8, 128, 4096, 64, 64, 128, 128, 64, 128, 32, 4, 2048, 4096, "tekosun-8b-shape")
TEKOSUN_1B = tekosun_stack(2048, 32000, 4, 16, 4, 128, 1024, 32, 64, 96, 64, 64, 128, 32, 4, 1024, 2048, "tekosun-1b-shape")

PRESETS = {c.name: c for c in (TINY_LLAMA, LLAMA3_8B, LLAMA3_70B, GPT2_SMALL, GPT_OSS_20B, FOLIRAX_8B, FOLIRAX_1B, PESORAX_8B, PESORAX_1B, KAZOLORN_8B,
                               KAZOLORN_MOE, TEKOSUN_8B, TEKOSUN_1B)}
