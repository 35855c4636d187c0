"""Tensor inventories, seeded random initialisation and GGUF save/load of whole models.

Weights are N(0, 0.02) from a seeded generator (one stream per tensor, so the values do not depend
on creation order); norm gains are ones and stay F32 in the file.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass

import torch

from ..gguf import GGUFFile, GGUFWriter, GgmlType, type_block
from .config import ModelConfig


@dataclass
class TensorSpec:
    name: str
    shape: tuple[int, ...]
    kind: str   # "matrix" | "embed" | "output" | "norm" | "bias" | "expert" | "router" | "sink" | "pos" | "average"


def tensor_specs(cfg: ModelConfig) -> list[TensorSpec]:
    d, f, V = cfg.d_model, cfg.ffn, cfg.vocab
    if cfg.layers:
        return hybrid_tensor_specs(cfg)
    s: list[TensorSpec] = [TensorSpec("token_embd.weight", (V, d), "embed")]
    if cfg.arch == "gpt2":
        s.append(TensorSpec("position_embd.weight", (cfg.context, d), "pos"))
    for i in range(cfg.n_layers):
        p = f"blk.{i}."
        if cfg.arch == "gpt2":
            s += [TensorSpec(p + "attn_norm.weight", (d,), "norm"), TensorSpec(p + "attn_norm.bias", (d,), "bias"),
                  TensorSpec(p + "attn_qkv.weight", (3 * d, d), "matrix"), TensorSpec(p + "attn_qkv.bias", (3 * d,), "bias"),
                  TensorSpec(p + "attn_output.weight", (d, d), "matrix"), TensorSpec(p + "attn_output.bias", (d,), "bias"),
                  TensorSpec(p + "ffn_norm.weight", (d,), "norm"), TensorSpec(p + "ffn_norm.bias", (d,), "bias"),
                  TensorSpec(p + "ffn_up.weight", (f, d), "matrix"), TensorSpec(p + "ffn_up.bias", (f,), "bias"),
                  TensorSpec(p + "ffn_down.weight", (d, f), "matrix"), TensorSpec(p + "ffn_down.bias", (d,), "bias")]
            continue
        s += [TensorSpec(p + "attn_norm.weight", (d,), "norm"),
              TensorSpec(p + "attn_q.weight", (cfg.q_dim, d), "matrix"),
              TensorSpec(p + "attn_k.weight", (cfg.kv_dim, d), "matrix"),
              TensorSpec(p + "attn_v.weight", (cfg.kv_dim, d), "matrix"),
              TensorSpec(p + "attn_output.weight", (d, cfg.q_dim), "matrix")]
        if cfg.qkv_bias:
            s += [TensorSpec(p + "attn_q.bias", (cfg.q_dim,), "bias"), TensorSpec(p + "attn_k.bias", (cfg.kv_dim,), "bias"),
                  TensorSpec(p + "attn_v.bias", (cfg.kv_dim,), "bias"), TensorSpec(p + "attn_output.bias", (d,), "bias")]
        if cfg.attn_sinks:
            s.append(TensorSpec(p + "attn_sinks.weight", (cfg.n_heads,), "sink"))
        s.append(TensorSpec(p + "ffn_norm.weight", (d,), "norm"))
        if cfg.n_experts:
            E = cfg.n_experts
            s += [TensorSpec(p + "ffn_gate_inp.weight", (E, d), "router"),
                  TensorSpec(p + "ffn_gate_exps.weight", (E, f, d), "expert"),
                  TensorSpec(p + "ffn_up_exps.weight", (E, f, d), "expert"),
                  TensorSpec(p + "ffn_down_exps.weight", (E, d, f), "expert")]
        else:
            s += [TensorSpec(p + "ffn_gate.weight", (f, d), "matrix"),
                  TensorSpec(p + "ffn_up.weight", (f, d), "matrix"),
                  TensorSpec(p + "ffn_down.weight", (d, f), "matrix")]
    s.append(TensorSpec("output_norm.weight", (d,), "norm"))
    if cfg.arch == "gpt2":
        s.append(TensorSpec("output_norm.bias", (d,), "bias"))
    if not cfg.tied_embeddings:
        s.append(TensorSpec("output.weight", (V, d), "output"))
    return s


def hybrid_tensor_specs(cfg: ModelConfig) -> list[TensorSpec]:
    """Hybrid stacks go by their checkpoints' own tensor names.  Norms stored around zero are of kind "bias" (initialised to 0)."""
    d = cfg.d_model

    def norm(name):
        if cfg.norm == "dyt":
            return [TensorSpec(name, (d,), "norm"), TensorSpec(name + ".b", (d,), "bias"), TensorSpec(name + ".alpha", (1,), "norm")]
        return [TensorSpec(name, (d,), "norm" if cfg.norm == "rms1" else "bias")]
    s = [TensorSpec("embed", (cfg.vocab, d), "embed")]
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        for n in ("norm1", "norm2") if l.ffn else ("norm1",):
            s += norm(p + n) + (norm(p + n + "b") if cfg.post_norm and cfg.pre_norm else [])
        p += "mix."
        if m.kind == "latent":
            qk = m.dim + m.rot_dim
            s += [TensorSpec(p + "dq", (m.q_rank, d), "matrix"), TensorSpec(p + "dq.norm", (m.q_rank,), "norm"),
                  TensorSpec(p + "uq", (m.heads * qk, m.q_rank), "matrix"), TensorSpec(p + "dkv", (m.kv_rank + m.rot_dim, d), "matrix"),
                  TensorSpec(p + "dkv.norm", (m.kv_rank,), "norm"), TensorSpec(p + "uk", (m.heads * m.dim, m.kv_rank), "matrix"),
                  TensorSpec(p + "uv", (m.heads * m.vdim, m.kv_rank), "matrix")]
            if m.sink:
                s.append(TensorSpec(p + "sink", (m.heads,), "bias"))
            if m.out_gate:
                s.append(TensorSpec(p + "g", (m.heads * m.vdim, d), "matrix"))
        elif m.kind == "delta":
            hd = m.heads * m.dim
            s += [TensorSpec(p + n, (hd, d), "matrix") for n in ("r", "k", "v", "g", "a")]
            s += [TensorSpec(p + "a.b", (hd,), "bias"), TensorSpec(p + "w1", (m.rank, d), "matrix"), TensorSpec(p + "w2", (hd, m.rank), "matrix"),
                  TensorSpec(p + "w0", (hd,), "bias"), TensorSpec(p + "norm", (hd,), "norm")]
        elif m.kind == "ssd":
            inner = m.heads * m.vdim
            s += [TensorSpec(p + "in", (inner + m.channels + m.heads, d), "matrix"), TensorSpec(p + "conv", (m.channels, m.conv), "sink"),
                  TensorSpec(p + "conv.b", (m.channels,), "bias"), TensorSpec(p + "dt_bias", (m.heads,), "bias"), TensorSpec(p + "A_log", (m.heads,), "bias"),
                  TensorSpec(p + "D", (m.heads,), "norm"), TensorSpec(p + "norm", (inner,), "norm")]
        else:
            s.append(TensorSpec(p + "q", (m.maps * m.heads * m.dim, d), "matrix"))
        if m.kind == "gla":
            s += [TensorSpec(p + "k", (m.heads * m.dim, d), "matrix"), TensorSpec(p + "v", (m.heads * m.vdim, d), "matrix"),
                  TensorSpec(p + "g", (m.heads * m.vdim, d), "matrix"), TensorSpec(p + "norm", (m.vdim,), "norm"),
                  TensorSpec(p + "a1", (m.rank, d), "matrix"), TensorSpec(p + "a2", (m.heads * m.dim, m.rank), "matrix"),
                  TensorSpec(p + "a2.b", (m.heads * m.dim,), "bias")]
        elif m.kind == "attention":
            if m.bias:
                s.append(TensorSpec(p + "q.b", (m.maps * m.heads * m.dim,), "bias"))
            if m.kv_from is None:
                for n, rows in [("k", m.maps * m.kv_heads * m.dim)] + ([] if m.tied_kv else [("v", m.kv_heads * m.vdim)]):
                    s += [TensorSpec(p + n, (rows, d), "matrix")] + ([TensorSpec(f"{p}{n}.b", (rows,), "bias")] if m.bias else [])
            if m.head_gate:
                s.append(TensorSpec(p + "g", (m.heads, d), "matrix"))
            if m.row_norm:
                s += [TensorSpec(p + "q.norm", (m.heads * m.dim,), "norm"), TensorSpec(p + "k.norm", (m.kv_heads * m.dim,), "norm")]
            if m.v_mix:
                s.append(TensorSpec(p + "vmix", (1,), "sink"))
            if m.maps == 2:
                s += [TensorSpec(p + n, (m.dim,), "bias") for n in ("lq1", "lk1", "lq2", "lk2")]
            if m.mix_heads:
                s.append(TensorSpec(p + "talk", (m.heads, m.heads), "sink"))
        s.append(TensorSpec(p + "o", (d, m.heads * m.vdim), "matrix"))
        if m.out_bias:
            s.append(TensorSpec(p + "o.b", (d,), "bias"))
        p = f"l{i}.mlp."
        if l.moe:
            parts = (["gate"] if l.act == "swiglu" else []) + ["up", "down"]
            for e, f in [(f"e{e}", l.ffn) for e in range(l.moe.experts)] + ([("shared", l.moe.shared)] if l.moe.shared else []):
                s += [TensorSpec(f"{p}{e}.{n}", (d, f) if n == "down" else (f, d), "matrix") for n in parts]
            s.append(TensorSpec(p + "router", (l.moe.experts, d), "router"))
        elif l.ffn:
            s += [TensorSpec(p + "up", (l.ffn, d), "matrix"), TensorSpec(p + "down", (d, l.ffn), "matrix")]
            if l.act == "polynorm":
                s.append(TensorSpec(p + "act", (4,), "norm"))
        if cfg.layer_scale:
            s += [TensorSpec(f"l{i}.{n}", (d,), "norm") for n in (("ls1", "ls2") if l.ffn else ("ls1",))]
        if cfg.depth_average:
            s.append(TensorSpec(f"l{i}.dwa", (i + 2,), "average"))
    return s + norm("final.norm") + [TensorSpec("head", (cfg.vocab, d), "output")]


@dataclass(frozen=True)
class QuantPlan:
    """Which block format each tensor kind is stored in."""
    matrix: GgmlType = GgmlType.Q8_0
    embed: GgmlType = GgmlType.Q8_0
    output: GgmlType = GgmlType.Q8_0
    expert: GgmlType = GgmlType.MXFP4
    router: GgmlType = GgmlType.F32

    def type_for(self, spec: TensorSpec) -> GgmlType:
        if spec.kind in ("norm", "bias", "sink", "pos", "average"):
            return GgmlType.F32
        t = {"matrix": self.matrix, "embed": self.embed, "output": self.output,
             "expert": self.expert, "router": self.router}[spec.kind]
        be, _ = type_block(t)
        # A row that does not divide into blocks falls back to F16, as GGUF converters do.
        return t if spec.shape[-1] % be == 0 else GgmlType.F16


PLAN_Q8_0 = QuantPlan()
PLAN_Q4_K = QuantPlan(matrix=GgmlType.Q4_K, embed=GgmlType.Q6_K, output=GgmlType.Q6_K)
PLAN_BF16 = QuantPlan(matrix=GgmlType.BF16, embed=GgmlType.BF16, output=GgmlType.BF16, expert=GgmlType.BF16)
PLAN_F32 = QuantPlan(matrix=GgmlType.F32, embed=GgmlType.F32, output=GgmlType.F32, expert=GgmlType.F32)
PLAN_MOE = QuantPlan(matrix=GgmlType.BF16, embed=GgmlType.BF16, output=GgmlType.BF16, expert=GgmlType.MXFP4)


def init_tensor(spec: TensorSpec, seed: int, device="cpu", std: float = 0.02) -> torch.Tensor:
    if spec.kind == "norm":
        return torch.ones(spec.shape, dtype=torch.float32, device=device)
    if spec.kind == "bias":
        return torch.zeros(spec.shape, dtype=torch.float32, device=device)
    if spec.kind == "average":             # the latest result, and a little of the others
        w = torch.full(spec.shape, 0.1 / spec.shape[0], dtype=torch.float32, device=device)
        w[-1] += 0.9
        return w
    g = torch.Generator(device=device)
    g.manual_seed((seed * 1000003 + zlib.crc32(spec.name.encode())) & 0x7FFFFFFF)
    return torch.randn(spec.shape, generator=g, dtype=torch.float32, device=device) * std


def random_weights(cfg: ModelConfig, seed: int = 0) -> dict[str, torch.Tensor]:
    return {s.name: init_tensor(s, seed) for s in tensor_specs(cfg)}


def save_gguf(path: str, cfg: ModelConfig, weights: dict[str, torch.Tensor], plan: QuantPlan = PLAN_Q8_0,
              extra_meta: dict | None = None):
    w = GGUFWriter(path)
    for k, v in cfg.to_gguf_metadata().items():
        w.add_meta(k, v)
    w.add_meta("general.file_type", int(plan.matrix))
    for k, v in (extra_meta or {}).items():
        w.add_meta(k, v)
    for spec in tensor_specs(cfg):
        x = weights[spec.name].detach().to(torch.float32).cpu().numpy()
        w.add_tensor(spec.name, x, plan.type_for(spec))
    w.write()


def load_gguf_float(path: str) -> tuple[ModelConfig, dict[str, torch.Tensor]]:
    """Load and dequantize every tensor to fp32 (CPU backend and oracle)."""
    with GGUFFile(path) as f:
        cfg = ModelConfig.from_gguf_metadata(f.metadata)
        W = {n: torch.from_numpy(t.to_float().copy()) for n, t in f.tensors.items()}
    return cfg, W
