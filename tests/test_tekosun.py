"""Tekosun on the host: configuration, checkpoint folders, and the plain implementation itself."""
import json
import math

import pytest
import torch

import tekosun_ref as R
from openagents_b200.models.checkpoint_dir import CheckpointDirSource
from openagents_b200.models.config import PRESETS, ExpertSpec, MixerSpec, ModelConfig, config_from_json, hybrid_to_json, tekosun_stack
from openagents_b200.models.hybrid_engine import HybridEngine
from openagents_b200.models.weights import random_weights, tensor_specs

CFG = R.config([R.layer_delta(24, 3, R.moe(40, 6, 2, 2.5, 56)), R.layer_mamba(6, 20, 12, 3, 4, 3, R.moe(16, 3, 3, shared=0)),
                R.layer_attention(40, 24, 6, 2, 16, 9, 5000.0, (4.0, 1.0, 3.0, 64), 0.3), R.layer_attention(16, 24, 4, 2, 0, v_mix=False), R.layer_attention(16, 24, 2, 2, 8)],
               width=100, vocab=131, scale=3.0)


# ---------------------------------------------------------------- configuration and registry
def test_configuration_is_read_layer_by_layer():
    c = config_from_json(CFG, {0: 8})
    d, s, a, b, e = (x.mixer for x in c.layers)
    assert (c.arch, c.n_layers, c.d_model, c.vocab, c.norm_eps, c.norm) == ("tekosun", 5, 100, 131, 1e-5, "rms1")
    assert (c.walk, c.pre_norm, c.post_norm, c.has_state, c.embed_scale) == ("serial", False, True, True, 3.0)
    assert (d.kind, d.heads, d.dim, d.vdim, d.rank, d.log_decay) == ("delta", 3, 24, 24, 8, math.exp(-0.5))
    assert (s.kind, s.heads, s.vdim, s.dim, s.groups, s.norm_groups, s.conv, s.channels) == ("ssd", 6, 20, 12, 3, 4, 3, 6 * 20 + 2 * 3 * 12)
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale) == ("attention", 6, 2, 40, 24, 9, 0.3)
    assert (a.rope_dims, a.rope_base, a.rope_style, a.rope_scaling) == (16, 5000.0, "half", (4.0, 1.0, 3.0, 64.0))
    assert (a.row_norm, a.v_norm, a.v_mix, b.v_mix, e.v_mix, b.window, b.rope_dims) == (True, True, True, False, True, 0, 0)
    assert [(x.ffn, x.act, x.moe) for x in c.layers[:3]] == [(40, "relu2", ExpertSpec(6, 2, "softmax", 2.5, "output", 56)),
                                                             (16, "relu2", ExpertSpec(3, 3, "softmax", 1.0, "output", 0)), (0, "relu2", None)]
    assert config_from_json(hybrid_to_json(c)) == c and ModelConfig.from_gguf_metadata(c.to_gguf_metadata()) == c


@pytest.mark.parametrize("path,value", [
    (("architecture",), "Other"), (("layers",), []), (("width",), "72"), (("norm",), {}), (("embedding", "scale"), "2"), (("layers", 0, "type"), "gla"),
    (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "mixer", "heads"), None), (("layers", 1, "mixer", "groups"), 4), (("layers", 1, "mixer", "norm_groups"), 7),
    (("layers", 1, "mixer", "conv"), 0), (("layers", 1, "mixer", "state"), None), (("layers", 2, "mixer", "mask", "size"), 0), (("layers", 2, "mixer", "mask", "size"), True),
    (("layers", 2, "mixer", "kv_heads"), 4), (("layers", 2, "mixer", "scale"), None), (("layers", 2, "mixer", "rot", "dims"), 42), (("layers", 2, "mixer", "rot", "dims"), 7),
    (("layers", 2, "mixer", "rot", "scaling", "high"), 0.5), (("layers", 2, "mixer", "rot", "scaling", "factor"), None), (("layers", 2, "mixer", "v_mix"), 1),
    (("layers", 4, "mixer", "vdim"), 16), (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mlp", "expert"), 3), (("layers", 0, "mlp", "router", "top"), 7),
    (("layers", 0, "mlp", "router", "top"), 0), (("layers", 0, "mlp", "shared", "ff"), 0)])
def test_a_bad_configuration_is_refused(path, value):
    c = json.loads(json.dumps(CFG))
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ValueError):
        config_from_json(c)


def test_mixers_that_do_not_fit_together_are_refused():
    ok = dict(kind="attention", heads=4, dim=16, vdim=16, kv_heads=2)
    MixerSpec(**ok, row_norm=True, v_norm=True, v_mix=True, window=5)
    for bad in (dict(row_norm=True, qk_norm=True), dict(v_mix=True, kv_from=0), dict(v_norm=True, tied_kv=True), dict(rope_scaling=(2.0, 1.0, 4.0, 32.0)),
                dict(row_norm=True, bias=True)):
        with pytest.raises(ValueError):
            MixerSpec(**ok, **bad)
    with pytest.raises(ValueError):
        MixerSpec("delta", 2, 16, 16)
    with pytest.raises(ValueError):
        ExpertSpec(4, 2, "other")


def test_registry_picks_engine_and_source(tmp_path):
    from openagents_b200.models.registry import build_engine, engine_class, open_source, peek_architecture
    from openagents_b200.serve.backend import open_backend
    folder = R.save_model(str(tmp_path / "m"), CFG, R.random_weights(CFG))
    src = open_source(folder, "cpu")
    assert peek_architecture(folder) == "tekosun" and engine_class(src.cfg) is HybridEngine and "tekosun" in HybridEngine.ARCHS
    assert src.cfg.layers[0].mixer.rank == 8           # from the tensor's shape
    with pytest.raises(ValueError, match="cuda backend only"):
        open_backend(folder, "cpu")
    with pytest.raises(ValueError, match="one GPU"):
        build_engine(src, "cpu", 1, 64, tp_world=2)


def test_presets_and_inventory():
    for name in ("tekosun-8b-shape", "tekosun-1b-shape"):
        c = PRESETS[name]
        specs = {s.name: s for s in tensor_specs(c)}
        assert c.n_params() == sum(torch.Size(s.shape).numel() for s in specs.values())
        assert config_from_json(hybrid_to_json(c), name=name) == c
    small = tekosun_stack(64, 300, 1, 4, 2, 32, 48, 2, 24, 8, 4, 16, 24, 6, 2, 40, 56, "x")
    assert [l.mixer.kind for l in small.layers] == ["delta", "attention", "delta", "ssd"]
    assert set(random_weights(small)) == {s.name for s in tensor_specs(small)}


# ---------------------------------------------------------------- checkpoint folders
def test_checkpoint_folder_round_trip(tmp_path):
    W = R.random_weights(CFG)
    src = CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, W), "cpu")
    assert set(W) == {s.name for s in tensor_specs(src.cfg)}
    for name, w in W.items():
        assert src.has(name) and torch.equal(src.get(name).to_float().double().view(w.shape), w)


def test_missing_and_misshapen_tensors_are_named(tmp_path):
    W = R.random_weights(CFG)
    for bad, msg in ((lambda w: w.pop("l0.mix.w0"), "l0.mix.w0"), (lambda w: w.pop("l0.mlp.shared.up"), "l0.mlp.shared.up"), (lambda w: w.pop("l2.mix.k.norm"), "l2.mix.k.norm"),
                     (lambda w: w.pop("l4.mix.vmix"), "l4.mix.vmix"), (lambda w: w.update({"l1.mix.conv": torch.ones(192, 4)}), "l1.mix.conv"),
                     (lambda w: w.update({"l1.mix.A_log": torch.ones(3)}), "l1.mix.A_log"), (lambda w: w.update({"l0.mix.w2": torch.ones(72, 9)}), "l0.mix.w2")):
        V = dict(W)
        bad(V)
        with pytest.raises(ValueError, match=msg):
            CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, V), "cpu")


# ---------------------------------------------------------------- the plain implementation against itself, and by hand
def test_reference_portions_equal_the_whole():
    W = R.random_weights(CFG, seed=1)
    toks = torch.randint(0, 131, (40,), generator=torch.Generator().manual_seed(0)).tolist()
    whole = R.forward(CFG, W, toks, R.Sequence())
    for cuts in ([1] * 40, [2, 17, 21], [39, 1]):
        seq, rows, at = R.Sequence(), [], 0
        for n in cuts:
            rows.append(R.forward(CFG, W, toks[at: at + n], seq))
            at += n
        assert (torch.cat(rows) - whole).abs().max() < 1e-9


def test_reference_mechanisms_by_hand():
    t = lambda *v: torch.tensor(v, dtype=torch.float64)        # noqa: E731
    S = t(1.0, 2.0).view(1, 2, 1)                               # one head, two key channels, one value column
    k = t(3.0, 0.0).view(1, 2)
    u = R.unit_key(k)
    assert torch.allclose(u, t(3.0 / math.sqrt(9.0 + 1e-6), 0.0).view(1, 2))
    new = R.delta_step(S, t(0.5, 1.0).view(1, 2), t(0.25, 0.75).view(1, 2), k, t(10.0).view(1, 1))
    assert torch.allclose(new[0, :, 0], t(0.5 - 0.25 + 30.0, 2.0), atol=1e-5)       # decayed, less a quarter of what the key read, plus the product
    assert torch.allclose(R.delta_decay(torch.zeros(1, 1, dtype=torch.float64), t(1.0).view(1, 1), t(1.0).view(1, 1), t(0.0)), torch.exp(t(-0.5 * math.exp(-0.5))))
    y, last = R.causal_conv(t(1.0, 10.0, 100.0).view(3, 1), t(7.0, 5.0).view(2, 1), t(1.0, 2.0, 3.0).view(1, 3), t(0.5))
    assert torch.allclose(y[:, 0], t(7.0 + 10.0 + 3.0, 5.0 + 2.0 + 30.0, 1.0 + 20.0 + 300.0) + 0.5) and last[:, 0].tolist() == [10.0, 100.0]
    y, S = R.ssd(t(4.0).view(1, 1, 1), t(3.0).view(1, 1, 1), t(2.0).view(1, 1, 1), t(0.5).view(1, 1), t(math.log(2.0)), t(10.0), t(6.0).view(1, 1, 1))
    assert torch.allclose(S, 6.0 * torch.exp(t(-1.0)) + 0.5 * 12.0) and torch.allclose(y, 2.0 * S + 40.0)
    assert torch.allclose(R.group_rms_norm(t(3.0, 3.0, 1.0, 7.0), t(1.0, 1.0, 2.0, 1.0), 2, 0.0), t(1.0, 1.0, 0.4, 1.4))
    f = R.frequencies(8, 100.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 40.0})
    base = [100.0 ** (-i / 4) for i in range(4)]
    turns = [40.0 * b / (2 * math.pi) for b in base]           # 6.4, 2.0, 0.64, 0.2
    s = (turns[1] - 1.0) / 3.0
    assert f[0] == base[0] and f[2:] == [base[2] / 8, base[3] / 8] and f[1] == pytest.approx((1 - s) * base[1] / 8 + s * base[1])
    m = MixerSpec("attention", 1, 8, 8, kv_heads=1, rope_base=100.0, rope_dims=8, row_norm=True, rope_scaling=(8.0, 1.0, 4.0, 40.0))
    assert m.rope_frequencies() == pytest.approx(f)
    x = R.rotate(t(1.0, 0.0, 0.0, 5.0).view(1, 1, 4), [2], {"base": 10.0, "dims": 2})
    assert torch.allclose(x[0, 0], torch.cat([torch.cos(t(2.0)), torch.sin(t(2.0)), t(0.0, 5.0)]))
    assert R.visible(4, 2, 7, 3).int().tolist() == [[0, 0, 1, 1, 1, 0, 0], [0, 0, 0, 1, 1, 1, 0]]
    assert R.visible(1, 1, 3, 0).int().tolist() == [[1, 1, 0]]
    e, w = R.route(t(1.0).view(1, 1), t(0.0, 1.0, 3.0).view(3, 1), 2, 2.0)
    assert e.tolist() == [[2, 1]] and torch.allclose(w[0], 2.0 * torch.softmax(t(3.0, 1.0), 0))
    assert torch.allclose(R.relu2_ff(t(2.0).view(1, 1), {"up": t(-1.0, 3.0).view(2, 1), "down": t(5.0, 1.0).view(1, 2)}, ""), t(36.0).view(1, 1))
