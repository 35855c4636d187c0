"""Kazolorn on the host: configuration, checkpoint folders, and the plain implementation itself."""
import json

import pytest
import torch

import kazolorn_ref as R
from openagents_b200.models.checkpoint_dir import CheckpointDirSource
from openagents_b200.models.config import PRESETS, ExpertSpec, MixerSpec, ModelConfig, config_from_json, hybrid_to_json, kazolorn_stack
from openagents_b200.models.hybrid_engine import HybridEngine
from openagents_b200.models.weights import random_weights, tensor_specs

CFG = R.config([R.layer(40, 6, 2, 24, ff=100), R.layer(24, 4, 4, 7, ff=36, experts=5, top=2), R.layer(16, 3, 1, 9, scale=0.4)], width=100, vocab=131)


# ---------------------------------------------------------------- configuration and registry
def test_configuration_is_read_layer_by_layer():
    c = config_from_json(CFG)
    a, b, s = (x.mixer for x in c.layers)
    assert (c.arch, c.n_layers, c.d_model, c.vocab, c.norm_eps, c.norm) == ("kazolorn", 3, 100, 131, 1e-5, "rms1")
    assert (c.walk, c.layer_scale, c.depth_average, c.post_norm, c.has_state) == ("parallel", True, True, False, False)
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale) == ("attention", 6, 2, 40, 40, 24, 40 ** -0.5)
    assert a.tied_kv and a.bias and a.out_bias and a.distance_bias and a.mix_heads and a.silent_sink and not a.rope_dims
    assert (b.window, s.window, s.scale) == (7, 9, 0.4)
    assert [(x.ffn, x.act, x.moe) for x in c.layers] == [(100, "polynorm", None), (36, "swiglu", ExpertSpec(5, 2)), (0, "polynorm", None)]
    assert config_from_json(hybrid_to_json(c)) == c and ModelConfig.from_gguf_metadata(c.to_gguf_metadata()) == c


@pytest.mark.parametrize("path,value", [
    (("architecture",), "Other"), (("layers",), []), (("width",), "72"), (("norm",), {}), (("layers", 0, "type"), "gla"), (("layers", 0, "mixer", "mask"), None),
    (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "mask", "size"), True), (("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "kv_heads"), 0),
    (("layers", 0, "mixer", "scale"), None), (("layers", 0, "mixer", "vdim"), 24), (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "mlp", "kind"), "other"),
    (("layers", 0, "mlp", "ff"), None), (("layers", 0, "mlp", "ff"), 0), (("layers", 1, "mlp", "router"), None), (("layers", 1, "mlp", "router", "top"), 6),
    (("layers", 1, "mlp", "router", "top"), 0), (("layers", 1, "mlp", "router", "experts"), 1.5), (("layers", 1, "mlp", "expert"), 36)])
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
    MixerSpec(**ok, window=5, tied_kv=True, mix_heads=True)
    for bad in (dict(window=5, chunk=5), dict(window=-1), dict(tied_kv=True, kv_from=0), dict(mix_heads=True), dict(tied_kv=True, mix_heads=True, head_gate=True),
                dict(tied_kv=True, mix_heads=True, rope_dims=4)):
        with pytest.raises(ValueError):
            MixerSpec(**ok, **bad)
    with pytest.raises(ValueError):
        MixerSpec("attention", 4, 16, 24, kv_heads=2, tied_kv=True)


def test_registry_picks_engine_and_source(tmp_path):
    from openagents_b200.models.registry import build_engine, engine_class, open_source, peek_architecture
    from openagents_b200.serve.backend import open_backend
    folder = R.save_model(str(tmp_path / "m"), CFG, R.random_weights(CFG))
    src = open_source(folder, "cpu")
    assert peek_architecture(folder) == "kazolorn" and engine_class(src.cfg) is HybridEngine and "kazolorn" in HybridEngine.ARCHS
    with pytest.raises(ValueError, match="cuda backend only"):
        open_backend(folder, "cpu")
    with pytest.raises(ValueError, match="one GPU"):
        build_engine(src, "cpu", 1, 64, tp_world=2)


def test_presets_and_inventory():
    for name in ("kazolorn-8b-shape", "kazolorn-moe-shape"):
        c = PRESETS[name]
        specs = {s.name: s for s in tensor_specs(c)}
        assert c.n_params() == sum(torch.Size(s.shape).numel() for s in specs.values())
        assert config_from_json(hybrid_to_json(c), name=name).with_(ffn=c.ffn) == c
    small = kazolorn_stack(64, 96, 300, 4, 4, 2, 32, 48, "x", experts=6, top=3, expert_ffn=40, dense=2)
    assert [l.moe for l in small.layers] == [None, None, ExpertSpec(6, 3), ExpertSpec(6, 3)] and [l.ffn for l in small.layers] == [96, 96, 40, 40]
    W = random_weights(small)
    assert all(abs(float(W[f"l{i}.dwa"].sum()) - 1.0) < 1e-6 and W[f"l{i}.dwa"].numel() == i + 2 for i in range(4))


# ---------------------------------------------------------------- checkpoint folders
def test_checkpoint_folder_round_trip(tmp_path):
    W = R.random_weights(CFG)
    src = CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, W), "cpu")
    assert set(W) == {s.name for s in tensor_specs(src.cfg)}
    for name, w in W.items():
        assert src.has(name) and torch.equal(src.get(name).to_float().double(), w)


def test_missing_and_misshapen_tensors_are_named(tmp_path):
    W = R.random_weights(CFG)
    for bad, msg in ((lambda w: w.pop("l0.mix.talk"), "l0.mix.talk"), (lambda w: w.pop("l1.mlp.e4.down"), "l1.mlp.e4.down"), (lambda w: w.pop("l2.ls1"), "l2.ls1"),
                     (lambda w: w.update({"l0.mix.o.b": torch.ones(3)}), "l0.mix.o.b"), (lambda w: w.update({"l1.dwa": torch.ones(2)}), "l1.dwa"),
                     (lambda w: w.update({"l0.mlp.act": torch.ones(3)}), "l0.mlp.act")):
        V = dict(W)
        bad(V)
        with pytest.raises(ValueError, match=msg):
            CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, V), "cpu")


# ---------------------------------------------------------------- the plain implementation against itself
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
    assert R.slopes(4).tolist() == [0.25, 0.0625, 0.015625, 0.00390625] and R.slopes(3)[2] == 2.0 ** -8
    assert R.visible(4, 2, 7, 3).int().tolist() == [[0, 0, 1, 1, 1, 0, 0], [0, 0, 0, 1, 1, 1, 0]]
    p = R.weights_with_silent_sink(torch.zeros(1, 1, 3, dtype=torch.float64), torch.tensor([[True, True, False]]))
    assert torch.allclose(p[0, 0], t(1 / 3, 1 / 3, 0.0))       # the sink weighs as much as either key
    p = R.weights_with_silent_sink(torch.full((1, 1, 1), -900.0, dtype=torch.float64), torch.tensor([[True]]))
    assert p.item() == 0.0
    s = torch.zeros(2, 1, 2, dtype=torch.float64)
    s[1, 0, 1] = 3.0
    assert torch.allclose(R.talk(s, t(1.0, 2.0, 0.0, 1.0).view(2, 2))[:, 0, 1], t(6.0, 3.0))
    assert torch.allclose(R.distance_bias(torch.zeros(2, 1, 3, dtype=torch.float64), 2)[:, 0], torch.outer(-R.slopes(2), t(2.0, 1.0, 0.0)))
    z = t(1.0, -2.0)
    want = 2.0 * z / t(2.5).sqrt() + 3.0 * z ** 2 / t(8.5).sqrt() - z ** 3 / t(32.5).sqrt() + 0.5
    assert torch.allclose(R.poly_norm(z, t(2.0, 3.0, -1.0, 0.5), 0.0), want)
    e, w = R.route(t(1.0, 0.0).view(1, 2), t(0.0, 0.0, 3.0, 0.0, -1.0, 5.0).view(3, 2), 2)
    assert e.tolist() == [[1, 0]] and torch.allclose(w[0], torch.sigmoid(t(3.0, 0.0)))
    W = {"e0.gate": t(1.0).view(1, 1), "e0.up": t(2.0).view(1, 1), "e0.down": t(3.0).view(1, 1), "router": t(0.7).view(1, 1)}
    h, s = 1.5, torch.sigmoid(t(1.05)).item()
    g = s * h                                                  # the weight goes in with the token, so the result is not linear in it
    assert R.expert_ff(t(h).view(1, 1), W, "", 1).item() == pytest.approx(3.0 * g / (1 + torch.exp(t(-g)).item()) * 2.0 * g)
    assert torch.equal(R.depth_average([t(1.0), t(10.0)], t(2.0, 0.5)), t(7.0))
    o = R.attention(torch.zeros(1, 2, 4, dtype=torch.float64), torch.ones(3, 1, 4, dtype=torch.float64), torch.zeros(2, 2, dtype=torch.float64), 1.0, 2, 2)
    assert torch.allclose(o, torch.full((1, 2, 4), 2 / 3, dtype=torch.float64))       # two keys in the window, one silent
