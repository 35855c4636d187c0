"""Pesorax on the host: configuration, checkpoint folders, the layout of mixed batches, and the plain implementation itself."""
import json

import pytest
import torch

import pesorax_ref as R
from openagents_b200.models.checkpoint_dir import CheckpointDirSource
from openagents_b200.models.config import PRESETS, ModelConfig, config_from_json, hybrid_to_json, pesorax_stack
from openagents_b200.models.hybrid_engine import SHORT_TOKENS, HybridEngine, plan_latent_batch
from openagents_b200.models.weights import tensor_specs

CFG = R.config([R.layer_attention(40, 24, 6, 2, 24, ff=100), R.layer_latent(24, 10, 40, 3, 36, 20, base=500.0, ff=36), R.layer_attention(16, 56, 3, 1, 7, diff=0.1)],
               width=100, vocab=131, loop=(1, 3, 3))


# ---------------------------------------------------------------- configuration and registry
def test_configuration_is_read_layer_by_layer():
    c = config_from_json(CFG)
    a, l, s = (x.mixer for x in c.layers)
    assert c.arch == "pesorax" and (c.n_layers, c.d_model, c.vocab, c.norm_eps, c.norm, c.post_norm) == (3, 100, 131, 1e-5, "dyt", False)
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.chunk, a.diff, a.bias, a.rope_dims) == ("attention", 6, 2, 40, 24, 2, 24, 0.4, True, 0)
    assert (l.kind, l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.q_rank) == ("latent", 3, 24, 10, 40, 36, 20)
    assert (l.rope_base, l.rope_dims, l.rope_style, l.sink, l.out_gate) == (500.0, 10, "half", True, True)
    assert s.chunk == 7 and s.diff == 0.1 and [x.ffn for x in c.layers] == [100, 36, 0] and c.layers[0].act == "gelu"
    assert c.loop == (1, 3, 3) and c.residual_mult == 0.6 and not c.has_state
    assert config_from_json(hybrid_to_json(c)) == c and ModelConfig.from_gguf_metadata(c.to_gguf_metadata()) == c
    plain = json.loads(json.dumps(CFG))
    del plain["loop"], plain["layers"][1]["mixer"]["q_rank"]
    plain["layers"][2]["mixer"]["mask"] = None
    p = config_from_json(plain, {1: 44})
    assert p.loop is None and p.layers[1].mixer.q_rank == 44 and p.layers[2].mixer.chunk == 0 and config_from_json(hybrid_to_json(p)) == p


def test_layer_runs_follow_the_loop():
    for loop in (None, (0, 3, 2), (1, 3, 3), (2, 3, 1), (0, 1, 4)):
        c = dict(CFG, loop=None if loop is None else dict(zip(("start", "stop", "times"), loop)))
        assert config_from_json(c).layer_runs() == R.order(c)
    assert config_from_json(CFG).layer_runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False)]


@pytest.mark.parametrize("path,value", [
    (("architecture",), "Other"), (("layers",), []), (("width",), "72"), (("norm",), {}), (("residual_mult",), "1"), (("loop", "stop"), 4), (("loop", "start"), 3),
    (("loop", "times"), 0), (("loop", "start"), -1), (("loop",), 2), (("layers", 0, "type"), "gla"), (("layers", 0, "mixer", "mask", "size"), 0),
    (("layers", 0, "mixer", "mask"), 3), (("layers", 0, "mixer", "diff"), None), (("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "scale"), None),
    (("layers", 1, "mixer", "rot"), None), (("layers", 1, "mixer", "rot", "dims"), 12), (("layers", 1, "mixer", "rot", "dims"), 5), (("layers", 1, "mixer", "kv_rank"), 0),
    (("layers", 1, "mixer", "q_rank"), None), (("layers", 1, "mixer", "rot_dim"), True), (("layers", 1, "mlp", "kind"), "moe"), (("layers", 1, "mlp", "ff"), None)])
def test_a_bad_configuration_is_refused(path, value):
    c = json.loads(json.dumps(CFG))
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ValueError):
        config_from_json(c)


def test_registry_picks_engine_and_source(tmp_path):
    from openagents_b200.models.registry import build_engine, engine_class, open_source, peek_architecture
    from openagents_b200.serve.backend import open_backend
    folder = R.save_model(str(tmp_path / "m"), CFG, R.random_weights(CFG))
    src = open_source(folder, "cpu")
    assert peek_architecture(folder) == "pesorax" and engine_class(src.cfg) is HybridEngine and "pesorax" in HybridEngine.ARCHS
    with pytest.raises(ValueError, match="cuda backend only"):
        open_backend(folder, "cpu")
    with pytest.raises(ValueError, match="one GPU"):
        build_engine(src, "cpu", 1, 64, tp_world=2)


def test_presets_and_inventory():
    for name in ("pesorax-8b-shape", "pesorax-1b-shape"):
        c = PRESETS[name]
        specs = {s.name: s for s in tensor_specs(c)}
        assert c.n_params() == sum(torch.Size(s.shape).numel() for s in specs.values())
        assert config_from_json(hybrid_to_json(c), name=name) == c
    small = pesorax_stack(64, 96, 300, 2, 4, 2, 32, 48, 64, 3, 24, 8, 16, 40, 20, "x", loop=(2, 5, 2))
    assert [l.mixer.kind for l in small.layers] == ["attention"] * 3 + ["latent"] + ["attention"] * 3 + ["latent"] and len(small.layer_runs()) == 11


# ---------------------------------------------------------------- checkpoint folders
def test_checkpoint_folder_round_trip(tmp_path):
    W = R.random_weights(CFG)
    src = CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, W), "cpu")
    assert set(W) == {s.name for s in tensor_specs(src.cfg)}
    for name, w in W.items():                       # numbers without an axis come as vectors of one
        assert src.has(name) and torch.equal(src.get(name).to_float().double(), w.reshape(w.shape or (1,)))
    slim = json.loads(json.dumps(CFG))
    del slim["layers"][1]["mixer"]["q_rank"]        # a size that the tensor's shape gives
    assert CheckpointDirSource(R.save_model(str(tmp_path / "n"), slim, W), "cpu").cfg.layers == src.cfg.layers


def test_missing_and_misshapen_tensors_are_named(tmp_path):
    W = R.random_weights(CFG)
    for bad, msg in ((lambda w: w.pop("l1.mix.sink"), "l1.mix.sink"), (lambda w: w.pop("l0.norm2.alpha"), "l0.norm2.alpha"),
                     (lambda w: w.update({"l0.mix.q.b": torch.ones(3)}), "l0.mix.q.b"), (lambda w: w.update({"final.norm.alpha": torch.ones(2)}), "final.norm.alpha")):
        V = dict(W)
        bad(V)
        with pytest.raises(ValueError, match=msg):
            CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, V), "cpu")


# ---------------------------------------------------------------- layout of mixed batches
def test_short_entries_come_first_and_the_rest_fits_the_workspace():
    g = torch.Generator().manual_seed(0)
    for _ in range(300):
        B = int(torch.randint(1, 9, (1,), generator=g))
        q = sorted(int(x) for x in torch.randint(1, 60, (B,), generator=g))
        ctx = [n + int(torch.randint(0, 100, (1,), generator=g)) for n in q]
        p, rows, base = plan_latent_batch(q, ctx, 40, 170)
        assert p.t_short == sum(q[: p.n_short]) <= 40 and all(n <= SHORT_TOKENS for n in q[: p.n_short])
        assert rows == [b for b in range(p.n_short) for _ in range(q[b])]
        assert all(c <= p.short_pages * 16 for c in ctx[: p.n_short])
        at = p.n_short
        for lo, hi, group_q, group_ctx, n in p.groups:
            assert lo == at and hi > lo and n == sum(ctx[lo:hi]) <= 170
            assert group_q == max(q[lo:hi]) and group_ctx == max(ctx[lo:hi])
            assert base[lo:hi] == [sum(ctx[lo:b]) for b in range(lo, hi)]
            at = hi
        assert at == B


def test_batch_order_is_stable_and_only_where_needed():
    e = HybridEngine.__new__(HybridEngine)
    e.ctx_rows = 128
    assert e._batch_order([1, 1, 1]) is None and e._batch_order([1, 5, 9]) is None
    assert e._batch_order([30, 1, 4, 1]) == [1, 3, 2, 0]
    e.ctx_rows = 0                                  # no latent layers
    assert e._batch_order([30, 1]) is None


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
    W = {"n": t(2.0, 1.0), "n.b": t(0.5, 0.0), "n.alpha": torch.tensor(2.0, dtype=torch.float64)}
    assert torch.allclose(R.dyt(t(1.0, -0.5), W, "n"), t(2 * torch.tanh(t(2.0)).item() + 0.5, -torch.tanh(t(1.0)).item()))
    r = R.rotate_half(t(1.0, 0.0, 0.0, 1.0, 5.0).view(1, 1, 5), torch.tensor([2]), 4, 100.0)[0, 0]
    a, b = t(2.0), t(0.2)
    assert torch.allclose(r, torch.cat([a.cos(), -b.sin(), a.sin(), b.cos(), t(5.0)]))
    ok = R.visible(4, 3, 8, chunk=3)                           # positions 4, 5, 6 in chunks [3, 5] and [6, 8]
    assert ok.int().tolist() == [[0, 0, 0, 1, 1, 0, 0, 0], [0, 0, 0, 1, 1, 1, 0, 0], [0, 0, 0, 0, 0, 0, 1, 0]]
    w = R.weights_over_keys(torch.zeros(1, 1, 3, dtype=torch.float64), torch.tensor([[True, True, False]]), t(torch.log(t(2.0)).item()))
    assert torch.allclose(w[0, 0], t(0.25, 0.25, 0.0))         # the sink weighs as much as both keys
    L = {"lq1": t(1.0, 0.0), "lk1": t(0.5, 9.0), "lq2": t(0.0, 1.0), "lk2": t(9.0, 0.25)}
    assert R.lambda_of(L, "", 0.3).item() == pytest.approx(2.718281828 ** 0.5 - 2.718281828 ** 0.25 + 0.3)
    q, k, v = torch.zeros(1, 2, 2, 4, dtype=torch.float64), torch.zeros(2, 1, 2, 4, dtype=torch.float64), t(1.0, 3.0).view(2, 1, 1)
    q[0, 1, 1, 0], k[1, 0, 1, 0] = 50.0, 1.0                   # head 1's second map looks at key 1 only
    a1, a2 = R.differential_attention(q, k, v, 1.0, 0, 1)
    assert a1[0, :, 0].tolist() == pytest.approx([2.0, 2.0]) and a2[0, :, 0].tolist() == pytest.approx([2.0, 3.0])
