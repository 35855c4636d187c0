"""Folirax on the host: configuration, checkpoint folders, state slots, the trace protocol, and the plain implementation itself."""
import json
import os
import struct

import pytest
import torch

import folirax_ref as R
from openagents_b200.models.checkpoint_dir import CheckpointDirSource, SafetensorsFile
from openagents_b200.models.config import PRESETS, ModelConfig, config_from_json, folirax_stack, hybrid_to_json
from openagents_b200.models.paged import KVPool
from openagents_b200.models.weights import PLAN_BF16, tensor_specs

CFG = R.config([R.layer_gla(24, 40, 3, tau=8.0, ff=36), R.layer_attention(40, 24, 6, 2, 16, ff=100), R.layer_attention(40, 24, 6, 2, 16, kv_from=1, scale=0.3)],
               width=72, vocab=131)


# ---------------------------------------------------------------- configuration and registry
def test_configuration_is_read_layer_by_layer():
    c = config_from_json(CFG, {0: 8})
    g, a, s = (l.mixer for l in c.layers)
    assert c.arch == "folirax" and (c.n_layers, c.d_model, c.vocab, c.norm_eps) == (3, 72, 131, 1e-6)
    assert (g.kind, g.heads, g.dim, g.vdim, g.tau, g.rank) == ("gla", 3, 24, 40, 8.0, 8)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.rope_dims, a.rope_base, a.kv_from) == (6, 2, 40, 24, 16, 10000.0, None)
    assert a.qk_norm and a.head_gate and s.kv_from == 1 and s.scale == 0.3
    assert [l.ffn for l in c.layers] == [36, 100, 0] and (c.logit_scale, c.logit_softcap) == (0.7, 20.0)
    assert c.has_state and not config_from_json(dict(CFG, layers=[CFG["layers"][1]])).has_state
    assert config_from_json(hybrid_to_json(c)) == c
    plain = json.loads(json.dumps(dict(CFG, logit_scale=None, logit_softcap=None)))
    plain["layers"][1]["mixer"]["rot"] = None
    plain["layers"][2]["mixer"]["rot"] = None
    p = config_from_json(plain)
    assert (p.logit_scale, p.logit_softcap, p.layers[1].mixer.rope_dims) == (1.0, 0.0, 0)
    assert ModelConfig.from_gguf_metadata(c.to_gguf_metadata()) == c


@pytest.mark.parametrize("path,value", [
    (("architecture",), "Other"), (("layers",), []), (("layers",), None), (("width",), "72"), (("norm",), {}), (("logit_scale",), "1"),
    (("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "tau"), 0), (("layers", 1, "mixer", "rot"), 16), (("layers", 1, "mixer", "rot", "dims"), 48),
    (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "dim"), True), (("layers", 1, "mlp", "kind"), "moe"),
    (("layers", 2, "mixer", "kv_from"), 0), (("layers", 2, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_from"), -1), (("layers", 2, "mixer", "vdim"), 16)])
def test_a_bad_configuration_is_refused(path, value):
    c = json.loads(json.dumps(CFG))
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ValueError):
        config_from_json(c)


def test_registry_picks_engine_and_source(tmp_path):
    from openagents_b200.models.hybrid_engine import HybridEngine
    from openagents_b200.models.registry import build_engine, engine_class, open_source, peek_architecture, tokenizer_metadata, weights_file
    from openagents_b200.serve.backend import open_backend
    folder = R.save_model(str(tmp_path / "m"), CFG, R.random_weights(CFG))
    src = open_source(folder, "cpu")
    assert peek_architecture(folder) == "folirax" and engine_class(src.cfg) is HybridEngine
    assert tokenizer_metadata(folder) == {} and weights_file(folder).endswith("model.safetensors")
    with pytest.raises(ValueError, match="cuda backend only"):
        open_backend(folder, "cpu")
    with pytest.raises(ValueError, match="one GPU"):
        build_engine(src, "cpu", 1, 64, tp_world=2)
    with pytest.raises(ValueError, match="no 32-bit mode"):
        class Llama:
            cfg = PRESETS["tiny-llama"]
        build_engine(Llama, "cpu", 1, 64, dtype="float32")


def test_presets_and_inventory():
    c = PRESETS["folirax-1b-shape"]
    specs = {s.name: s for s in tensor_specs(c)}
    assert c.n_params() == sum(torch.Size(s.shape).numel() for s in specs.values())
    shared = [i for i, l in enumerate(c.layers) if l.mixer.kv_from is not None]
    assert shared and all(c.layers[c.layers[i].mixer.kv_from].mixer.kv_from is None and f"l{i}.mix.k" not in specs for i in shared)
    small = folirax_stack(64, 96, 300, 2, 4, 2, 32, 2, 16, 24, "x", ratio=1)
    assert [l.mixer.kind for l in small.layers] == ["gla", "attention", "attention"] * 2
    assert [l.mixer.kv_from for l in small.layers] == [None, None, 1, None, None, 4]


# ---------------------------------------------------------------- checkpoint folders
def test_checkpoint_folder_round_trip(tmp_path):
    W = R.random_weights(CFG, rank=5)
    src = CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, W), "cpu")
    assert src.cfg.name == "m" and src.cfg.layers[0].mixer.rank == 5        # a size that only the tensor's shape gives
    for name, w in W.items():
        assert src.has(name) and torch.equal(src.get(name).to_float().double(), w)
    cfg2, W2 = R.load(str(tmp_path / "m"))
    assert cfg2 == CFG and all(torch.equal(W[k], W2[k]) for k in W)


def test_missing_and_misshapen_tensors_are_named(tmp_path):
    W = R.random_weights(CFG)
    for bad, msg in ((lambda w: w.pop("l1.mix.v"), "l1.mix.v"), (lambda w: w.update({"l0.mix.norm": torch.ones(3)}), "l0.mix.norm")):
        V = dict(W)
        bad(V)
        with pytest.raises(ValueError, match=msg):
            CheckpointDirSource(R.save_model(str(tmp_path / "m"), CFG, V), "cpu")


def test_damaged_safetensors_files_are_refused(tmp_path):
    p = str(tmp_path / "t.safetensors")
    R.write_safetensors(p, {"a": torch.ones(3, 4), "t": torch.arange(5)})
    f = SafetensorsFile(p)
    assert torch.equal(f.tensor("t"), torch.arange(5, dtype=torch.int32)) and f.tensor("a").shape == (3, 4)
    good = open(p, "rb").read()
    n = struct.unpack("<Q", good[:8])[0]
    header = json.loads(good[8: 8 + n])

    def with_header(h):
        b = json.dumps(h).encode() if not isinstance(h, bytes) else h
        return struct.pack("<Q", len(b)) + b + good[8 + n:]
    bad = [b"", b"1234", struct.pack("<Q", 1 << 40) + good[8:], good[: 8 + n // 2], with_header(b"{not json"), with_header([1]), good[:-4]]
    for key, v in (("dtype", "F64"), ("shape", [3, 5]), ("shape", [-3, -4]), ("data_offsets", [0, 1 << 30]), ("data_offsets", [8, 0]), ("data_offsets", [1]), ("shape", None)):
        bad.append(with_header({**header, "a": {**header["a"], key: v}}))
    for i, b in enumerate(bad):
        open(p, "wb").write(b)
        with pytest.raises(ValueError):
            SafetensorsFile(p)
    g = torch.Generator().manual_seed(0)
    for _ in range(300):                            # random damage to the header: an error or a readable file, never a stray view
        b = bytearray(good)
        for _ in range(3):
            b[int(torch.randint(0, 8 + n, (1,), generator=g))] = int(torch.randint(0, 256, (1,), generator=g))
        open(p, "wb").write(bytes(b))
        try:
            f = SafetensorsFile(p)
            for name in f.entries:
                f.tensor(name)
        except ValueError:
            pass


# ---------------------------------------------------------------- state slots in the page pool
def test_state_slots_are_held_from_begin_to_end():
    p = KVPool(8, state_slots=2)
    assert p.begin(1, list(range(40))) == 0 and p.begin(2) == 0 and p.free_slots == 0
    a, b = p.slots([1, 2])
    assert {a, b} == {0, 1} and p.slots([2, 1]) == [b, a]
    with pytest.raises(MemoryError):
        p.begin(3)
    assert p.length(3) == -1                        # nothing was opened
    p.extend(1, 40)
    p.publish(1, list(range(40)))                   # no sharing between sequences with state
    p.end(1)
    assert p.free_slots == 1 and p.free_pages == 8 and p.retained_pages == 0
    assert p.begin(4, list(range(40))) == 0 and p.slots([4]) == [a]
    with pytest.raises(KeyError):
        p.slots([1])
    p.truncate(4, 0)
    assert p.slots([4]) == [a]
    assert KVPool(4).free_slots == 0


def test_slot_accounting_under_random_use():
    g = torch.Generator().manual_seed(3)
    p, live = KVPool(32, state_slots=5), {}
    for step in range(2000):
        seq = int(torch.randint(0, 9, (1,), generator=g))
        if seq in live:
            p.end(seq)
            del live[seq]
        elif len(live) == 5:
            with pytest.raises(MemoryError):
                p.begin(seq)
        else:
            p.begin(seq)
            p.extend(seq, 1 + step % 60)
            live[seq] = p.slots([seq])[0]
        assert len(set(live.values())) == len(live) and p.free_slots == 5 - len(live)
        assert p.slots(list(live)) == list(live.values())


# ---------------------------------------------------------------- trace protocol
class FakeBackend:
    """Logits that name the sequence's own tokens: row i of a sequence is [its length so far, the token]."""

    class cfg:
        vocab = 50

    def __init__(self):
        self.seqs, self.log = {}, []

    def begin(self, seq, prompt):
        assert seq not in self.seqs
        self.seqs[seq] = 0

    def end(self, seq):
        del self.seqs[seq]

    def forward_at(self, seqs, feeds, wants):
        self.log.append((len(seqs), [len(f) for f in feeds]))
        rows = []
        for s, f, want in zip(seqs, feeds, wants):
            rows += [[self.seqs[s] + w, f[w]] for w in want]
            self.seqs[s] += len(f)
        return torch.tensor(rows, dtype=torch.float32).view(-1, 2)


def test_trace_steps_write_what_is_wanted(tmp_path):
    import numpy as np
    from openagents_b200.serve.trace import TraceRunner
    be = FakeBackend()
    r = TraceRunner(be, str(tmp_path))
    r.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}, {"id": "b", "tokens": [7], "want": []}], "end": []})
    r.step({"step": 1, "entries": [{"id": "b", "tokens": [8, 9], "want": []}], "end": ["b"]})
    r.step({"step": 2, "entries": [{"id": "b", "tokens": [5], "want": [0]}, {"id": "a", "tokens": [4], "want": [0]}], "end": ["a", "b", "nobody"]})
    r.step({"step": 3, "entries": [], "end": []})
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, 2).tolist()        # noqa: E731
    assert read(0) == [[2, 3], [0, 1]] and read(2) == [[0, 5], [3, 4]]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32"] and be.seqs == {}
    assert be.log == [(2, [3, 1]), (1, [2]), (2, [1, 1])]


@pytest.mark.parametrize("entry", [{"id": "a", "tokens": [], "want": []}, {"id": "a", "tokens": [50], "want": []}, {"id": "a", "tokens": [-1], "want": []},
                                   {"id": "a", "tokens": [1], "want": [1]}])
def test_trace_refuses_bad_steps(tmp_path, entry):
    from openagents_b200.serve.trace import TraceRunner
    with pytest.raises(ValueError):
        TraceRunner(FakeBackend(), str(tmp_path)).step({"step": 0, "entries": [entry], "end": []})


def test_library_subset_stands_on_its_own():
    """The sources a fresh tree compiles for this family: the page pool, and every kernel file its ops call into."""
    from openagents_b200 import _build
    sub = _build.SUBSETS["hybrid"]
    host, cuda = _build._subset(_build.host_sources(), "host", "hybrid"), _build._subset(_build.cuda_sources(), "cuda", "hybrid")
    assert len(host) == len(sub["host"]) and len(cuda) == len(sub["cuda"])
    text = "".join(p.read_text() for p in cuda)
    import re
    eng = open(os.path.join(os.path.dirname(_build.__file__), "models", "hybrid_engine.py")).read()
    for op in set(re.findall(r"ops\.([a-z_0-9]+)\(", eng)) - {"argmax_scratch", "moe_choose"}:
        assert f"b200_{op}(" in text, op
    for p in (_build.CSRC / n for n in _build.PRECISE):
        assert "--use_fast_math" not in _build._flags_for(p, _build.NVCC_FLAGS)


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
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(R.centred_norm(x, torch.tensor([1.0, 0.0], dtype=torch.float64), 0.0), x / 12.5 ** 0.5 * torch.tensor([2.0, 1.0]))
    r = R.rotate(torch.tensor([[[1.0, 0.0, 0.0, 1.0, 5.0]]], dtype=torch.float64), torch.tensor([2]), 4, 100.0)[0, 0]
    want = torch.tensor([2.0, 2.0, 0.2, 0.2, 0.0], dtype=torch.float64)
    assert torch.allclose(r, torch.stack([want[0].cos(), want[0].sin(), -want[2].sin(), want[2].cos(), torch.tensor(5.0, dtype=torch.float64)]))
    S = torch.full((1, 1, 1), 4.0, dtype=torch.float64)
    q = k = v = torch.tensor([[[2.0]]], dtype=torch.float64)
    o, S1 = R.gla_recurrence(q, k, v, torch.log(torch.tensor([[[0.5]]], dtype=torch.float64)), S)
    assert S1.item() == pytest.approx(0.5 * 4 + 4) and o.item() == pytest.approx(12.0)
    assert PLAN_BF16.type_for(tensor_specs(config_from_json(CFG))[0]).name == "BF16"
