"""Host side of the bf16-weight hybrids, no GPU: configuration, checkpoint files, design registry, request state,
C-ABI declarations, what the drivers pass to the library, engine control flow, trace replay."""

import ctypes
import io
import json
import re
import sys
from pathlib import Path

import pytest
import torch

from quickdraw_b200 import _lib, hybrid, mixers, registry, replay, synthetic
from quickdraw_b200.engine import Engine
from quickdraw_b200.loader import hybrid_shapes, load_hybrid_checkpoint, save_hybrid_checkpoint
from quickdraw_b200.state import DecodeState, HybridState
from quickdraw_b200.weights import FezopelConfig, WindowAttnConfig
from tests import hybrid_cases as cases
from tests.recording import AsIfOnGpu, recorder  # noqa: F401 (a fixture)

ROOT = Path(__file__).resolve().parents[1]
HEADER = ROOT / "include" / "quickdraw_b200_hybrid.h"


# ------------------------------------------------------------------- configuration, files
@pytest.mark.parametrize("name", cases.MODELS)
def test_configuration_round_trip(name):
    cfg = cases.MODELS[name]()
    assert FezopelConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


@pytest.mark.parametrize("change,message", [
    (lambda d: d.update(architecture="Other"), "not a Fezopel"), (lambda d: d["layers"][0].update(type="mamba"), "unknown mixer"),
    (lambda d: d["layers"][1]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "do not divide")])
def test_configuration_refuses_what_it_does_not_know(change, message):
    data = cases.MODELS["mixed"]().to_dict()
    change(data)
    with pytest.raises(ValueError, match=message):
        FezopelConfig.from_dict(data)


def test_checkpoint_round_trip(tmp_path):
    cfg = cases.MODELS["mixed"]()
    tensors = cases.tensors(cfg)
    save_hybrid_checkpoint(cfg, tensors, tmp_path)
    assert registry.design_of_directory(tmp_path).name == "fezopel"
    ckpt = registry.design_of_directory(tmp_path).load(tmp_path, "cpu")
    assert ckpt.config == cfg and registry.design_of(ckpt).name == "fezopel"
    assert torch.equal(ckpt.layers[0].mixer.q_conv, tensors["l0.mix.q.conv"])
    assert torch.equal(ckpt.layers[2].mixer.a2_b, tensors["l2.mix.a2.b"])
    assert torch.equal(ckpt.layers[1].around_mlp.gate_b, tensors["l1.rg2.b"]) and ckpt.layers[0].mlp is None
    assert torch.equal(ckpt.final_norm.b, tensors["final.norm.b"]) and ckpt.layers[4].depth.shape == (6,)
    assert set(hybrid_shapes(cfg)) == set(tensors)


def test_checkpoint_with_a_missing_or_misshapen_tensor_is_refused(tmp_path):
    cfg = cases.MODELS["attention only"]()
    tensors = cases.tensors(cfg)
    save_hybrid_checkpoint(cfg, {k: v for k, v in tensors.items() if k != "l0.mix.sink"}, tmp_path / "a")
    with pytest.raises(ValueError, match="l0.mix.sink is missing"):
        load_hybrid_checkpoint(tmp_path / "a", "cpu")
    save_hybrid_checkpoint(cfg, tensors | {"l0.dwa": tensors["l0.dwa"][:1]}, tmp_path / "b")
    with pytest.raises(ValueError, match="l0.dwa has shape"):
        load_hybrid_checkpoint(tmp_path / "b", "cpu")


def test_registry_tells_the_designs_apart(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"text_config": {}}))
    assert registry.design_of_directory(tmp_path).name == "qwen3-next"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="no design"):
        registry.design_of_directory(tmp_path)
    with pytest.raises(ValueError, match="no design"):
        registry.design_of(object())


# --------------------------------------------------------------------------- request state
def test_windowed_layers_keep_a_ring_and_recurrent_layers_a_state():
    cfg = cases.MODELS["mixed"]()
    state = HybridState(cfg, max_context=1000, device="cpu", chunk=32)
    assert state.layers[1].k.shape == (19 - 1 + 32, 2, 24) and state.layers[1].v.shape == (50, 2, 40)
    assert state.layers[3].k.shape[0] == 5 - 1 + 32
    assert state.layers[0].rec.shape == (6, 24, 40) and state.layers[0].rec.dtype == torch.float32
    assert state.layers[0].conv.shape == (4, 2 * 3 * 24 + 6 * 40) and state.layers[2].conv is None
    assert all(v.data_ptr() % 64 == 0 for h in state.layers for v in (h.k, h.v, h.rec, h.conv) if v is not None)
    assert HybridState(cfg, max_context=20, device="cpu", chunk=32).layers[1].k.shape[0] == 20
    blank = state.blank()
    assert blank.layers[1].k.shape == state.layers[1].k.shape and blank.layers[1].k.data_ptr() != state.layers[1].k.data_ptr()
    assert len(state.history()) == 4 and not state.keeps_every_row


def test_views_of_a_state_do_not_overlap():
    state = HybridState(cases.MODELS["mixed"](), max_context=40, device="cpu", dtype=torch.float32)
    views = [v for h in state.layers for v in (h.k, h.v, h.rec, h.conv) if v is not None]
    for number, view in enumerate(views):
        view.fill_(number + 1)
    assert all(bool((view == number + 1).all()) for number, view in enumerate(views))


# ----------------------------------------------------------------------------------- C ABI
def declarations():
    text = re.sub(r"/\*.*?\*/", "", HEADER.read_text(), flags=re.S)
    return re.findall(r"\b(int|long long)\s+(qd_[a-z0-9_]+)\s*\(([^)]*)\)\s*;", text)


def test_hybrid_bindings_follow_the_header():
    kinds = {ctypes.c_void_p: "pointer", ctypes.c_int: "int", ctypes.c_float: "float", ctypes.c_longlong: "long long"}
    found = declarations()
    signatures = {name: kinds for names in _lib.HYBRID_LIBRARIES.values() for name, kinds in names.items()}
    assert {name for _, name, _ in found} | {"qd_set_chained_launches"} == set(signatures)
    for result, name, params in found:
        declared = ["pointer" if "*" in p else re.sub(r"\s+\w+$", "", p.strip()) for p in params.split(",")]
        assert [kinds[t] for t in signatures[name]] == declared, name
        assert (name in _lib.HYBRID_LONG_RESULTS) == (result == "long long"), name


def test_structures_follow_the_header():
    """Field by field: names, order and types (pointers first, so that there is no padding between them)."""
    kinds = {ctypes.c_void_p: "pointer", ctypes.c_int: "int", ctypes.c_float: "float", ctypes.c_longlong: "long long"}
    text = re.sub(r"/\*.*?\*/", "", HEADER.read_text(), flags=re.S)
    found = re.findall(r"typedef struct (\w+) \{(.*?)\} \1;", text, flags=re.S)
    assert {name for name, _ in found} == set(_lib.STRUCTURES)
    for name, body in found:
        declared = []
        for line in filter(None, (part.strip() for part in body.split(";"))):
            kind, names = re.match(r"(const void\*|void\*|const float\*|float\*|const int\*|unsigned int\*|long long|float|int)\s+(.*)", line, re.S).groups()
            declared += [(field.strip(), "pointer" if kind.endswith("*") else kind) for field in names.split(",")]
        assert [(field, kinds[kind]) for field, kind in _lib.STRUCTURES[name]._fields_] == declared, name


def test_hybrid_libraries_export_what_the_header_declares():
    for target, names in _lib.HYBRID_LIBRARIES.items():
        handle = _lib.hybrid_lib(target)
        for name in names:
            assert hasattr(handle, name), name
        assert handle.qd_error_string(4) == b"shape not covered by this kernel"


def test_every_source_belongs_to_one_library():
    from quickdraw_b200 import build
    owned = [path.stem for target in build.TARGETS for path in build.sources(target) if path.stem not in build.COMMON]
    everything = sorted(path.stem for path in build.CSRC.glob("*.cu"))
    assert sorted(owned + [name for name in build.COMMON]) == everything
    assert {t for design in registry.DESIGNS for t in design.libraries} == set(build.TARGETS)


def test_missing_hybrid_library_fails_loudly(monkeypatch, tmp_path):
    monkeypatch.setattr(_lib, "_hybrid", {})
    monkeypatch.setattr(_lib, "LIB_PATH", tmp_path / "libquickdraw_b200.so")
    for target in _lib.HYBRID_LIBRARIES:
        with pytest.raises(_lib.LibraryMissing, match=f"build {target}"):
            _lib.hybrid_lib(target)


@pytest.mark.parametrize("tokens", [1, 2, 40])
@pytest.mark.parametrize("name", cases.MODELS)
def test_drivers_pass_the_declared_number_of_arguments(recorder, name, tokens):
    cfg = cases.MODELS[name]()
    ckpt = synthetic.make_fezopel(cfg)
    model, state = hybrid.FezopelModel(ckpt), HybridState(cfg, 64, "cpu")
    ids = torch.arange(tokens).as_subclass(AsIfOnGpu)
    logits = model.run(ids, 3, state, [0, tokens - 1])
    assert logits.shape == (2, cfg.vocab_size) and logits.dtype == torch.float32
    names = [n for n, _ in recorder]
    assert names.count("qd_sublayer_close") == sum(1 + (layer.ff is not None) for layer in cfg.layers)
    windowed = sum(isinstance(layer.mixer, WindowAttnConfig) for layer in cfg.layers)
    assert names.count("qd_attention" if tokens > 1 else "qd_attention_step") == windowed
    recorder.clear()
    assert model.run(ids, 3, state) is None                       # nothing wanted: it ends behind the last mixer
    assert [n for n, _ in recorder].count("qd_layer_norm_rows") == 0
    assert [n for n, _ in recorder].count("qd_sublayer_close") < names.count("qd_sublayer_close")
    recorder.clear()
    assert model(ckpt, torch.tensor(5), torch.tensor(3, dtype=torch.int32), state).shape == (cfg.vocab_size,)
    assert recorder[-1][0] == "qd_greedy"


def test_stacked_matrices_start_on_multiples_of_eight_rows():
    parts = {"a": torch.randn(5, 4), "b": torch.randn(8, 4), "c": torch.randn(1, 4)}
    matrix, at = mixers.stack_rows(parts)
    assert at == {"a": 0, "b": 8, "c": 16} and matrix.shape == (24, 4)
    for name, part in parts.items():
        assert torch.equal(matrix[at[name]:at[name] + part.shape[0]], part)
    assert float(matrix[5:8].abs().sum()) == 0


def test_frequencies_carry_more_than_fp32(recorder):
    m = cases.attention(rotary_dims=16, base=1234.5)
    mixer = mixers.WindowAttention(synthetic.make_fezopel(cases.config([(m, None)])).layers[0].mixer, m, 1e-6, "cpu")
    exact = torch.tensor([1234.5 ** (-2.0 * i / 16) for i in range(8)], dtype=torch.float64)
    assert float((mixer.freq.double().sum(0) / exact - 1).abs().max()) < 1e-13


# ---------------------------------------------------------------------- engine control flow
class CountingStep:
    def __init__(self, vocab):
        self.vocab, self.calls = vocab, []

    def __call__(self, ckpt, token_id, position, state, **kwargs):
        self.calls.append((int(token_id), int(position)))
        state.rec_state.add_(1.0)
        return torch.nn.functional.one_hot(token_id, self.vocab).float()


def test_extend_continues_a_request_and_answers_in_the_order_asked():
    cfg = cases.MODELS["mixed"]()
    step = CountingStep(cfg.vocab_size)
    engine = Engine(synthetic.make_fezopel(cfg), max_context=12, device="cpu", step=step)
    assert isinstance(engine.state, HybridState)
    rows = engine.extend([7, 8, 9], [2, 0, 2])
    assert rows.shape == (3, cfg.vocab_size) and rows.argmax(1).tolist() == [9, 7, 9]
    assert engine.extend([4], []).shape == (0, cfg.vocab_size)
    assert step.calls == [(7, 0), (8, 1), (9, 2), (4, 3)] and engine.state.position == 4
    with pytest.raises(AssertionError, match="capacity"):
        engine.extend([1] * 9)
    with pytest.raises(AssertionError, match="vocabulary"):
        engine.extend([cfg.vocab_size])
    with pytest.raises(AssertionError, match="wanted place"):
        engine.extend([1], [1])
    engine.reset()
    assert engine.state.position == 0 and engine.extend([3], [0]).argmax().item() == 3 and step.calls[-1] == (3, 0)


def test_extend_serves_the_other_design_too():
    cfg = synthetic.model_config(num_layers=4, vocab_size=64)
    from quickdraw_b200.weights import Checkpoint
    step = CountingStep(64)
    engine = Engine(Checkpoint(config=cfg, embed_tokens=None, final_norm=None, lm_head=None, layers=[]), max_context=8, device="cpu", step=step)
    assert isinstance(engine.state, DecodeState)
    assert engine.extend([5, 6, 7], [1]).argmax(1).tolist() == [6] and step.calls[-1] == (7, 2)


def test_snapshots_of_a_windowed_state_copy_the_ring():
    cfg = cases.MODELS["mixed"]()
    engine = Engine(synthetic.make_fezopel(cfg), max_context=32, device="cpu", step=CountingStep(cfg.vocab_size))
    engine.extend([1, 2, 3])
    engine.state.kv_k.fill_(2.0)
    snap = engine.snapshot()
    engine.reset()
    engine.extend([9, 9, 9, 9])
    engine.state.kv_k.fill_(5.0)
    engine.restore(snap)
    assert engine.state.position == 3 and float(engine.state.kv_k.float().mean()) == 2.0
    assert snap.nbytes() == sum(engine.state.memory_bytes().values())


def test_float32_is_only_for_designs_that_have_it():
    cfg = synthetic.model_config(num_layers=4, vocab_size=64)
    from quickdraw_b200.weights import Checkpoint
    with pytest.raises(AssertionError, match="does not run in"):
        Engine(Checkpoint(config=cfg, embed_tokens=None, final_norm=None, lm_head=None, layers=[]), device="cpu",
               step=CountingStep(64), dtype=torch.float32)


# ----------------------------------------------------------------------------- trace replay
def replayed(monkeypatch, capsys, tmp_path, steps, dtype="bfloat16"):
    cfg = cases.MODELS["mixed"]()
    save_hybrid_checkpoint(cfg, cases.tensors(cfg), tmp_path / "model")
    built = []
    from quickdraw_b200 import build
    monkeypatch.setattr(build, "build", lambda targets: built.append(targets))
    engines = []

    def from_pretrained(path, **kwargs):
        engines.append(Engine(synthetic.make_fezopel(cfg), max_context=kwargs["max_context"], device="cpu",
                              step=CountingStep(cfg.vocab_size), dtype=kwargs["dtype"]))
        return engines[-1]

    monkeypatch.setattr(Engine, "from_pretrained", staticmethod(from_pretrained))
    monkeypatch.setattr(sys, "argv", ["trace_run", "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(tmp_path),
                                      "--max-tokens", "16"])
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    code = replay.main()
    assert built == [("hybrid", "recurrent")] and engines[0].dtype == getattr(torch, dtype)
    return code, capsys.readouterr().out.split("\n"), cfg.vocab_size


def test_replay_answers_every_step_and_writes_wanted_logits(monkeypatch, capsys, tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    code, lines, vocab = replayed(monkeypatch, capsys, tmp_path, steps, "float32")
    assert code == 0 and [x for x in lines if x] == ["done 0", "done 1", "done 2"]
    rows = torch.frombuffer(bytearray((tmp_path / "0.f32").read_bytes()), dtype=torch.float32).view(-1, vocab)
    assert rows.argmax(1).tolist() == [3, 5] and not (tmp_path / "1.f32").exists()
    assert (tmp_path / "2.f32").stat().st_size == 4 * vocab


def test_replay_refuses_two_live_requests(monkeypatch, capsys, tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [4], "want": []}], "end": []}]
    with pytest.raises(RuntimeError, match="one request at a time"):
        replayed(monkeypatch, capsys, tmp_path, steps)


def test_replay_refuses_a_number_format_the_design_does_not_have(monkeypatch, tmp_path, capsys):
    (tmp_path / "config.json").write_text(json.dumps({"text_config": {}}))
    monkeypatch.setattr(sys, "argv", ["trace_run", "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path)])
    assert replay.main() == 3
