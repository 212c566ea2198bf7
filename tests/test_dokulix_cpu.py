"""Host side of the Dokulix design, no GPU: configuration, checkpoint files, request state, what the drivers launch,
engine control flow, trace replay."""

import io
import json
import sys

import pytest
import torch

from quickdraw_b200 import hybrid, mixers, registry, replay, synthetic
from quickdraw_b200.engine import Engine
from quickdraw_b200.loader import hybrid_shapes, load_hybrid_checkpoint, save_hybrid_checkpoint
from quickdraw_b200.state import HybridState
from quickdraw_b200.weights import ChunkAttnConfig, DokulixConfig, LatentAttnConfig
from tests import dokulix_cases as cases
from tests.recording import AsIfOnGpu, recorder  # noqa: F401 (a fixture)


# ------------------------------------------------------------------- configuration, files
@pytest.mark.parametrize("name", cases.MODELS)
def test_configuration_round_trip(name):
    cfg = cases.MODELS[name]()
    assert DokulixConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_a_configuration_without_a_loop_entry():
    data = cases.MODELS["no loop"]().to_dict()
    del data["loop"]
    assert DokulixConfig.from_dict(data).loop is None


@pytest.mark.parametrize("change,message", [
    (lambda d: d.update(architecture="Other"), "not a Dokulix"), (lambda d: d["layers"][0].update(type="mamba"), "unknown mixer"),
    (lambda d: d["layers"][0]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda d: d["layers"][2]["mixer"].update(kv_heads=4), "do not divide"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), "rotated dimensions"),
    (lambda d: d["loop"].update(stop=5), "loop over layers"), (lambda d: d["loop"].update(start=3), "loop over layers")])
def test_configuration_refuses_what_it_does_not_know(change, message):
    data = cases.MODELS["middle loop"]().to_dict()
    change(data)
    with pytest.raises(ValueError, match=message):
        DokulixConfig.from_dict(data)


def test_layer_runs():
    assert cases.MODELS["middle loop"]().runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert cases.MODELS["one layer again"]().runs() == [(0, None), (1, 0), (1, 1), (1, 2), (1, 3)]
    assert cases.MODELS["no loop"]().runs() == [(0, None), (1, None)]


def test_checkpoint_round_trip(tmp_path):
    cfg = cases.MODELS["middle loop"]()
    tensors = cases.tensors(cfg)
    save_hybrid_checkpoint(cfg, tensors, tmp_path)
    design = registry.design_of_directory(tmp_path)
    assert design.name == "dokulix" and design.libraries == ("hybrid", "latent")
    ckpt = design.load(tmp_path, "cpu")
    assert ckpt.config == cfg and registry.design_of(ckpt) is design
    assert torch.equal(ckpt.layers[0].mixer.dkv_norm, tensors["l0.mix.dkv.norm"]) and torch.equal(ckpt.layers[2].mixer.o_b, tensors["l2.mix.o.b"])
    assert torch.equal(ckpt.layers[2].mixer.q_norm, tensors["l2.mix.q.norm"]) and torch.equal(ckpt.layers[3].mlp.up, tensors["l3.mlp.up"])
    assert ckpt.layers[1].mlp is None and ckpt.layers[1].norm2 is None and torch.equal(ckpt.loop_steps, tensors["loop.step"])
    assert set(hybrid_shapes(cfg)) == set(tensors)


def test_checkpoint_with_a_missing_or_misshapen_tensor_is_refused(tmp_path):
    cfg = cases.MODELS["middle loop"]()
    tensors = cases.tensors(cfg)
    save_hybrid_checkpoint(cfg, {k: v for k, v in tensors.items() if k != "loop.step"}, tmp_path / "a")
    with pytest.raises(ValueError, match="loop.step is missing"):
        load_hybrid_checkpoint(tmp_path / "a", "cpu")
    save_hybrid_checkpoint(cfg, tensors | {"l0.mix.uk": tensors["l0.mix.uk"][:1]}, tmp_path / "b")
    with pytest.raises(ValueError, match="l0.mix.uk has shape"):
        load_hybrid_checkpoint(tmp_path / "b", "cpu")


def test_an_unknown_architecture_is_refused(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="no bf16-weight design"):
        load_hybrid_checkpoint(tmp_path, "cpu")


# --------------------------------------------------------------------------- request state
def test_every_pass_over_a_looped_layer_has_its_own_rows():
    cfg = cases.MODELS["middle loop"]()
    state = HybridState(cfg, max_context=1000, device="cpu", chunk=32, dtype=torch.float32)
    assert len(state.layers) == 8
    assert state.layers[0].latent.shape == (19 - 1 + 32, 48) and state.layers[0].k is None       # 32 latent + 8 rotated columns
    assert state.layers[1].latent.shape[0] == state.layers[3].latent.shape[0] == 7 - 1 + 32
    assert state.layers[2].k.shape == (21 - 1 + 32, 2, 24) and state.layers[2].v.shape == (52, 2, 40)
    views = [v for h in state.layers for v in (h.k, h.v, h.latent) if v is not None]
    assert all(v.data_ptr() % 64 == 0 for v in views)
    for number, view in enumerate(views):
        view.fill_(number + 1)
    assert all(bool((view == number + 1).all()) for number, view in enumerate(views))
    assert HybridState(cfg, max_context=20, device="cpu", chunk=32).layers[7].latent.shape[0] == 20
    assert not state.keeps_every_row and state.blank().layers[7].latent.shape == state.layers[7].latent.shape


@pytest.mark.parametrize("kv_rank,rot_dim", [(32, 8), (19, 6), (136, 16), (72, 32), (512, 64), (8, 2)])
def test_cache_rows_are_aligned(kv_rank, rot_dim):
    m = cases.latent(kv_rank=kv_rank, rot_dim=rot_dim)
    assert m.rot_column >= kv_rank and m.rot_column % 8 == 0 and m.row % 16 == 0 and m.row >= m.rot_column + rot_dim
    assert -(-kv_rank // 16) * 16 <= m.row                       # value columns are read in groups of sixteen


def test_ring_segments():
    assert mixers.ring_segments(0, 5, 8) == [(0, 5)] and mixers.ring_segments(3, 5, 8) == [(3, 5)]
    assert mixers.ring_segments(6, 5, 8) == [(6, 2), (0, 3)] and mixers.ring_segments(22, 8, 8) == [(6, 2), (0, 6)]
    for first in range(20):
        for count in range(1, 8):
            rows = [r for row, n in mixers.ring_segments(first, count, 7) for r in range(row, row + n)]
            assert rows == [(first + i) % 7 for i in range(count)]


def test_slopes():
    assert ChunkAttnConfig(4, 2, 8, 8, 16, 1.0).slopes() == [0.25, 0.0625, 0.015625, 0.00390625]


# ------------------------------------------------------------------------------- launches
@pytest.mark.parametrize("tokens", [1, 2, 40])
@pytest.mark.parametrize("name", cases.MODELS)
def test_drivers_pass_the_declared_number_of_arguments(recorder, name, tokens):  # noqa: F811
    cfg = cases.MODELS[name]()
    ckpt = synthetic.make_dokulix(cfg)
    model, state = hybrid.DokulixModel(ckpt), HybridState(cfg, 64, "cpu")
    ids = torch.arange(tokens).as_subclass(AsIfOnGpu)
    logits = model.run(ids, 3, state, [0, tokens - 1] if tokens > 1 else [0])
    assert logits.shape == (min(tokens, 2), cfg.vocab_size) and logits.dtype == torch.float32
    names = [n for n, _ in recorder]
    mixed = [type(cfg.layers[i].mixer) for i, _ in cfg.runs()]
    if tokens > 1:
        assert names.count("qd_latent_prepare") == mixed.count(LatentAttnConfig) and names.count("qd_attention") == len(mixed)
    else:
        assert names.count("qd_latent_step") == mixed.count(LatentAttnConfig) and names.count("qd_attention_step") == mixed.count(ChunkAttnConfig)
    recorder.clear()
    assert model.run(ids, 3, state) is None                       # nothing wanted: it ends behind the last mixer
    assert len(recorder) < len(names)
    recorder.clear()
    assert model(ckpt, torch.tensor(5), torch.tensor(3, dtype=torch.int32), state).shape == (cfg.vocab_size,)
    assert recorder[-1][0] == "qd_greedy"


def test_one_token_needs_no_launches_for_norms_and_sums(recorder):  # noqa: F811
    """Five launches per layer with chunked attention, six calls with latent attention (whose step is three kernels)."""
    cfg = cases.MODELS["middle loop"]()
    model = hybrid.DokulixModel(synthetic.make_dokulix(cfg))
    model(model.ckpt, torch.tensor(5), torch.tensor(3, dtype=torch.int32), HybridState(cfg, 64, "cpu"))
    expected = 1 + 2                                             # embedding row; logits, choice
    for i, _ in cfg.runs():
        expected += (4 if isinstance(cfg.layers[i].mixer, LatentAttnConfig) else 3) + (2 if cfg.layers[i].ff else 0)
    assert len(recorder) == expected
    assert [n for n, _ in recorder].count("qd_stream_norm") == 1


def test_gate_and_up_rows_alternate():
    cfg = cases.MODELS["middle loop"]()
    ckpt = synthetic.make_dokulix(cfg)

    class Mixer:
        projections = {"q": ckpt.layers[2].mixer.q}
    part = hybrid._PreNorm(ckpt.layers[2], Mixer)
    assert torch.equal(part.glu[0::2], ckpt.layers[2].mlp.gate) and torch.equal(part.glu[1::2], ckpt.layers[2].mlp.up)


def test_what_the_last_product_of_a_run_adds(recorder):  # noqa: F811
    """Its bias where there is no feed-forward, and the vector of the pass that begins behind it."""
    cfg = cases.MODELS["one layer again"]()
    ckpt = synthetic.make_dokulix(cfg)
    model = hybrid.DokulixModel(ckpt)
    steps, bias = ckpt.loop_steps.float(), ckpt.layers[1].mixer.o_b.float()
    assert torch.equal(model.closing[0], steps[0])                # in front of the first pass, the layer has a feed-forward
    assert all(torch.equal(model.closing[r], bias + steps[r]) for r in (1, 2, 3)) and torch.equal(model.closing[4], bias)


# ------------------------------------------------------------------ engine, trace replay
class CountingStep:
    def __init__(self, vocab):
        self.vocab, self.calls = vocab, []

    def __call__(self, ckpt, token_id, position, state, **kwargs):
        self.calls.append((int(token_id), int(position)))
        return torch.nn.functional.one_hot((token_id + 1) % self.vocab, self.vocab).float()


def test_engine_generates_and_continues_with_this_design():
    cfg = cases.MODELS["middle loop"]()
    step = CountingStep(cfg.vocab_size)
    engine = Engine(synthetic.make_dokulix(cfg), max_context=16, device="cpu", step=step)
    assert isinstance(engine.state, HybridState) and len(engine.state.layers) == 8
    assert engine.generate([3, 4], 4) == [5, 6, 7, 8]
    engine.reset()
    assert engine.extend([7, 8, 9], [2, 0]).argmax(1).tolist() == [10, 8] and engine.state.position == 3


def test_replay_serves_this_design_and_builds_only_its_kernels(monkeypatch, capsys, tmp_path):
    cfg = cases.MODELS["one layer again"]()
    save_hybrid_checkpoint(cfg, cases.tensors(cfg), tmp_path / "model")
    built = []
    from quickdraw_b200 import build
    monkeypatch.setattr(build, "build", lambda targets: built.append(targets))
    monkeypatch.setattr(Engine, "from_pretrained", staticmethod(lambda path, **kw: Engine(
        registry.design_of_directory(path).load(path, "cpu"), max_context=kw["max_context"], device="cpu", step=CountingStep(cfg.vocab_size),
        dtype=kw["dtype"])))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [2, 0]}], "end": ["a"]},
             {"step": 1, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": []}]
    monkeypatch.setattr(sys, "argv", ["trace_run", "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path)])
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert replay.main() == 0 and built == [("hybrid", "latent")]
    assert [x for x in capsys.readouterr().out.split("\n") if x] == ["done 0", "done 1"]
    rows = torch.frombuffer(bytearray((tmp_path / "0.f32").read_bytes()), dtype=torch.float32).view(-1, cfg.vocab_size)
    assert rows.argmax(1).tolist() == [4, 6]
