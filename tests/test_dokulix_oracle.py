"""The plain implementation of the Dokulix design against independent formulations of its mechanisms (CPU)."""

import math

import pytest
import torch

from oracle import dokulix_oracle as O
from tests import dokulix_cases as cases

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def test_norms():
    x, w = rnd(5, 33), rnd(33, seed=1)
    torch.testing.assert_close(O.rms_norm(x, w, 1e-3), torch.nn.functional.rms_norm(x, (33,), w, 1e-3))
    torch.testing.assert_close(O.rms_norm_around_one(x, w, 1e-3), O.rms_norm(x, 1 + w, 1e-3))


def test_feed_forward():
    h, gate, up, down = rnd(4, 6), rnd(9, 6, seed=1), rnd(9, 6, seed=2), rnd(6, 9, seed=3)
    want = torch.stack([down @ (torch.relu(gate @ x) * (up @ x)) for x in h])
    torch.testing.assert_close(O.relu_glu(h, gate, up, down), want)


def test_rotation_pairs_the_halves_and_depends_on_distance_only():
    x = rnd(1, 1, 12).expand(9, 1, 12)
    at = O.rotate_half(x, torch.arange(9), 100.0, 8)
    assert torch.equal(at[0], x[0]) and torch.equal(at[..., 8:], x[..., 8:])
    torch.testing.assert_close((at[3] * at[5]).sum(), (at[6] * at[8]).sum())
    plane = torch.complex(x[0, 0, :4], x[0, 0, 4:8]) * torch.exp(1j * 5 * 100.0 ** (-torch.arange(4, dtype=F64) / 4))
    torch.testing.assert_close(at[5, 0, :8], torch.cat([plane.real, plane.imag]))


@pytest.mark.parametrize("sees,size", [(O.sees_window, 1), (O.sees_window, 6), (O.sees_chunk, 1), (O.sees_chunk, 7), (O.sees_chunk, 40)])
@pytest.mark.parametrize("extra", [False, True])
def test_attention_is_a_masked_softmax(sees, size, extra):
    q, k, v, slopes = rnd(20, 4, 6), rnd(20, 2, 6, seed=1), rnd(20, 2, 5, seed=2), O.distance_slopes(4)
    got = O.masked_attention(q, k, v, 0.7, lambda i, j: sees(i, j, size), slopes, extra)
    i, j = torch.arange(20)[:, None], torch.arange(20)[None]
    visible = (j <= i) & ((i - j < size) if sees is O.sees_window else (i // size == j // size))
    for h in range(4):
        scores = q[:, h] @ k[:, h // 2].T * 0.7 - slopes[h] * (i - j)
        scores = scores.masked_fill(~visible, -math.inf)
        if extra:
            scores = torch.cat([scores, torch.zeros(20, 1, dtype=F64)], 1)
        torch.testing.assert_close(got[:, h], torch.softmax(scores, 1)[:, :20] @ v[:, h // 2])


def test_slopes_halve_over_an_eighth_of_the_heads():
    assert O.distance_slopes(8) == [2.0 ** -(h + 1) for h in range(8)]
    assert O.distance_slopes(1) == [2.0 ** -8]


def test_order_of_layer_runs():
    assert O.layer_runs(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert O.layer_runs(2, None) == [(0, None), (1, None)]


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_model_is_causal_and_finite(name):
    cfg = cases.MODELS[name]()
    weights, tokens = cases.tensors(cfg), cases.prompt(cfg, 24)
    logits, stream = O.forward(cfg.to_dict(), weights, tokens)
    assert logits.shape == (24, cfg.vocab_size) and stream.shape[0] == len(cfg.runs()) and torch.isfinite(logits).all()
    shorter, _ = O.forward(cfg.to_dict(), weights, tokens[:13])
    torch.testing.assert_close(shorter, logits[:13])


def test_a_loop_is_its_layers_written_out():
    """The same layers, copied, without a loop; the pass vectors added by hand in front of the first of each pass."""
    cfg = cases.MODELS["middle loop"]()
    w = {n: t.double() for n, t in cases.tensors(cfg).items()}
    tokens, eps = cases.prompt(cfg, 15), cfg.norm_eps
    x = w["embed"][torch.tensor(tokens)]
    one = lambda i, x: O.forward({"layers": [cfg.to_dict()["layers"][i]], "norm": {"eps": eps}, "vocab": 1, "width": 1},
                                 {"embed": x, "head": x[:1], "final.norm": w["final.norm"]} | {"l0." + n.split(".", 1)[1]: t for n, t in w.items()
                                                                                              if n.startswith(f"l{i}.")}, range(15))[1][0]
    for i, t in ((0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)):
        x = one(i, x if t is None else x + w["loop.step"][t])
    torch.testing.assert_close(O.rms_norm_around_one(x, w["final.norm"], eps) @ w["head"].T, O.forward(cfg.to_dict(), w, tokens)[0])
