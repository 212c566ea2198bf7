"""The plain implementation of the Fezopel design against independent formulations of its mechanisms (CPU)."""

import math

import pytest
import torch

from oracle import fezopel_oracle as O
from tests import hybrid_cases as cases

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def test_layer_norm_is_torch_layer_norm():
    x, w, b = rnd(5, 33), rnd(33, seed=1), rnd(33, seed=2)
    torch.testing.assert_close(O.layer_norm(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (33,), w, b, 1e-3))


@pytest.mark.parametrize("window", [1, 4, 30])
def test_window_attention_is_a_masked_softmax_with_an_extra_column(window):
    q, k, v, sinks = rnd(20, 4, 6), rnd(20, 2, 6, seed=1), rnd(20, 2, 5, seed=2), rnd(4, seed=3)
    got = O.window_sink_attention(q, k, v, sinks, 0.7, window)
    i, j = torch.arange(20)[:, None], torch.arange(20)[None]
    for h in range(4):
        scores = (q[:, h] @ k[:, h // 2].T * 0.7).masked_fill((j > i) | (i - j >= window), -math.inf)
        weights = torch.softmax(torch.cat([scores, sinks[h].expand(20, 1)], 1), 1)[:, :20]
        torch.testing.assert_close(got[:, h], weights @ v[:, h // 2])


def test_rotation_keeps_norms_and_depends_on_distance_only():
    x = rnd(1, 1, 12).expand(9, 1, 12)
    at = O.rotate_interleaved(x, torch.arange(9), 100.0, 8)
    assert torch.equal(at[0], x[0]) and torch.equal(at[..., 8:], x[..., 8:])
    torch.testing.assert_close(at.norm(dim=-1), x.norm(dim=-1))
    torch.testing.assert_close((at[3] * at[5]).sum(), (at[6] * at[8]).sum())


def test_gla_recurrence_is_a_decayed_sum():
    q, k, v, a = rnd(7, 2, 3), rnd(7, 2, 3, seed=1), rnd(7, 2, 4, seed=2), torch.sigmoid(rnd(7, 2, 3, seed=3))
    got, state = O.gla_recurrence(q, k, v, a)
    for t in range(7):
        want = sum(((q[t] * a[j + 1:t + 1].prod(0) * k[j]).sum(-1, keepdim=True) * v[j]) for j in range(t + 1))
        torch.testing.assert_close(got[t], want)
    again, _ = O.gla_recurrence(q[4:], k[4:], v[4:], a[4:], O.gla_recurrence(q[:4], k[:4], v[:4], a[:4])[1])
    torch.testing.assert_close(again, got[4:])


def test_delta_rule_with_full_steps_stores_the_value():
    """beta = 1 and unit keys: reading the key back right after the write returns the value."""
    k, v = O.unit(rnd(6, 2, 5)), rnd(6, 2, 4, seed=1)
    g, beta = torch.sigmoid(rnd(6, 2, 5, seed=2)), torch.ones(6, 2, dtype=F64)
    got, _ = O.channel_delta_recurrence(k, k, v, g, beta)
    torch.testing.assert_close(got, v, rtol=1e-4, atol=1e-4)      # unit() has an eps inside its root


def test_convolution_is_causal_and_its_last_tap_is_the_present():
    x, taps = rnd(8, 3), rnd(3, 4, seed=1)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (3, 0)), taps[:, None], groups=3)[0].T
    torch.testing.assert_close(O.causal_conv(x, taps), want)
    assert torch.equal(O.causal_conv(x, torch.tensor([[0.0, 0, 0, 1]] * 3, dtype=F64)), x)


def test_decays():
    z = rnd(50) * 6
    torch.testing.assert_close(O.gla_decay(z, 4.0) ** 4, torch.sigmoid(z))
    torch.testing.assert_close(O.softplus(z), torch.nn.functional.softplus(z))
    torch.testing.assert_close(O.channel_delta_decay(z.view(1, 1, 50), torch.zeros(1, dtype=F64)).flatten(), torch.sigmoid(-z))


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_model_is_causal_and_finite(name):
    cfg = cases.MODELS[name]()
    weights, tokens = cases.tensors(cfg), cases.prompt(cfg, 24)
    logits, stream = O.forward(cfg.to_dict(), weights, tokens)
    assert logits.shape == (24, cfg.vocab_size) and stream.shape[0] == len(cfg.layers) and torch.isfinite(logits).all()
    shorter, _ = O.forward(cfg.to_dict(), weights, tokens[:13])
    torch.testing.assert_close(shorter, logits[:13])
