"""Small Fezopel models for the tests: configurations, seeded tensors, and what the oracle says about them."""

import torch

from quickdraw_b200 import synthetic
from quickdraw_b200.weights import ChannelDeltaConfig, FezopelConfig, GLAConfig, HybridLayerConfig, WindowAttnConfig


def attention(heads=6, kv_heads=2, dim=24, vdim=40, window=19, rotary_dims=8, base=2.0e4, scale=0.3):
    return WindowAttnConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window, rotary_dims=rotary_dims,
                            rotary_base=base, scale=scale)


def gla(heads=3, dim=40, vdim=24, tau=7.0):
    return GLAConfig(heads=heads, dim=dim, vdim=vdim, tau=tau)


def delta(heads=6, kv_heads=3, dim=24, vdim=40, conv=4):
    return ChannelDeltaConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def config(layers, width=96, vocab=203, eps=1e-5):
    return FezopelConfig(vocab_size=vocab, hidden_size=width, norm_eps=eps,
                         layers=[HybridLayerConfig(mixer, ff) for mixer, ff in layers])


# name -> configuration: every mixer with and without a feed-forward, shared and own key/value heads, partial and
# full rotation, convolutions of one to five taps, widths and heads that are and are not multiples of 8, 16, 32
MODELS = {
    "mixed": lambda: config([(delta(), None), (attention(), 112), (gla(), 56), (attention(heads=2, kv_heads=2, dim=16, vdim=16, window=5,
                                                                              rotary_dims=16), None), (delta(heads=2, kv_heads=2, conv=2), 80)]),
    "attention first": lambda: config([(attention(heads=4, kv_heads=1, dim=80, vdim=56, window=33, rotary_dims=80, base=500.0, scale=0.11), 160),
                                       (gla(heads=2, dim=72, vdim=48, tau=1.0), None), (delta(heads=4, kv_heads=4, dim=48, vdim=72, conv=3), None)],
                                      width=160, vocab=512, eps=1e-3),
    "odd sizes": lambda: config([(gla(heads=1, dim=20, vdim=36, tau=3.0), 50), (delta(heads=3, kv_heads=1, dim=18, vdim=10, conv=5), None),
                                 (attention(heads=3, kv_heads=3, dim=14, vdim=9, window=7, rotary_dims=6), 33),
                                 (delta(heads=1, kv_heads=1, dim=34, vdim=33, conv=1), None)], width=60, vocab=101),
    "window of one": lambda: config([(attention(window=1), 64), (gla(), None)]),
    "attention only": lambda: config([(attention(window=48), 96)], width=64),
}


def tensors(cfg, seed=3, rank=12):
    return synthetic.fezopel_tensors(cfg, seed, "cpu", rank)


def prompt(cfg, count, seed=0):
    return torch.randint(0, cfg.vocab_size, (count,), generator=torch.Generator().manual_seed(seed)).tolist()
