"""Small Dokulix models for the tests: configurations, seeded tensors, prompts."""

import torch

from quickdraw_b200 import synthetic
from quickdraw_b200.weights import ChunkAttnConfig, DokulixConfig, LatentAttnConfig, LoopConfig, PreNormLayerConfig


def latent(heads=5, dim=24, rot_dim=8, vdim=40, q_rank=48, kv_rank=32, window=19, base=2.0e4, scale=0.25):
    return LatentAttnConfig(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, window=window, rotary_base=base,
                            scale=scale)


def chunked(heads=6, kv_heads=2, dim=24, vdim=40, span=21, scale=0.3):
    return ChunkAttnConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, span=span, scale=scale)


def config(layers, width=96, vocab=203, eps=1e-5, loop=None):
    return DokulixConfig(vocab_size=vocab, hidden_size=width, norm_eps=eps, loop=None if loop is None else LoopConfig(*loop),
                         layers=[PreNormLayerConfig(mixer, ff) for mixer, ff in layers])


# name -> configuration: both mixers with and without a feed-forward, loops in the middle, over everything, over one layer,
# once, never; sizes that are and are not multiples of 8 and 16, more than sixteen latent heads, one key/value head
MODELS = {
    "middle loop": lambda: config([(latent(), 112), (latent(heads=3, window=7, vdim=24), None), (chunked(), 56), (latent(window=50), 72)], loop=(1, 3, 3)),
    "loop over everything": lambda: config([(chunked(heads=4, kv_heads=1, dim=80, vdim=56, span=33), 160),
                                            (latent(heads=18, dim=16, rot_dim=16, vdim=8, kv_rank=136, q_rank=24, window=64), None)], width=160,
                                           vocab=512, eps=1e-3, loop=(0, 2, 2)),
    "one layer again": lambda: config([(latent(rot_dim=32, kv_rank=72), 64), (chunked(heads=2, kv_heads=2, dim=32, vdim=16, span=8), None)],
                                      width=64, loop=(1, 2, 4)),
    "loop of one pass": lambda: config([(chunked(), 64), (latent(window=12), 40)], loop=(0, 1, 1)),
    "no loop": lambda: config([(chunked(span=200), None), (latent(window=300), 88)]),
    "odd sizes": lambda: config([(latent(heads=3, dim=14, rot_dim=6, vdim=9, q_rank=21, kv_rank=19, window=7), 50),
                                 (chunked(heads=3, kv_heads=3, dim=13, vdim=9, span=11), 33)], width=60, vocab=101, loop=(0, 2, 2)),
    "spans of one": lambda: config([(latent(window=1), 64), (chunked(span=1), None)], loop=(1, 2, 2)),
}


def tensors(cfg, seed=3):
    return synthetic.dokulix_tensors(cfg, seed)


def prompt(cfg, count, seed=0):
    return torch.randint(0, cfg.vocab_size, (count,), generator=torch.Generator().manual_seed(seed)).tolist()
