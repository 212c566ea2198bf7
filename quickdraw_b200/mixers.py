"""Token mixers of the bf16-weight hybrids: each knows its input projections (to be stacked with the
other products of the same input into one matrix), its form for a chunk of tokens and its one-launch
form for a single token.

``proj`` is the product of the stacked matrix and the chunk's normed rows; ``at`` maps a projection's
name to its first column.  Both forms return the rows that go into the output projection ``o`` and
leave the layer's history advanced.  ``position`` is that of the chunk's first token: an int, or a 0-d
int32 CUDA tensor so that a captured graph can be replayed at other positions.
"""

from __future__ import annotations

import torch

from ._lib import call_hybrid, hybrid_lib, ptr, stream_of
from .state import LayerHistory
from .weights import (ChannelDeltaConfig, ChannelDeltaWeights, GLAConfig, GLAWeights, WindowAttnConfig,
                      WindowAttnWeights)

BF16, F32 = torch.bfloat16, torch.float32
DTYPE_CODE = {BF16: 0, F32: 1}
SILU, SIGMOID = 0, 1


def column(t: torch.Tensor, offset: int):
    """Address of a row's element ``offset`` (of the first row)."""
    from ctypes import c_void_p
    return c_void_p(t.data_ptr() + offset * t.element_size())


def place(position) -> tuple:
    """(device pointer or NULL, host value) of a position."""
    return (ptr(position), 0) if isinstance(position, torch.Tensor) else (None, int(position))


def linear(x, x_column: int, ldx: int, weight, out, *, tokens: int, status, gelu_columns: int = 0) -> None:
    """out[t] = W x[t, x_column : x_column + in_features]; the first ``gelu_columns`` outputs through the exact GELU."""
    call_hybrid("qd_linear", column(x, x_column), ldx, DTYPE_CODE[x.dtype], ptr(weight), ptr(out), out.shape[1],
                DTYPE_CODE[out.dtype], tokens, weight.shape[0], weight.shape[1], gelu_columns, ptr(status), stream_of(x))


def step_covers(m) -> bool:
    """Whether the one-launch decode form of a recurrence takes these sizes (a cluster of at most eight blocks of 32 value columns)."""
    return m.vdim <= 256


class WindowAttention:
    KEYS_PER_SPLIT, MAX_SPLITS = 32, 64

    def __init__(self, weights: WindowAttnWeights, m: WindowAttnConfig, eps: float, device):
        self.w, self.m, self.eps = weights, m, eps
        self.projections = {"q": weights.q, "k": weights.k, "v": weights.v, "g": weights.g}
        self.out_columns = m.heads * m.vdim
        # frequencies as fp32 high and low parts: the angle keeps fp32 accuracy at any position
        exact = torch.tensor([m.rotary_base ** (-2.0 * i / m.rotary_dims) for i in range(m.rotary_dims // 2)], dtype=torch.float64)
        high = exact.to(F32)
        self.freq = torch.stack([high, (exact - high.double()).to(F32)]).contiguous().to(device)
        sms = torch.cuda.get_device_properties(device).multi_processor_count
        self.splits = max(1, min(-(-m.window // self.KEYS_PER_SPLIT), -(-2 * sms // m.kv_heads), self.MAX_SPLITS))
        floats = hybrid_lib().qd_window_attention_step_floats(m.heads, m.vdim, self.splits)
        self.partial = torch.empty(floats, dtype=F32, device=device)
        self.counters = torch.zeros(m.kv_heads, dtype=torch.int32, device=device)

    def _common(self, proj, at):
        return [column(proj, at[name]) for name in ("q", "k", "v", "g")]

    def _norms(self):
        return [ptr(self.w.q_norm), ptr(self.w.k_norm), ptr(self.freq), self.m.rotary_dims, ptr(self.w.sink), self.m.scale, self.eps]

    def _cache(self, history: LayerHistory):
        capacity = history.k.shape[0]
        return [ptr(history.k), ptr(history.v), capacity, min(self.m.window, capacity)]

    def chunk(self, proj, at, history: LayerHistory, position, status):
        m, tokens = self.m, proj.shape[0]
        q = torch.empty((tokens, m.heads * m.dim), dtype=proj.dtype, device=proj.device)
        out = torch.empty((tokens, self.out_columns), dtype=proj.dtype, device=proj.device)
        call_hybrid("qd_window_attention", *self._common(proj, at), proj.shape[1], *self._norms(), *self._cache(history), *place(position),
                    ptr(q), ptr(out), tokens, m.heads, m.kv_heads, m.dim, m.vdim, DTYPE_CODE[proj.dtype], stream_of(proj))
        return out

    def step(self, proj, at, history: LayerHistory, position, status):
        m = self.m
        out = torch.empty((1, self.out_columns), dtype=proj.dtype, device=proj.device)
        call_hybrid("qd_window_attention_step", *self._common(proj, at), *self._norms(), *self._cache(history), *place(position),
                    ptr(self.partial), ptr(self.counters), self.splits, ptr(out), m.heads, m.kv_heads, m.dim, m.vdim,
                    DTYPE_CODE[proj.dtype], stream_of(proj))
        return out


class LinearRecurrence:
    """What the two recurrences share: the fp32 operands of a chunk, the walk over its tokens, the per-head norm and gate."""

    def __init__(self, weights, m, eps: float, kv_heads: int):
        self.w, self.m, self.eps, self.kv_heads = weights, m, eps, kv_heads
        self.out_columns = m.heads * m.vdim

    def _operands(self, proj, at, status):
        m, tokens, dev = self.m, proj.shape[0], proj.device
        new = lambda *shape: torch.empty(shape, dtype=F32, device=dev)
        decay = new(tokens, m.heads * m.dim)
        linear(proj, at["a1"], proj.shape[1], self.w.a2, decay, tokens=tokens, status=status)      # logits; decays in place later
        return (new(tokens, self.kv_heads * m.dim), new(tokens, self.kv_heads * m.dim), decay, new(tokens, m.heads * m.vdim))

    def _walk(self, q, k, decay, v, beta, scales, history, gate, gate_column: int, act: int, dtype):
        m, tokens = self.m, q.shape[0]
        raw = torch.empty((tokens, self.out_columns), dtype=F32, device=q.device)
        call_hybrid("qd_linear_recurrence", ptr(q), ptr(k), ptr(decay), ptr(v), ptr(beta), ptr(scales), ptr(history.rec), ptr(raw), tokens,
                    m.heads, self.kv_heads, m.dim, m.vdim, int(beta is not None), stream_of(q))
        out = torch.empty((tokens, self.out_columns), dtype=dtype, device=q.device)
        call_hybrid("qd_head_norm_gate", ptr(raw), ptr(self.w.norm), column(gate, gate_column), gate.shape[1], ptr(out), tokens, m.heads,
                    m.vdim, self.eps, act, DTYPE_CODE[dtype], stream_of(q))
        return out


class GatedLinearAttention(LinearRecurrence):
    def __init__(self, weights: GLAWeights, m: GLAConfig, eps: float, device):
        super().__init__(weights, m, eps, m.heads)
        self.projections = {"q": weights.q, "k": weights.k, "v": weights.v, "g": weights.g, "a1": weights.a1}

    def chunk(self, proj, at, history: LayerHistory, position, status):
        m, tokens = self.m, proj.shape[0]
        q, k, decay, v = self._operands(proj, at, status)
        call_hybrid("qd_gla_prepare", *[column(proj, at[n]) for n in "qkv"], proj.shape[1], ptr(decay), ptr(self.w.a2_b), m.tau, ptr(q),
                    ptr(k), ptr(decay), ptr(v), tokens, m.heads, m.dim, m.vdim, DTYPE_CODE[proj.dtype], stream_of(proj))
        return self._walk(q, k, decay, v, None, None, history, proj, at["g"], SILU, proj.dtype)

    def step(self, proj, at, history: LayerHistory, position, status):
        m = self.m
        if not step_covers(m):
            return self.chunk(proj, at, history, position, status)
        out = torch.empty((1, self.out_columns), dtype=proj.dtype, device=proj.device)
        call_hybrid("qd_gla_step", *[column(proj, at[n]) for n in ("q", "k", "v", "a1")], ptr(self.w.a2), ptr(self.w.a2_b),
                    self.w.a2.shape[1], m.tau, column(proj, at["g"]), ptr(self.w.norm), self.eps, ptr(history.rec), ptr(out), m.heads,
                    m.dim, m.vdim, DTYPE_CODE[proj.dtype], stream_of(proj))
        return out


class ChannelDelta(LinearRecurrence):
    def __init__(self, weights: ChannelDeltaWeights, m: ChannelDeltaConfig, eps: float, device):
        super().__init__(weights, m, eps, m.kv_heads)
        self.projections = {"q": weights.q, "k": weights.k, "v": weights.v, "b": weights.b, "a1": weights.a1, "g1": weights.g1}

    def _convolution(self, history):
        w = self.w
        return [ptr(w.A_log), ptr(w.q_conv), ptr(w.k_conv), ptr(w.v_conv), ptr(history.conv), self.m.conv]

    def chunk(self, proj, at, history: LayerHistory, position, status):
        m, tokens, dev = self.m, proj.shape[0], proj.device
        q, k, decay, v = self._operands(proj, at, status)
        beta = torch.empty((tokens, m.heads), dtype=F32, device=dev)
        scales = torch.empty((tokens, m.kv_heads, 3), dtype=F32, device=dev)
        call_hybrid("qd_channel_delta_prepare", *[column(proj, at[n]) for n in "qkvb"], proj.shape[1], ptr(decay), ptr(self.w.dt_bias),
                    *self._convolution(history), *place(position), ptr(q), ptr(k), ptr(decay), ptr(v), ptr(beta), ptr(scales), tokens,
                    m.heads, m.kv_heads, m.dim, m.vdim, DTYPE_CODE[proj.dtype], stream_of(proj))
        gate = torch.empty((tokens, self.out_columns), dtype=proj.dtype, device=dev)
        linear(proj, at["g1"], proj.shape[1], self.w.g2, gate, tokens=tokens, status=status)
        return self._walk(q, k, decay, v, beta, scales, history, gate, 0, SIGMOID, proj.dtype)

    def step(self, proj, at, history: LayerHistory, position, status):
        m = self.m
        if not step_covers(m):
            return self.chunk(proj, at, history, position, status)
        out = torch.empty((1, self.out_columns), dtype=proj.dtype, device=proj.device)
        call_hybrid("qd_channel_delta_step", *[column(proj, at[n]) for n in ("q", "k", "v", "b", "a1")], ptr(self.w.a2), ptr(self.w.dt_bias),
                    self.w.a2.shape[1], *self._convolution(history), *place(position), column(proj, at["g1"]), ptr(self.w.g2),
                    self.w.g2.shape[1], ptr(self.w.norm), self.eps, ptr(history.rec), ptr(out), m.heads, m.kv_heads, m.dim, m.vdim,
                    DTYPE_CODE[proj.dtype], stream_of(proj))
        return out


MIXERS = {WindowAttnConfig: WindowAttention, GLAConfig: GatedLinearAttention, ChannelDeltaConfig: ChannelDelta}
