"""Token mixers of the bf16-weight hybrids: each knows its input projections (to be stacked with the
other products of the same input into one matrix), its form for a chunk of tokens and its one-launch
form for a single token (latent attention: three launches).

``proj`` is the product of the stacked matrix and the chunk's normed rows; ``at`` maps a projection's
name to its first column.  Both forms return the rows that go into the output projection ``o`` and
leave the layer's history advanced.  ``position`` is that of the chunk's first token: an int, or a 0-d
int32 CUDA tensor so that a captured graph can be replayed at other positions.
"""

from __future__ import annotations

from ctypes import byref, c_void_p

import torch

from ._lib import AttentionArgs, LatentArgs, call_hybrid, ptr, size_hybrid, stream_of
from .state import LayerHistory
from .weights import (ChannelDeltaConfig, ChannelDeltaWeights, ChunkAttnConfig, ChunkAttnWeights, GLAConfig, GLAWeights, LatentAttnConfig,
                      LatentAttnWeights, WindowAttnConfig, WindowAttnWeights)

BF16, F32 = torch.bfloat16, torch.float32
DTYPE_CODE = {BF16: 0, F32: 1}
SILU, SIGMOID = 0, 1
MASK_WINDOW, MASK_CHUNK = 0, 1                                   # kinds of qd_attention_args
NORM_NONE, NORM_ROW, NORM_HEAD = 0, 1, 2
SINK_NONE, SINK_LEARNED, SINK_ZERO = 0, 1, 2
GATE_NONE, GATE_HEAD, GATE_VALUE = 0, 1, 2


def column(t: torch.Tensor, offset: int):
    """Address of a row's element ``offset`` (of the first row)."""
    return c_void_p(t.data_ptr() + offset * t.element_size())


def place(position) -> tuple:
    """(device pointer or NULL, host value) of a position."""
    return (ptr(position), 0) if isinstance(position, torch.Tensor) else (None, int(position))


def linear(x, x_column: int, ldx: int, weight, out, *, tokens: int, status, gelu_columns: int = 0, glu: bool = False, bias=None,
           add: bool = False, norm=None, norm_offset: float = 0.0, eps: float = 0.0) -> None:
    """out[t] = W x[t, x_column : x_column + in_features] (+ fp32 ``bias``); the first ``gelu_columns`` outputs through the exact
    GELU; ``glu``: weight rows 2i and 2i + 1 are a gate and its partner, out[i] = relu(gate) * partner; ``add``: onto
    what ``out`` holds; ``norm`` (a few tokens only): x / rms(x) * (norm_offset + norm) in the place of x."""
    call_hybrid("qd_linear", column(x, x_column), ldx, DTYPE_CODE[x.dtype], ptr(weight), ptr(out), out.shape[1],
                DTYPE_CODE[out.dtype], tokens, weight.shape[0], weight.shape[1], gelu_columns, int(glu), ptr(bias), int(add), ptr(norm),
                norm_offset, eps, ptr(status), stream_of(x))


def stack_rows(parts: dict[str, torch.Tensor]) -> tuple[torch.Tensor, dict[str, int]]:
    """The matrices of one input below one another, each starting at a multiple of eight rows (an output
    column on a 16-byte boundary), and the first row of each."""
    rows, at, blocks = 0, {}, []
    for name, part in parts.items():
        at[name] = rows
        pad = -part.shape[0] % 8
        blocks += [part, part.new_zeros((pad, *part.shape[1:]))] if pad else [part]
        rows += part.shape[0] + pad
    return torch.cat(blocks).contiguous(), at


def frequencies(base: float, dims: int, device) -> torch.Tensor:
    """base^(-2i / dims) as fp32 high and low parts: an angle keeps fp32 accuracy at any position."""
    exact = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    high = exact.to(F32)
    return torch.stack([high, (exact - high.double()).to(F32)]).contiguous().to(device)


def ring_segments(first: int, count: int, capacity: int) -> list[tuple[int, int]]:
    """(row, rows) of the positions first .. first + count - 1 in a ring, in order."""
    row = first % capacity
    head = min(count, capacity - row)
    return [(row, head)] + ([(0, count - head)] if count > head else [])


def step_covers(m) -> bool:
    """Whether the one-launch decode form of a recurrence takes these sizes (a cluster of at most eight blocks of 32 value columns)."""
    return m.vdim <= 256


class GroupedAttention:
    """Grouped-query attention over a bounded span of positions; ``constants`` are fields of ``qd_attention_args``."""
    inner = ()                                                  # matrices between the input and the output projections
    KEYS_PER_SPLIT, MAX_SPLITS = 32, 64

    def __init__(self, m, eps: float, device, tensors: dict, **constants):
        self.m, self.tensors = m, tensors                       # the arguments hold addresses only
        self.out_columns = m.heads * m.vdim
        sms = torch.cuda.get_device_properties(device).multi_processor_count
        self.splits = max(1, min(-(-m.span // self.KEYS_PER_SPLIT), -(-2 * sms // m.kv_heads), self.MAX_SPLITS))
        self.partial = torch.empty(size_hybrid("qd_attention_step_floats", m.heads, m.vdim, self.splits), dtype=F32, device=device)
        self.counters = torch.zeros(m.kv_heads, dtype=torch.int32, device=device)
        self.args = AttentionArgs(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, eps=eps, ld_k=m.kv_heads * m.dim,
                                  ld_v=m.kv_heads * m.vdim, partial=ptr(self.partial), counters=ptr(self.counters),
                                  **{name: ptr(t) for name, t in tensors.items()}, **constants)

    def _bind(self, proj, at, history: LayerHistory, position):
        a, capacity = self.args, history.k.shape[0]
        a.q, a.k, a.v = (column(proj, at[name]) for name in "qkv")
        if "g" in at and a.gate_kind != GATE_NONE:
            a.gate = column(proj, at["g"])
        a.k_cache, a.v_cache, a.capacity, a.span = ptr(history.k), ptr(history.v), capacity, min(self.m.span, capacity)
        a.ld = a.ld_gate = proj.shape[1]
        a.position_ptr, a.position = place(position)
        a.tokens, a.dtype, a.splits = proj.shape[0], DTYPE_CODE[proj.dtype], self.splits
        out = torch.empty((a.tokens, self.out_columns), dtype=proj.dtype, device=proj.device)
        queries = torch.empty((a.tokens, self.m.heads * self.m.dim), dtype=proj.dtype, device=proj.device)
        a.out, a.q_rows = ptr(out), ptr(queries)
        return out, queries                                     # the queries live until the launch

    def chunk(self, proj, at, history: LayerHistory, position, status):
        out, queries = self._bind(proj, at, history, position)
        call_hybrid("qd_attention", byref(self.args), stream_of(proj))
        return out

    def step(self, proj, at, history: LayerHistory, position, status):
        out, queries = self._bind(proj, at, history, position)
        call_hybrid("qd_attention_step", byref(self.args), stream_of(proj))
        return out


class WindowAttention(GroupedAttention):
    """Sliding window, learned sinks, norms over the whole projections, interleaved rotation, a gate per head."""

    def __init__(self, weights: WindowAttnWeights, m: WindowAttnConfig, eps: float, device):
        self.w, self.freq = weights, frequencies(m.rotary_base, m.rotary_dims, device)
        self.projections = {"q": weights.q, "k": weights.k, "v": weights.v, "g": weights.g}
        super().__init__(m, eps, device, {"q_norm": weights.q_norm, "k_norm": weights.k_norm, "sink": weights.sink, "freq": self.freq},
                         rot=m.rotary_dims, norm=NORM_ROW, sink_kind=SINK_LEARNED, gate_kind=GATE_HEAD, mask=MASK_WINDOW)


class ChunkAttention(GroupedAttention):
    """Chunks counted from position 0, a penalty on the distance, one added to the denominator, norms per head."""

    def __init__(self, weights: ChunkAttnWeights, m: ChunkAttnConfig, eps: float, device):
        self.w, self.slopes = weights, torch.tensor(m.slopes(), dtype=F32, device=device)
        self.projections = {"q": weights.q, "k": weights.k, "v": weights.v}
        self.biases = {"q": weights.q_b, "k": weights.k_b, "v": weights.v_b}
        super().__init__(m, eps, device, {"q_norm": weights.q_norm, "k_norm": weights.k_norm, "slopes": self.slopes}, norm=NORM_HEAD,
                         sink_kind=SINK_ZERO, gate_kind=GATE_NONE, mask=MASK_CHUNK)


class LatentAttention:
    """Latent attention in a sliding window with a gate per value column.  The cache holds latents.  A chunk expands the
    visible ones into keys and values; one token works on the latents (the expansions move to its query and to its result)."""
    KEYS_PER_SPLIT, MAX_SPLITS, HEADS_PER_BLOCK = 32, 64, 16

    def __init__(self, weights: LatentAttnWeights, m: LatentAttnConfig, eps: float, device):
        self.w, self.m, self.eps, self.freq = weights, m, eps, frequencies(m.rotary_base, m.rot_dim, device)
        self.projections = {"dq": weights.dq, "dkv": weights.dkv, "g": weights.g}
        self.out_columns = m.heads * m.vdim
        self.expand, self.expand_at = stack_rows({"k": weights.uk, "v": weights.uv})
        self.inner = (weights.uq, self.expand)
        sms = torch.cuda.get_device_properties(device).multi_processor_count
        blocks = -(-m.heads // self.HEADS_PER_BLOCK)
        self.splits = max(1, min(-(-m.span // self.KEYS_PER_SPLIT), -(-sms // blocks), self.MAX_SPLITS))
        self.partial = torch.empty(size_hybrid("qd_latent_step_floats", m.heads, m.kv_rank, self.splits), dtype=F32, device=device)
        self.absorbed = torch.empty((m.heads, m.row), dtype=F32, device=device)
        self.latent = LatentArgs(
            heads=m.heads, dim=m.dim, rot=m.rot_dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, rot_column=m.rot_column, ld_cache=m.row,
            scale=m.scale, eps=eps, dq_norm=ptr(weights.dq_norm), dkv_norm=ptr(weights.dkv_norm), freq=ptr(self.freq),
            uk=ptr(self.expand), uv=c_void_p(self.expand.data_ptr() + self.expand_at["v"] * self.expand.stride(0) * self.expand.element_size()),
            partial=ptr(self.partial), absorbed=ptr(self.absorbed))
        # a chunk's attention: the heads' own key columns from the expansion, the shared ones from the cache
        self.args = AttentionArgs(heads=m.heads, kv_heads=m.heads, dim=m.dim, vdim=m.vdim, shared_dim=m.rot_dim, scale=m.scale, eps=eps,
                                  norm=NORM_NONE, sink_kind=SINK_NONE, gate_kind=GATE_VALUE, mask=MASK_WINDOW,
                                  ld_k=self.expand.shape[0], ld_v=self.expand.shape[0], ld_shared=m.row)

    def _bind(self, proj, at, history: LayerHistory, position):
        a, capacity = self.latent, history.latent.shape[0]
        a.dq, a.dkv, a.gate = (column(proj, at[name]) for name in ("dq", "dkv", "g"))
        a.ld, a.cache, a.capacity, a.span = proj.shape[1], ptr(history.latent), capacity, min(self.m.span, capacity)
        a.position_ptr, a.position = place(position)
        a.tokens, a.dtype, a.splits = proj.shape[0], DTYPE_CODE[proj.dtype], self.splits

    def _prepare(self, proj):
        """The normed query latents; the cache rows are written too."""
        normed = torch.empty((proj.shape[0], self.m.q_rank), dtype=proj.dtype, device=proj.device)
        self.latent.q_latent = ptr(normed)
        call_hybrid("qd_latent_prepare", byref(self.latent), stream_of(proj))
        return normed

    def chunk(self, proj, at, history: LayerHistory, position: int, status):
        m, tokens, dev = self.m, proj.shape[0], proj.device
        self._bind(proj, at, history, position)
        a, capacity = self.args, history.latent.shape[0]
        queries = torch.empty((tokens, m.heads * (m.dim + m.rot_dim)), dtype=proj.dtype, device=dev)
        linear(self._prepare(proj), 0, m.q_rank, self.w.uq, queries, tokens=tokens, status=status)
        call_hybrid("qd_rotate_half", ptr(queries), ptr(self.freq), *place(position), tokens, m.heads, m.dim + m.rot_dim, m.rot_dim,
                    DTYPE_CODE[proj.dtype], stream_of(proj))
        first = max(0, position - m.span + 1)
        expanded = torch.empty((capacity, self.expand.shape[0]), dtype=proj.dtype, device=dev)
        for row, rows in ring_segments(first, position + tokens - first, capacity):
            linear(history.latent[row:], 0, m.row, self.expand, expanded[row:], tokens=rows, status=status)
        out = torch.empty((tokens, self.out_columns), dtype=proj.dtype, device=dev)
        a.gate, a.ld_gate, a.k_cache, a.v_cache = column(proj, at["g"]), proj.shape[1], ptr(expanded), column(expanded, self.expand_at["v"])
        a.k_shared, a.capacity, a.span = column(history.latent, m.rot_column), capacity, min(m.span, capacity)
        a.position, a.tokens, a.dtype, a.q_rows, a.out = position, tokens, DTYPE_CODE[proj.dtype], ptr(queries), ptr(out)
        call_hybrid("qd_attention", byref(a), stream_of(proj))
        return out

    def step(self, proj, at, history: LayerHistory, position, status):
        m, dev = self.m, proj.device
        self._bind(proj, at, history, position)
        query = torch.empty((1, m.heads * (m.dim + m.rot_dim)), dtype=proj.dtype, device=dev)
        if m.q_rank % 8 == 0:
            linear(proj, at["dq"], proj.shape[1], self.w.uq, query, tokens=1, status=status, norm=self.w.dq_norm, eps=self.eps)
        else:
            linear(self._prepare(proj), 0, m.q_rank, self.w.uq, query, tokens=1, status=status)
        out = torch.empty((1, self.out_columns), dtype=proj.dtype, device=dev)
        self.latent.q, self.latent.out = ptr(query), ptr(out)
        call_hybrid("qd_latent_step", byref(self.latent), stream_of(proj))
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


MIXERS = {WindowAttnConfig: WindowAttention, GLAConfig: GatedLinearAttention, ChannelDeltaConfig: ChannelDelta,
          ChunkAttnConfig: ChunkAttention, LatentAttnConfig: LatentAttention}
