"""Per-request history buffers (reference: quickdraw/kvcache/state.py:8-20).

Shapes (reference: quickdraw/engine/engine.py:43-59):
  kv_k, kv_v  bf16 [full_attention_layers, max_context, kv_heads, head_dim]
  rec_state   fp32 [linear_layers, value_heads, key_dim, value_dim]
  conv_state  bf16 [linear_layers, conv_channels, conv_width - 1], oldest tap first
``position`` counts processed tokens; the engine advances it, the step never does.

``HybridState`` is the same for models whose layers have caches and states of different sizes:
flat buffers with one view per layer, windowed key/value rings instead of a full-length cache.
"""

from dataclasses import dataclass

import torch


def _same_request_buffers(state):
    """A state of the same shapes whose histories are empty (the buffers of a warm-up run)."""
    return (torch.empty_like(state.kv_k), torch.empty_like(state.kv_v), torch.zeros_like(state.rec_state),
            torch.zeros_like(state.conv_state))


@dataclass
class DecodeState:
    kv_k: torch.Tensor
    kv_v: torch.Tensor
    rec_state: torch.Tensor
    conv_state: torch.Tensor
    position: int

    def memory_bytes(self) -> dict[str, int]:
        return {name: getattr(self, name).nbytes
                for name in ("kv_k", "kv_v", "rec_state", "conv_state")}

    keeps_every_row = True       # cache rows of processed positions stay until another request rewrites them

    def blank(self) -> "DecodeState":
        return DecodeState(*_same_request_buffers(self), 0)

    def history(self) -> list[torch.Tensor]:
        """What a snapshot copies: everything that later tokens of the request overwrite."""
        return [self.rec_state, self.conv_state]

    @classmethod
    def allocate(cls, config, max_context: int, device) -> "DecodeState":
        full = config.layer_types.count("full_attention")
        linear = config.layer_types.count("linear_attention")
        kv_shape = (full, max_context, config.num_key_value_heads, config.head_dim)
        return cls(
            kv_k=torch.empty(kv_shape, dtype=torch.bfloat16, device=device),
            kv_v=torch.empty(kv_shape, dtype=torch.bfloat16, device=device),
            rec_state=torch.zeros(
                (linear, config.linear_num_value_heads, config.linear_key_head_dim,
                 config.linear_value_head_dim), dtype=torch.float32, device=device),
            conv_state=torch.zeros(
                (linear, config.conv_channels, config.linear_conv_kernel_dim - 1),
                dtype=torch.bfloat16, device=device),
            position=0)


@dataclass
class LayerHistory:
    """One layer's views: ``k``, ``v`` [capacity, kv_heads, dim / vdim] (attention), ``latent`` [capacity, row]
    (latent attention), ``rec`` fp32 [heads, dim, vdim], ``conv`` [taps, channels] (position p in row p mod taps)."""
    k: torch.Tensor | None = None
    v: torch.Tensor | None = None
    latent: torch.Tensor | None = None
    rec: torch.Tensor | None = None
    conv: torch.Tensor | None = None


class HybridState:
    """History of one request of a bf16-weight hybrid, one entry of ``layers`` for every layer run (a looped layer
    has one per pass).  An attention layer keeps the last ``capacity`` positions, position p in row p mod
    capacity: the span a query sees plus the rows a prompt chunk of ``chunk`` tokens adds before its first
    token has attended.  Rows are only read for positions of the current request, so a reset leaves them."""

    keeps_every_row = False

    def __init__(self, config, max_context: int, device, chunk: int = 2048, dtype: torch.dtype = torch.bfloat16):
        self._args = (config, max_context, device, chunk, dtype)
        self.position = 0
        plans, sizes = [], {"kv_k": 0, "kv_v": 0, "rec_state": 0, "conv_state": 0}

        def take(buffer: str, *shape: int):
            start, count = sizes[buffer], 1
            for n in shape:
                count *= n
            sizes[buffer] += -(-count // 64) * 64            # every view starts on a 128-byte boundary
            return buffer, start, count, shape

        for index, _ in config.runs():
            m, plan = config.layers[index].mixer, {}
            capacity = min(max_context, m.span - 1 + chunk) if hasattr(m, "span") else 0
            if hasattr(m, "kv_rank"):
                plan["latent"] = take("kv_k", capacity, m.row)
            elif hasattr(m, "span"):
                plan["k"] = take("kv_k", capacity, m.kv_heads, m.dim)
                plan["v"] = take("kv_v", capacity, m.kv_heads, m.vdim)
            else:
                plan["rec"] = take("rec_state", m.heads, m.dim, m.vdim)
                if hasattr(m, "conv"):
                    plan["conv"] = take("conv_state", m.conv, 2 * m.kv_heads * m.dim + m.heads * m.vdim)
            plans.append(plan)
        for buffer, size in sizes.items():
            fresh = torch.empty if buffer.startswith("kv") else torch.zeros
            kind = torch.float32 if buffer == "rec_state" else dtype
            setattr(self, buffer, fresh(size, dtype=kind, device=device))
        self.layers = [LayerHistory(**{name: getattr(self, buffer)[start:start + count].view(shape)
                                       for name, (buffer, start, count, shape) in plan.items()}) for plan in plans]

    def blank(self) -> "HybridState":
        return HybridState(*self._args)

    def history(self) -> list[torch.Tensor]:
        return [self.rec_state, self.conv_state, self.kv_k, self.kv_v]

    def memory_bytes(self) -> dict[str, int]:
        return {name: getattr(self, name).nbytes for name in ("kv_k", "kv_v", "rec_state", "conv_state")}
