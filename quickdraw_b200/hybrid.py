"""The bf16-weight hybrids on the device: one object that advances a ``HybridState`` over a chunk of
prompt tokens or over one token (the step callable of the engine).

Per sublayer: ONE product for everything that reads the normed input (the mixer's projections, or
the up projection with its GELU, and the residual gate), the mixer, the output product, and one launch that
closes the sublayer (gate, norm, residual sum, depth average, next norm).  The residual stream and the
layer results that the depth average needs are fp32.  ``dtype`` float32 runs the same kernels with fp32
activations (weights stay bf16, which is what the checkpoint holds).
"""

from __future__ import annotations

import torch

from ._lib import call_hybrid, ptr, stream_of
from .mixers import BF16, DTYPE_CODE, F32, MIXERS, column, linear
from .state import HybridState
from .weights import FezopelCheckpoint

GREEDY_BLOCKS = 128


def stack_rows(parts: dict[str, torch.Tensor]) -> tuple[torch.Tensor, dict[str, int]]:
    """The matrices of one input below one another, each starting at a multiple of eight rows (an output
    column on a 16-byte boundary), and the first row of each."""
    rows, at, blocks = 0, {}, []
    for name, part in parts.items():
        at[name] = rows
        pad = -part.shape[0] % 8
        blocks += [part, part.new_zeros((pad, part.shape[1]))] if pad else [part]
        rows += part.shape[0] + pad
    return torch.cat(blocks).contiguous(), at


class _Sublayer:
    """Stacked input matrix of a sublayer, where its parts are, the output matrix and what surrounds it."""

    def __init__(self, parts, out, around, gelu_columns: int = 0):
        self.matrix, self.at = stack_rows({**parts, "gate": around.gate})
        self.out, self.around, self.gelu_columns = out, around, gelu_columns


class HybridModel:
    """``__call__(ckpt, token, position, state)`` is the engine's step; ``run`` is a chunk of tokens."""

    def __init__(self, ckpt: FezopelCheckpoint, dtype: torch.dtype = BF16):
        assert dtype in DTYPE_CODE
        self.ckpt, self.dtype, self.device = ckpt, dtype, ckpt.embed_tokens.device
        c = ckpt.config
        self.mixers, self.mix, self.mlp = [], [], []
        for layer, cfg in zip(ckpt.layers, c.layers):
            mixer = MIXERS[type(cfg.mixer)](layer.mixer, cfg.mixer, c.norm_eps, self.device)
            self.mixers.append(mixer)
            self.mix.append(_Sublayer(mixer.projections, layer.mixer.o, layer.around_mixer))
            self.mlp.append(None if layer.mlp is None else
                            _Sublayer({"up": layer.mlp.up}, layer.mlp.down, layer.around_mlp, gelu_columns=cfg.ff))
        self.status = torch.zeros(1, dtype=torch.int32, device=self.device)
        self.next_token = torch.zeros((), dtype=torch.long, device=self.device)
        self._keys = torch.empty(GREEDY_BLOCKS, dtype=torch.int64, device=self.device)
        self._counter = torch.zeros(1, dtype=torch.int32, device=self.device)

    # ------------------------------------------------------------------ building blocks
    def _rows(self, tokens, columns, dtype=None):
        return torch.empty((tokens, columns), dtype=dtype or self.dtype, device=self.device)

    def _project(self, sub: _Sublayer, normed):
        out = self._rows(normed.shape[0], sub.matrix.shape[0])
        linear(normed, 0, normed.shape[1], sub.matrix, out, tokens=normed.shape[0], status=self.status, gelu_columns=sub.gelu_columns)
        return out

    def _close(self, sub: _Sublayer, proj, y, source, stream, normed, following, results=None, depth=None, older=-1):
        """End of a sublayer: ``stream`` from ``source`` (may be the same) and, if ``following`` is a norm, normed."""
        c, tokens = self.ckpt.config, y.shape[0]
        stride = 0 if results is None else results.stride(0)
        call_hybrid("qd_sublayer_close", ptr(y), column(proj, sub.at["gate"]), proj.shape[1], ptr(sub.around.gate_b),
                    ptr(sub.around.post.w), ptr(sub.around.post.b), ptr(source), ptr(stream), ptr(results), stride, ptr(depth), older,
                    ptr(following.w) if following else None, ptr(following.b) if following else None, ptr(normed), tokens,
                    c.hidden_size, c.norm_eps, DTYPE_CODE[self.dtype], stream_of(y))

    def _layers(self, token_ids, position, state: HybridState, tokens: int, finish: bool, record=None):
        """All layers; the stream after the last one.  ``finish`` False: stop behind the last mixer (no more state is
        written).  ``record`` receives a copy of the stream after every layer."""
        c, layers = self.ckpt.config, self.ckpt.layers
        width = c.hidden_size
        # embedding output and layer results of this chunk, for the depth average
        results = torch.empty((len(layers) + 1, tokens, width), dtype=F32, device=self.device)
        source, stream = results[0], self._rows(tokens, width, F32)
        normed = self._rows(tokens, width)
        first = layers[0].around_mixer.norm
        call_hybrid("qd_embed_norm", ptr(token_ids), ptr(self.ckpt.embed_tokens), c.vocab_size, ptr(source), ptr(first.w), ptr(first.b),
                    ptr(normed), tokens, width, c.norm_eps, DTYPE_CODE[self.dtype], stream_of(results))
        for i, layer in enumerate(layers):
            mixer, sub, mlp = self.mixers[i], self.mix[i], self.mlp[i]
            proj = self._project(sub, normed)
            form = mixer.step if tokens == 1 else mixer.chunk
            core = form(proj, sub.at, state.layers[i], position, self.status)
            last = i + 1 == len(layers)
            if last and not finish:
                return None
            y = self._rows(tokens, width)
            linear(core, 0, core.shape[1], sub.out, y, tokens=tokens, status=self.status)
            following = None if last else layers[i + 1].around_mixer.norm
            ending = dict(results=results, depth=layer.depth, older=i + 1)
            if mlp is None:
                self._close(sub, proj, y, source, stream, normed, following, **ending)
            else:
                self._close(sub, proj, y, source, stream, normed, mlp.around.norm)
                hidden = self._project(mlp, normed)
                linear(hidden, 0, hidden.shape[1], mlp.out, y, tokens=tokens, status=self.status)
                self._close(mlp, hidden, y, stream, stream, normed, following, **ending)
            source = stream
            if record is not None:
                record.append(stream.clone())
        return stream

    def _head(self, stream, rows=None):
        """fp32 logits of the given rows of the stream (all without ``rows``)."""
        c, norm = self.ckpt.config, self.ckpt.final_norm
        count = stream.shape[0] if rows is None else rows.numel()
        normed = self._rows(count, c.hidden_size)
        call_hybrid("qd_layer_norm_rows", ptr(stream), ptr(rows), ptr(norm.w), ptr(norm.b), ptr(normed), count, c.hidden_size, c.norm_eps,
                    DTYPE_CODE[self.dtype], stream_of(stream))
        logits = self._rows(count, c.vocab_size, F32)
        linear(normed, 0, c.hidden_size, self.ckpt.lm_head, logits, tokens=count, status=self.status)
        return logits

    # --------------------------------------------------------------------------- chunk, step
    @torch.inference_mode()
    def run(self, token_ids: torch.Tensor, position0: int, state: HybridState, want=None, record=None):
        """Advance ``state`` over the tokens at position0 ..; logits [len(want), vocab] of the wanted places among them."""
        assert token_ids.ndim == 1 and token_ids.dtype == torch.long and token_ids.is_cuda and token_ids.is_contiguous()
        stream = self._layers(token_ids, position0, state, token_ids.numel(), bool(want) or record is not None, record)
        if not want:
            return None
        rows = torch.tensor(list(want), dtype=torch.int32, device=self.device)
        assert 0 <= min(want) and max(want) < token_ids.numel()
        return self._head(stream, rows)

    @torch.inference_mode()
    def __call__(self, ckpt, token_id, position, state: HybridState, *, logits: bool = True):
        """One token; logits [vocab] fp32, the greedy choice in ``next_token``."""
        assert ckpt is self.ckpt and token_id.ndim == 0 and token_id.dtype == torch.long
        stream = self._layers(token_id, position, state, 1, logits)
        if not logits:
            return None
        out = self._head(stream)[0]
        call_hybrid("qd_greedy", ptr(out), out.numel(), ptr(self._keys), ptr(self._counter), ptr(self.next_token), stream_of(out))
        return out

    def check(self) -> int:
        """Status word of the tensor-core products (0 = clean)."""
        return int(self.status.item())
