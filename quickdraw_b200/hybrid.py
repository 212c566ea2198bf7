"""The bf16-weight designs on the device: one object that advances a ``HybridState`` over a chunk of
prompt tokens or over one token (the step callable of the engine).

``HybridModel`` holds what they share; a design is a subclass that runs the layers.  The residual stream is
fp32.  ``dtype`` float32 runs the same kernels with fp32 activations (weights stay bf16, which is what the
checkpoint holds).

``FezopelModel``, per sublayer: ONE product for everything that reads the normed input (the mixer's projections, or
the up projection with its GELU, and the residual gate), the mixer, the output product, and one launch that
closes the sublayer (gate, norm, residual sum, depth average, next norm).

``DokulixModel``, per sublayer of a chunk: one product for everything that reads the normed input (the mixer's
projections with their biases, or gate and up with the gated unit in the epilogue), the mixer, the output product,
and one launch for the residual sum and the next norm.  One token needs no launches for norms and sums: a product
norms its input row itself and the output products add to the stream.
"""

from __future__ import annotations

import torch

from ._lib import call_hybrid, ptr, stream_of
from .mixers import BF16, DTYPE_CODE, F32, MIXERS, column, linear, stack_rows
from .state import HybridState
from .weights import DokulixCheckpoint, FezopelCheckpoint

GREEDY_BLOCKS = 128


class _Sublayer:
    """Stacked input matrix of a sublayer, where its parts are, the output matrix and what surrounds it."""

    def __init__(self, parts, out, around, gelu_columns: int = 0):
        self.matrix, self.at = stack_rows({**parts, "gate": around.gate})
        self.out, self.around, self.gelu_columns = out, around, gelu_columns


class HybridModel:
    """``__call__(ckpt, token, position, state)`` is the engine's step; ``run`` is a chunk of tokens."""

    def __init__(self, ckpt, dtype: torch.dtype = BF16):
        assert dtype in DTYPE_CODE
        self.ckpt, self.dtype, self.device = ckpt, dtype, ckpt.embed_tokens.device
        c = ckpt.config
        self.mixers = [MIXERS[type(cfg.mixer)](layer.mixer, cfg.mixer, c.norm_eps, self.device) for layer, cfg in zip(ckpt.layers, c.layers)]
        self.status = torch.zeros(1, dtype=torch.int32, device=self.device)
        self.next_token = torch.zeros((), dtype=torch.long, device=self.device)
        self._keys = torch.empty(GREEDY_BLOCKS, dtype=torch.int64, device=self.device)
        self._counter = torch.zeros(1, dtype=torch.int32, device=self.device)

    def _rows(self, tokens, columns, dtype=None):
        return torch.empty((tokens, columns), dtype=dtype or self.dtype, device=self.device)

    def _layers(self, token_ids, position, state: HybridState, tokens: int, finish: bool, record=None):
        """All layers; the stream after the last one.  ``finish`` False: stop behind the last mixer (no more state is
        written).  ``record`` receives a copy of the stream after every layer run."""
        raise NotImplementedError

    def _head(self, stream, rows=None):
        """fp32 logits of the given rows of the stream (all without ``rows``)."""
        raise NotImplementedError

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

    def products(self) -> list[torch.Tensor]:
        """The matrices a token is multiplied with, logits aside (a looped layer's once per pass)."""
        raise NotImplementedError

    def check(self) -> int:
        """Status word of the tensor-core products (0 = clean)."""
        return int(self.status.item())


class FezopelModel(HybridModel):
    def __init__(self, ckpt: FezopelCheckpoint, dtype: torch.dtype = BF16):
        super().__init__(ckpt, dtype)
        self.mix, self.mlp = [], []
        for layer, cfg, mixer in zip(ckpt.layers, ckpt.config.layers, self.mixers):
            self.mix.append(_Sublayer(mixer.projections, layer.mixer.o, layer.around_mixer))
            self.mlp.append(None if layer.mlp is None else
                            _Sublayer({"up": layer.mlp.up}, layer.mlp.down, layer.around_mlp, gelu_columns=cfg.ff))

    def products(self):
        return [m for sub in self.mix + self.mlp if sub is not None for m in (sub.matrix, sub.out)]

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
        c, norm = self.ckpt.config, self.ckpt.final_norm
        count = stream.shape[0] if rows is None else rows.numel()
        normed = self._rows(count, c.hidden_size)
        call_hybrid("qd_layer_norm_rows", ptr(stream), ptr(rows), ptr(norm.w), ptr(norm.b), ptr(normed), count, c.hidden_size, c.norm_eps,
                    DTYPE_CODE[self.dtype], stream_of(stream))
        logits = self._rows(count, c.vocab_size, F32)
        linear(normed, 0, c.hidden_size, self.ckpt.lm_head, logits, tokens=count, status=self.status)
        return logits


class _PreNorm:
    """Weights of a pre-norm layer as its launches take them: stacked input matrices, fp32 biases."""

    def __init__(self, layer, mixer):
        self.matrix, self.at = stack_rows(mixer.projections)
        biases = getattr(mixer, "biases", None)
        self.bias = None if biases is None else stack_rows(biases)[0].float()
        out_bias = getattr(layer.mixer, "o_b", None)
        self.out, self.out_bias = layer.mixer.o, None if out_bias is None else out_bias.float()
        self.norm1, self.norm2, mlp = layer.norm1, layer.norm2, layer.mlp
        self.glu = None if mlp is None else torch.stack([mlp.gate, mlp.up], 1).flatten(0, 1).contiguous()      # rows in pairs
        self.down = None if mlp is None else mlp.down


class DokulixModel(HybridModel):
    def __init__(self, ckpt: DokulixCheckpoint, dtype: torch.dtype = BF16):
        super().__init__(ckpt, dtype)
        c = ckpt.config
        self.parts = [_PreNorm(layer, mixer) for layer, mixer in zip(ckpt.layers, self.mixers)]
        self.runs = c.runs()
        self.steps = [None if t is None else ckpt.loop_steps[t] for _, t in self.runs]      # added in front of a run
        # one token: what the last product of a run adds besides its result, its bias and the next run's vector
        self.closing = []
        for r, (i, _) in enumerate(self.runs):
            bias = self.parts[i].out_bias if self.parts[i].glu is None else None
            step = self.steps[r + 1] if r + 1 < len(self.runs) else None
            self.closing.append(bias if step is None else step.float() if bias is None else bias + step.float())
        self.folded = c.hidden_size % 8 == 0          # whether one token's products can take the stream itself

    def products(self):
        parts = [(self.parts[i], self.mixers[i]) for i, _ in self.runs]
        return [m for part, mixer in parts for m in (part.matrix, part.out, *mixer.inner, part.glu, part.down) if m is not None]

    def _stream(self, count, *, source=None, token_ids=None, index=None, y=None, step=None, out=None, norm=None, normed=None):
        """Stream rows: embedding rows of the tokens or rows of ``source``, + ``y``, + ``step``; their norm."""
        c = self.ckpt.config
        call_hybrid("qd_stream_norm", ptr(token_ids), None if token_ids is None else ptr(self.ckpt.embed_tokens), c.vocab_size, ptr(source), ptr(index),
                    ptr(y), ptr(step), ptr(out), ptr(norm), 1.0, ptr(normed), count, c.hidden_size, c.norm_eps, DTYPE_CODE[self.dtype],
                    stream_of(self.status))

    def _layers(self, token_ids, position, state: HybridState, tokens: int, finish: bool, record=None):
        if tokens == 1 and self.folded and record is None:
            return self._one_token(token_ids, position, state, finish)
        width, args = self.ckpt.config.hidden_size, dict(tokens=tokens, status=self.status)
        stream, normed, y = self._rows(tokens, width, F32), self._rows(tokens, width), self._rows(tokens, width)
        if not self.runs:
            self._stream(tokens, token_ids=token_ids, out=stream)
            return stream
        self._stream(tokens, token_ids=token_ids, step=self.steps[0], out=stream, norm=self.parts[self.runs[0][0]].norm1, normed=normed)
        for r, (i, _) in enumerate(self.runs):
            part, mixer, last = self.parts[i], self.mixers[i], r + 1 == len(self.runs)
            proj = self._rows(tokens, part.matrix.shape[0])
            linear(normed, 0, width, part.matrix, proj, bias=part.bias, **args)
            form = mixer.step if tokens == 1 else mixer.chunk
            core = form(proj, part.at, state.layers[r], position, self.status)
            if last and not finish:
                return None
            linear(core, 0, core.shape[1], part.out, y, bias=part.out_bias, **args)
            if part.glu is not None:
                self._stream(tokens, source=stream, y=y, out=stream, norm=part.norm2, normed=normed)
                hidden = self._rows(tokens, part.glu.shape[0] // 2)
                linear(normed, 0, width, part.glu, hidden, glu=True, **args)
                linear(hidden, 0, hidden.shape[1], part.down, y, **args)
            ahead = {} if last else dict(step=self.steps[r + 1], norm=self.parts[self.runs[r + 1][0]].norm1, normed=normed)
            if record is None:
                self._stream(tokens, source=stream, y=y, out=stream, **ahead)
            else:                                     # the sum before what comes ahead of the next run
                self._stream(tokens, source=stream, y=y, out=stream)
                record.append(stream.clone())
                if not last:
                    self._stream(tokens, source=stream, out=stream, **ahead)
        return stream

    def _one_token(self, token_id, position, state: HybridState, finish: bool):
        c = self.ckpt.config
        width, args = c.hidden_size, dict(tokens=1, status=self.status)
        folded = dict(norm_offset=1.0, eps=c.norm_eps)
        stream = self._rows(1, width, F32)
        self._stream(1, token_ids=token_id, step=self.steps[0] if self.steps else None, out=stream)
        for r, (i, _) in enumerate(self.runs):
            part = self.parts[i]
            proj = self._rows(1, part.matrix.shape[0])
            linear(stream, 0, width, part.matrix, proj, bias=part.bias, norm=part.norm1, **folded, **args)
            core = self.mixers[i].step(proj, part.at, state.layers[r], position, self.status)
            if r + 1 == len(self.runs) and not finish:
                return None
            linear(core, 0, core.shape[1], part.out, stream, add=True, bias=self.closing[r] if part.glu is None else part.out_bias, **args)
            if part.glu is not None:
                hidden = self._rows(1, part.glu.shape[0] // 2)
                linear(stream, 0, width, part.glu, hidden, glu=True, norm=part.norm2, **folded, **args)
                linear(hidden, 0, hidden.shape[1], part.down, stream, add=True, bias=self.closing[r], **args)
        return stream

    def _head(self, stream, rows=None):
        c, norm = self.ckpt.config, self.ckpt.final_norm
        count = stream.shape[0] if rows is None else rows.numel()
        logits = self._rows(count, c.vocab_size, F32)
        if stream.shape[0] == count == 1 and self.folded:
            linear(stream, 0, c.hidden_size, self.ckpt.lm_head, logits, tokens=1, status=self.status, norm=norm, norm_offset=1.0, eps=c.norm_eps)
            return logits
        normed = self._rows(count, c.hidden_size)
        self._stream(count, source=stream, index=rows, norm=norm, normed=normed)
        linear(normed, 0, c.hidden_size, self.ckpt.lm_head, logits, tokens=count, status=self.status)
        return logits
