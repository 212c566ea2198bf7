"""Throughput of the bf16-weight designs on random weights at sizes of real models' layers, beside the closest
model of this package at equal width, depth and vocabulary, and every kernel of the design beside the like kernel
of that model: ``python bench.py --model fezopel`` (beside the NVFP4 hybrid MoE), ``--model dokulix`` (beside Fezopel).

Kernels are timed inside CUDA graphs over operand sets that together exceed L2 (no host time in the
numbers); a fraction is algorithmic bytes or floating-point operations per second over the measured
copy bandwidth or bf16 product throughput.
"""

from __future__ import annotations

import json
import os
from ctypes import byref

import torch

from . import synthetic
from ._lib import HYBRID_LIBRARIES, call, call_hybrid, hybrid_lib, lib, ptr, stream_of
from .engine import Engine
from .mixers import BF16, F32, ChannelDelta, ChunkAttention, GatedLinearAttention, LatentAttention, WindowAttention, column, linear
from .state import LayerHistory
from .weights import (ChannelDeltaConfig, ChannelDeltaWeights, ChunkAttnConfig, ChunkAttnWeights, GLAConfig, GLAWeights, LatentAttnConfig,
                      LatentAttnWeights, LoopConfig, WindowAttnConfig, WindowAttnWeights)

L2_BYTES = 160e6


def graph_time(calls, reps: int = 5, chained: bool = True) -> float:
    """Seconds per call: ``calls`` (closures on different operands) captured into one graph, best of ``reps`` replays."""
    libraries = [lib(), *map(hybrid_lib, HYBRID_LIBRARIES)]
    old = [library.qd_set_chained_launches(int(chained)) for library in libraries]
    try:
        for fn in calls[:2]:
            fn()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for fn in calls:
                fn()
    finally:
        for library, before in zip(libraries, old):
            library.qd_set_chained_launches(before)
    graph.replay()
    best = float("inf")
    for _ in range(reps):
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        begin.record()
        graph.replay()
        end.record()
        torch.cuda.synchronize()
        best = min(best, begin.elapsed_time(end) * 1e-3 / len(calls))
    return best


def sets_for(bytes_per_set: float, least: int = 4, most: int = 64) -> int:
    return int(max(least, min(most, -(-L2_BYTES // bytes_per_set) + 1)))


class Cases:
    def __init__(self, device, hbm_gbs: float, tflops: float):
        self.device, self.hbm, self.tensor = device, hbm_gbs * 1e9, tflops * 1e12
        self.src = synthetic.Source(5, device)
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self.rows = []
        self.launches = 0

    def leg(self, calls, nbytes=0.0, flops=0.0):
        seconds = graph_time(calls)
        frac = max(nbytes / seconds / self.hbm, flops / seconds / self.tensor)
        return {"us": round(seconds * 1e6, 2), "frac": round(frac, 3)}

    def pair(self, name, own, like_name, like):
        a, b = self.leg(*own), self.leg(*like)
        self.rows.append({"kernel": name, **a, "like": like_name, "like_us": b["us"], "like_frac": b["frac"],
                          "times_as_far": round(b["frac"] / a["frac"], 2) if a["frac"] else None})

    def rnd(self, *shape, dtype=BF16, std=1.0):
        return (torch.randn(shape, device=self.device, dtype=F32) * std).to(dtype)

    # ------------------------------------------------------------------------ products
    def products(self, tokens, rows, width):
        flops = 2.0 * tokens * rows * width
        x = self.rnd(tokens, width)
        w, out = self.rnd(rows, width, std=width ** -0.5), self.rnd(tokens, rows)
        proj = self.src.nvfp4("w", rows, width)
        like = lambda: call("qd_nvfp4_matmul", ptr(x), ptr(proj.weight), ptr(proj.weight_scale), ptr(proj.weight_scale_2), ptr(out), tokens,
                            rows, width, 16, ptr(self.status), stream_of(x))
        own = lambda: linear(x, 0, width, w, out, tokens=tokens, status=self.status)
        self.pair(f"linear_umma_kernel {tokens} x [{rows}, {width}]", ([own] * 8, 0, flops), "nvfp4_gemm_kernel (W4A16)", ([like] * 8, 0, flops))

    def matvec(self, rows, width):
        own_bytes, like_bytes = rows * width * 2, rows * width * (0.5 + 1 / 16)
        x, out, out_like = self.rnd(1, width), self.rnd(1, rows, dtype=F32), self.rnd(rows)
        own, like = [], []
        for i in range(sets_for(own_bytes)):
            w = self.rnd(rows, width, std=width ** -0.5)
            own.append(lambda w=w: linear(x, 0, width, w, out, tokens=1, status=self.status))
        for i in range(sets_for(like_bytes)):
            p = self.src.nvfp4(f"w{i}", rows, width)
            like.append(lambda p=p: call("qd_nvfp4_gemv", ptr(x), ptr(p.weight), ptr(p.weight_scale), ptr(p.weight_scale_2), None, ptr(out_like),
                                         rows, width, 16, 0, stream_of(x)))
        self.pair(f"linear_rows_kernel 1 x [{rows}, {width}]", (own, own_bytes), "nvfp4 matvec (qd_nvfp4_gemv)", (like, like_bytes))

    # --------------------------------------------------------------------- recurrences
    def _gdn(self, tokens, hk, hv, d):
        channels = 2 * hk * d + hv * d
        return dict(mixed=self.rnd(tokens, channels), taps=self.rnd(channels, 4, std=0.5), conv=self.rnd(channels, 3),
                    a=self.rnd(tokens, hv), b=self.rnd(tokens, hv), a_log=self.rnd(hv), dt=self.rnd(hv), z=self.rnd(tokens, hv * d),
                    norm=self.rnd(d), rec=self.rnd(hv, d, d, dtype=F32, std=0.1))

    def _mixer(self, kind, heads, kv, d, rank, hidden=2048):
        w = lambda *s: self.rnd(*s, std=s[-1] ** -0.5)
        if kind == "gla":
            m = GLAConfig(heads=heads, dim=d, vdim=d, tau=16.0)
            weights = GLAWeights(q=None, k=None, v=None, g=None, o=None, a1=None, a2=w(heads * d, rank), a2_b=self.rnd(heads * d), norm=self.rnd(d))
            return GatedLinearAttention(weights, m, 1e-6, self.device), {"q": heads * d, "k": heads * d, "v": heads * d, "g": heads * d, "a1": rank}
        m = ChannelDeltaConfig(heads=heads, kv_heads=kv, dim=d, vdim=d, conv=4)
        weights = ChannelDeltaWeights(q=None, k=None, v=None, b=None, o=None, q_conv=w(kv * d, 4), k_conv=w(kv * d, 4), v_conv=w(heads * d, 4),
                                      A_log=self.rnd(heads), dt_bias=self.rnd(heads * d), a1=None, a2=w(heads * d, rank), g1=None,
                                      g2=w(heads * d, rank), norm=self.rnd(d))
        return ChannelDelta(weights, m, 1e-6, self.device), {"q": kv * d, "k": kv * d, "v": heads * d, "b": heads, "a1": rank, "g1": rank}

    def _laid_out(self, widths, tokens):
        at, total = {}, 0
        for name, width in widths.items():
            at[name] = total
            total += -(-width // 8) * 8
        return self.rnd(tokens, total), at

    def recurrences(self, tokens, heads, kv, d, rank):
        g = self._gdn(tokens, kv, heads, d)
        conv, core, gated = torch.empty_like(g["mixed"]), self.rnd(tokens, heads * d), self.rnd(tokens, heads * d)
        state_bytes = 2 * heads * d * d * 4
        scratch = torch.empty(lib().qd_seq_gdn_chunk_scratch_bytes(tokens, heads), dtype=torch.uint8, device=self.device)

        def like_walk():
            call("qd_seq_gdn_recurrence_chunked", ptr(conv), ptr(g["a"]), ptr(g["b"]), ptr(g["a_log"]), ptr(g["dt"]), ptr(g["rec"]), ptr(core),
                 tokens, kv, heads, d, d, ptr(scratch), stream_of(conv))

        def like_prepare():
            call("qd_seq_gdn_conv", ptr(g["mixed"]), ptr(g["taps"]), ptr(g["conv"]), ptr(conv), tokens, conv.shape[1], 4, stream_of(conv))

        like_prepare()
        walk_flops = 2.0 * 4 * tokens * heads * d * d
        fp32 = {n: self.rnd(tokens, w, dtype=F32, std=0.05) for n, w in
                (("q", kv * d), ("k", kv * d), ("v", heads * d), ("beta", heads), ("kq", 3 * kv))}
        fp32["g"] = -torch.rand(tokens, heads * d, device=self.device) * 0.1
        rec, raw = self.rnd(heads, d, d, dtype=F32, std=0.1), self.rnd(tokens, heads * d, dtype=F32)
        walk = lambda delta: lambda: call_hybrid("qd_linear_recurrence", ptr(fp32["q"]), ptr(fp32["k"]), ptr(fp32["g"]), ptr(fp32["v"]),
                                                 ptr(fp32["beta"]), ptr(fp32["kq"]), ptr(rec), ptr(raw), tokens, heads, kv, d, d, delta, stream_of(rec))
        like_bytes = tokens * (2 * kv * d + 2 * heads * d) * 2 + state_bytes
        own_bytes = tokens * (2 * kv * d + 3 * heads * d) * 4 + state_bytes
        self.pair(f"linear_recurrence_kernel delta, {tokens} tokens, {heads} heads of {d}", ([walk(1)] * 4, own_bytes), "gdn_chunk kernels",
                  ([like_walk] * 4, like_bytes))
        q_fp32 = {n: self.rnd(tokens, heads * d, dtype=F32, std=0.05) for n in "qk"}
        gla_walk = lambda: call_hybrid("qd_linear_recurrence", ptr(q_fp32["q"]), ptr(q_fp32["k"]), ptr(fp32["g"]), ptr(fp32["v"]), None, None,
                                       ptr(rec), ptr(raw), tokens, heads, heads, d, d, 0, stream_of(rec))
        self.pair(f"linear_recurrence_kernel gla, {tokens} tokens, {heads} heads of {d}",
                  ([gla_walk] * 4, tokens * 5 * heads * d * 4 + state_bytes), "gdn_chunk kernels", ([like_walk] * 4, like_bytes))
        # operands of a chunk
        mixer, widths = self._mixer("delta", heads, kv, d, rank)
        proj, at = self._laid_out(widths, tokens)
        hist = self.rnd(4, 2 * kv * d + heads * d)
        z = self.rnd(tokens, heads * d, dtype=F32)
        pos = torch.tensor(7, dtype=torch.int32, device=self.device)
        prepare = lambda: call_hybrid("qd_channel_delta_prepare", ptr(proj), ptr(proj), ptr(proj), ptr(proj), proj.shape[1], ptr(z),
                                      ptr(mixer.w.dt_bias), *mixer._convolution(LayerHistory(conv=hist)), ptr(pos), 0, ptr(fp32["q"]),
                                      ptr(fp32["k"]), ptr(fp32["g"]), ptr(fp32["v"]), ptr(fp32["beta"]), ptr(fp32["kq"]), tokens, heads, kv, d,
                                      d, 0, stream_of(proj))
        channels = 2 * kv * d + heads * d
        self.pair(f"delta_prepare_kernel {tokens} tokens", ([prepare] * 4, tokens * (channels * 6 + heads * d * 8)), "seq_gdn_conv",
                  ([like_prepare] * 4, tokens * channels * 4))
        gla_prepare = lambda: call_hybrid("qd_gla_prepare", ptr(proj), ptr(proj), ptr(proj), proj.shape[1], ptr(z), ptr(mixer.w.dt_bias), 16.0,
                                          ptr(q_fp32["q"]), ptr(q_fp32["k"]), ptr(fp32["g"]), ptr(fp32["v"]), tokens, heads, d, d, 0, stream_of(proj))
        self.pair(f"gla_prepare_kernel {tokens} tokens", ([gla_prepare] * 4, tokens * heads * d * (3 * 6 + 8)), "seq_gdn_conv",
                  ([like_prepare] * 4, tokens * channels * 4))
        out = self.rnd(tokens, heads * d)
        norm_gate = lambda: call_hybrid("qd_head_norm_gate", ptr(raw), ptr(g["norm"]), ptr(g["z"]), heads * d, ptr(out), tokens, heads, d, 1e-6, 1, 0,
                                        stream_of(raw))
        like_norm = lambda: call("qd_gdn_gated_norm", ptr(core), ptr(g["z"]), ptr(g["norm"]), ptr(gated), tokens * heads, d, 1e-6, stream_of(core))
        self.pair(f"head_norm_gate_kernel {tokens} tokens", ([norm_gate] * 4, tokens * heads * d * 8), "gdn_gated_norm",
                  ([like_norm] * 4, tokens * heads * d * 6))

    def recurrence_steps(self, heads, kv, d, rank):
        state_bytes = 2 * heads * d * d * 4
        n = sets_for(state_bytes / 2)
        g = self._gdn(1, kv, heads, d)
        recs = [self.rnd(heads, d, d, dtype=F32, std=0.1) for _ in range(n)]
        conv, core, gated = torch.empty_like(g["mixed"]), self.rnd(1, heads * d), self.rnd(1, heads * d)

        def like(rec):
            call("qd_gdn_conv", ptr(g["mixed"]), ptr(g["taps"]), ptr(g["conv"]), ptr(conv), conv.shape[1], 4, stream_of(conv))
            call("qd_gdn_recurrence", ptr(conv), ptr(g["a"]), ptr(g["b"]), ptr(g["a_log"]), ptr(g["dt"]), ptr(rec), ptr(core), kv, heads, d, d, 0,
                 stream_of(conv))
            call("qd_gdn_gated_norm", ptr(core), ptr(g["z"]), ptr(g["norm"]), ptr(gated), heads, d, 1e-6, stream_of(core))

        like_calls = [lambda r=r: like(r) for r in recs]
        pos = torch.tensor(7, dtype=torch.int32, device=self.device)
        for kind in ("delta", "gla"):
            mixer, widths = self._mixer(kind, heads, kv, d, rank)
            proj, at = self._laid_out(widths, 1)
            hist = self.rnd(4, 2 * kv * d + heads * d)
            calls = [lambda r=r: mixer.step(proj, at, LayerHistory(rec=r, conv=hist), pos, self.status) for r in recs]
            ranks = (2 if kind == "delta" else 1) * heads * d * rank * 2
            self.pair(f"recurrence_step_kernel {kind}, {heads} heads of {d}, rank {rank}", (calls, state_bytes + ranks),
                      "gdn conv + recurrence + gated norm", (like_calls, state_bytes))

    # ----------------------------------------------------------------------- attention
    def attention(self, tokens, heads, kv, d, window):
        m = WindowAttnConfig(heads=heads, kv_heads=kv, dim=d, vdim=d, window=window, rotary_dims=d // 4, rotary_base=1e7, scale=d ** -0.5)
        weights = WindowAttnWeights(q=None, k=None, v=None, g=None, o=None, q_norm=self.rnd(heads * d), k_norm=self.rnd(kv * d), sink=self.rnd(heads))
        mixer = WindowAttention(weights, m, 1e-6, self.device)
        widths = {"q": heads * d, "k": kv * d, "v": kv * d, "g": heads}
        proj, at = self._laid_out(widths, tokens)
        hist = LayerHistory(k=self.rnd(window + tokens, kv, d), v=self.rnd(window + tokens, kv, d))
        own = lambda: mixer.chunk(proj, at, hist, 0, self.status)
        seen = sum(min(window, i + 1) for i in range(tokens))
        qg, k, v = self.rnd(tokens, 2 * heads * d), self.rnd(tokens, kv * d), self.rnd(tokens, kv * d)
        norm = self.rnd(d)
        q_scratch, out = self.rnd(tokens, heads * d), self.rnd(tokens, heads * d)
        like = lambda: call("qd_seq_attention", ptr(qg), ptr(k), ptr(v), ptr(norm), ptr(norm), ptr(hist.k), ptr(hist.v), ptr(q_scratch), ptr(out),
                            tokens, 0, window + tokens, heads, kv, d, d // 4, 1e7, 1e-6, stream_of(qg))
        self.pair(f"attn_prepare + attn_flash, {tokens} tokens, window {window}, {heads}/{kv} heads of {d}",
                  ([own] * 4, 0, 4.0 * seen * heads * d), "seq_flash_attention (causal)",
                  ([like] * 4, 0, 4.0 * (tokens * (tokens + 1) / 2) * heads * d))

    def attention_step(self, heads, kv, d, window):
        m = WindowAttnConfig(heads=heads, kv_heads=kv, dim=d, vdim=d, window=window, rotary_dims=d // 4, rotary_base=1e7, scale=d ** -0.5)
        weights = WindowAttnWeights(q=None, k=None, v=None, g=None, o=None, q_norm=self.rnd(heads * d), k_norm=self.rnd(kv * d), sink=self.rnd(heads))
        mixer = WindowAttention(weights, m, 1e-6, self.device)
        proj, at = self._laid_out({"q": heads * d, "k": kv * d, "v": kv * d, "g": heads}, 1)
        nbytes = 2 * window * kv * d * 2
        caches = [(self.rnd(window, kv, d), self.rnd(window, kv, d)) for _ in range(sets_for(nbytes))]
        pos = torch.tensor(window - 1, dtype=torch.int32, device=self.device)
        own = [lambda c=c: mixer.step(proj, at, LayerHistory(k=c[0], v=c[1]), pos, self.status) for c in caches]
        qg, k, v, norm, out = self.rnd(2 * heads * d), self.rnd(kv * d), self.rnd(kv * d), self.rnd(d), self.rnd(heads * d)
        scratch = torch.empty(lib().qd_attn_scratch_floats(heads, kv, d, 32), dtype=F32, device=self.device)
        counters = torch.zeros(kv, dtype=torch.int32, device=self.device)
        like = [lambda c=c: call("qd_attn_decode", ptr(qg), ptr(k), ptr(v), ptr(norm), ptr(norm), ptr(c[0]), ptr(c[1]), ptr(out), ptr(scratch),
                                 ptr(counters), ptr(pos), 0, window, heads, kv, d, d // 4, 1e7, 1e-6, 32, 0, stream_of(qg)) for c in caches]
        self.pair(f"attn_step_kernel, window {window}, {heads}/{kv} heads of {d}", (own, nbytes), "attn_decode_kernel", (like, nbytes))

    # ------------------------------------------------------------------------ residual
    def residual(self, tokens, width, older):
        stride_sets = 1 if tokens > 64 else 8
        nbytes = tokens * width * (2 + 2 + 4 + 4 + 4 + 2 + 4 * older)
        vec = self.rnd(width)
        y, gate, normed, depth = self.rnd(tokens, width), self.rnd(tokens, width), self.rnd(tokens, width), self.rnd(older + 1)
        stream = self.rnd(tokens, width, dtype=F32)
        results = [self.rnd(older + 1, tokens, width, dtype=F32) for _ in range(stride_sets)]
        own = [lambda r=r: call_hybrid("qd_sublayer_close", ptr(y), ptr(gate), width, ptr(vec), ptr(vec), ptr(vec), ptr(stream), ptr(stream),
                                       ptr(r), r.stride(0), ptr(depth), older, ptr(vec), ptr(vec), ptr(normed), tokens, width, 1e-6, 0,
                                       stream_of(y)) for r in results for _ in range(4)]
        gamma = self.rnd(width, dtype=F32)
        four = [[self.rnd(tokens, width) for _ in range(4)] for _ in range(sets_for(tokens * width * 8))]
        like = [lambda f=f: call("qd_seq_add_rms_norm", ptr(f[0]), ptr(f[1]), ptr(gamma), ptr(f[2]), ptr(f[3]), tokens, width, 1e-6, stream_of(y))
                for f in four]
        self.pair(f"sublayer_close_kernel {tokens} x {width}, {older} earlier results", (own, nbytes), "seq_add_norm", (like, tokens * width * 8))


class LatentCases(Cases):
    """Kernels of the Dokulix design beside those of Fezopel."""

    def product_forms(self, tokens, rows, width):
        flops = 2.0 * tokens * rows * width
        x, w = self.rnd(tokens, width), self.rnd(rows, width, std=width ** -0.5)
        out, half, bias = self.rnd(tokens, rows), self.rnd(tokens, rows // 2), self.rnd(rows, dtype=F32)
        plain = lambda: linear(x, 0, width, w, out, tokens=tokens, status=self.status)
        glu = lambda: linear(x, 0, width, w, half, tokens=tokens, status=self.status, glu=True)
        biased = lambda: linear(x, 0, width, w, out, tokens=tokens, status=self.status, bias=bias)
        for name, own in (("gated unit", glu), ("bias", biased)):
            self.pair(f"linear_umma_kernel, {name}, {tokens} x [{rows}, {width}]", ([own] * 8, 0, flops), "linear_umma_kernel", ([plain] * 8, 0, flops))

    def matvec_forms(self, rows, width):
        nbytes = rows * width * 2
        x, stream, out, half = self.rnd(1, width), self.rnd(1, width, dtype=F32), self.rnd(1, rows), self.rnd(1, rows // 2)
        held, norm = self.rnd(1, rows, dtype=F32), self.rnd(width)
        ws = [self.rnd(rows, width, std=width ** -0.5) for _ in range(sets_for(nbytes))]
        one = dict(tokens=1, status=self.status)
        plain = [lambda w=w: linear(x, 0, width, w, out, **one) for w in ws]
        forms = {"norm": [lambda w=w: linear(stream, 0, width, w, out, norm=norm, norm_offset=1.0, eps=1e-6, **one) for w in ws],
                 "norm, gated unit": [lambda w=w: linear(stream, 0, width, w, half, norm=norm, norm_offset=1.0, eps=1e-6, glu=True, **one) for w in ws],
                 "added to the stream": [lambda w=w: linear(x, 0, width, w, held, add=True, **one) for w in ws]}
        for name, own in forms.items():
            self.pair(f"linear_rows_kernel, {name}, 1 x [{rows}, {width}]", (own, nbytes), "linear_rows_kernel", (plain, nbytes))

    def _window(self, heads, kv, d, window):
        m = WindowAttnConfig(heads=heads, kv_heads=kv, dim=d, vdim=d, window=window, rotary_dims=d, rotary_base=1e6, scale=d ** -0.5)
        weights = WindowAttnWeights(q=None, k=None, v=None, g=None, o=None, q_norm=self.rnd(heads * d), k_norm=self.rnd(kv * d), sink=self.rnd(heads))
        return WindowAttention(weights, m, 1e-6, self.device), {"q": heads * d, "k": kv * d, "v": kv * d, "g": heads}

    def _chunked(self, heads, kv, d, span):
        m = ChunkAttnConfig(heads=heads, kv_heads=kv, dim=d, vdim=d, span=span, scale=d ** -0.5)
        weights = ChunkAttnWeights(q=None, k=None, v=None, o=None, q_b=None, k_b=None, v_b=None, o_b=None, q_norm=self.rnd(d), k_norm=self.rnd(d))
        return ChunkAttention(weights, m, 1e-6, self.device), {"q": heads * d, "k": kv * d, "v": kv * d}

    def _latent(self, heads, d, rot, rank, window):
        m = LatentAttnConfig(heads=heads, dim=d, rot_dim=rot, vdim=d, q_rank=1536, kv_rank=rank, window=window, rotary_base=1e6, scale=(d + rot) ** -0.5)
        w = lambda *shape: self.rnd(*shape, std=shape[-1] ** -0.5)
        weights = LatentAttnWeights(dq=None, dkv=None, g=None, o=None, dq_norm=self.rnd(m.q_rank), dkv_norm=self.rnd(rank),
                                    uq=w(heads * (d + rot), m.q_rank), uk=w(heads * d, rank), uv=w(heads * d, rank))
        return LatentAttention(weights, m, 1e-6, self.device), {"dq": m.q_rank, "dkv": rank + rot, "g": heads * d}

    def attentions(self, tokens, heads, kv, d, rot, rank, span):
        """Prompt chunks from position 0."""
        seen, within = sum(min(span, i + 1) for i in range(tokens)), sum(i % span + 1 for i in range(tokens))
        kv_rows = lambda g: LayerHistory(k=self.rnd(span + tokens, g, d), v=self.rnd(span + tokens, g, d))

        def like(g):
            mixer, widths = self._window(heads, g, d, span)
            proj, at = self._laid_out(widths, tokens)
            return [lambda h=kv_rows(g): mixer.chunk(proj, at, h, 0, self.status)] * 4, 0, 4.0 * seen * heads * d
        mixer, widths = self._chunked(heads, kv, d, span)
        proj, at = self._laid_out(widths, tokens)
        hist = kv_rows(kv)
        self.pair(f"attn_prepare + attn_flash, {tokens} tokens, chunks of {span}, {heads}/{kv} heads of {d}",
                  ([lambda: mixer.chunk(proj, at, hist, 0, self.status)] * 4, 0, 4.0 * within * heads * d), f"the same, window {span}", like(kv))
        latent, widths = self._latent(heads, d, rot, rank, span)
        rows, at_latent = self._laid_out(widths, tokens)
        cache = LayerHistory(latent=self.rnd(span + tokens, latent.m.row))
        latent.chunk(rows, at_latent, cache, 0, self.status)              # binds the arguments of the launches below
        q_rank = latent.m.q_rank
        prepare = lambda: latent._prepare(rows)
        prepare_like, widths = self._window(heads, heads, d, 1)
        proj_like, at_like = self._laid_out(widths, tokens)
        ring = LayerHistory(k=self.rnd(tokens, heads, d), v=self.rnd(tokens, heads, d))
        near = lambda: prepare_like.chunk(proj_like, at_like, ring, 0, self.status)
        self.pair(f"latent_prepare_kernel {tokens} tokens", ([prepare] * 4, tokens * (2 * q_rank + rank + rot + latent.m.row) * 2),
                  "attn_prepare + attn_flash, window of one", ([near] * 4, tokens * heads * d * 2 * 8))
        queries = self.rnd(tokens, heads * (d + rot))
        rotate = lambda: call_hybrid("qd_rotate_half", ptr(queries), ptr(latent.freq), None, 0, tokens, heads, d + rot, rot, 0, stream_of(queries))
        self.pair(f"rotate_half_kernel {tokens} tokens, {heads} heads, {rot} of {d + rot} columns", ([rotate] * 4, tokens * heads * rot * 4),
                  "attn_prepare + attn_flash, window of one", ([near] * 4, tokens * heads * d * 2 * 8))
        # the attention itself on expanded rows: everything but the products, the norm and the rotation
        a, expanded, out = latent.args, self.rnd(span + tokens, latent.expand.shape[0]), self.rnd(tokens, heads * d)
        a.q_rows, a.out, a.gate, a.ld_gate = ptr(queries), ptr(out), ptr(rows), rows.shape[1]
        a.k_cache, a.v_cache = ptr(expanded), column(expanded, latent.expand_at["v"])
        core = lambda: call_hybrid("qd_attention", byref(a), stream_of(queries))
        self.pair(f"attn_flash on expanded latents, {tokens} tokens, window {span}, {heads} heads of {d} + {rot}",
                  ([core] * 4, 0, 2.0 * seen * heads * (2 * d + rot)), f"attn_prepare + attn_flash, {heads}/{heads} heads of {d}", like(heads))

    def attention_steps(self, heads, kv, d, rot, rank, span):
        pos = torch.tensor(span - 1, dtype=torch.int32, device=self.device)
        nbytes = 2 * span * kv * d * 2
        caches = [LayerHistory(k=self.rnd(span, kv, d), v=self.rnd(span, kv, d)) for _ in range(sets_for(nbytes))]

        def steps(mixer, widths, histories):
            proj, at = self._laid_out(widths, 1)
            return [lambda h=h: mixer.step(proj, at, h, pos, self.status) for h in histories]
        like = (steps(*self._window(heads, kv, d, span), caches), nbytes)
        self.pair(f"attn_step_kernel, chunk of {span}, {heads}/{kv} heads of {d}", (steps(*self._chunked(heads, kv, d, span), caches), nbytes),
                  f"attn_step_kernel, window {span}", like)
        mixer, widths = self._latent(heads, d, rot, rank, span)
        own_bytes = span * mixer.m.row * 2 + mixer.expand.nbytes
        sets = sets_for(own_bytes)
        mixers = [mixer] + [self._latent(heads, d, rot, rank, span)[0] for _ in range(sets - 1)]
        rows, at = self._laid_out(widths, 1)
        calls = []
        for one in mixers:
            history = LayerHistory(latent=self.rnd(span, mixer.m.row))
            query, out = self.rnd(1, heads * (d + rot)), self.rnd(1, heads * d)
            one._bind(rows, at, history, pos)
            one.latent.q, one.latent.out, one.kept = ptr(query), ptr(out), (history, query, out)
            calls.append(lambda one=one: call_hybrid("qd_latent_step", byref(one.latent), stream_of(rows)))
        self.pair(f"latent absorb + mma + values kernels, window {span}, {heads} heads of {d} + {rot}, rank {rank}", (calls, own_bytes),
                  f"attn_step_kernel, window {span}, {heads}/{kv} heads of {d}", like)

    def stream_norm(self, tokens, width):
        y, normed, vec = self.rnd(tokens, width), self.rnd(tokens, width), self.rnd(width)
        streams = [self.rnd(tokens, width, dtype=F32) for _ in range(sets_for(tokens * width * 8) if tokens > 64 else 8)]
        own = [lambda r=r: call_hybrid("qd_stream_norm", None, None, 0, ptr(r), None, ptr(y), None, ptr(r), ptr(vec), 1.0, ptr(normed), tokens, width, 1e-6,
                                       0, stream_of(y)) for r in streams]
        gate = self.rnd(tokens, width)
        like = [lambda r=r: call_hybrid("qd_sublayer_close", ptr(y), ptr(gate), width, ptr(vec), ptr(vec), ptr(vec), ptr(r), ptr(r), None, 0, None, -1,
                                        ptr(vec), ptr(vec), ptr(normed), tokens, width, 1e-6, 0, stream_of(y)) for r in streams]
        self.pair(f"stream_norm_kernel {tokens} x {width}", (own, tokens * width * 12), "sublayer_close_kernel, no earlier results",
                  (like, tokens * width * 14))


def step_bytes(engine, position: int) -> float:
    """Algorithmic bytes of one token: every matrix once per use, recurrent states read and written, the visible rows."""
    model, c = engine.fused, engine.ckpt.config
    total = sum(m.nbytes for m in model.products()) + engine.ckpt.lm_head.nbytes
    for (index, _), history in zip(c.runs(), engine.state.layers):
        m = c.layers[index].mixer
        if history.rec is not None:
            total += 2 * history.rec.nbytes
            continue
        visible = position % m.span + 1 if isinstance(m, ChunkAttnConfig) else min(m.span, position + 1)
        total += visible * (m.row if history.latent is not None else m.kv_heads * (m.dim + m.vdim)) * 2
    return total


def matmul_flops(engine, tokens: int) -> float:
    return 2.0 * tokens * sum(m.numel() for m in engine.fused.products())


def timed(fn, reps: int = 3) -> float:
    fn()
    best = float("inf")
    for _ in range(reps):
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        begin.record()
        fn()
        end.record()
        torch.cuda.synchronize()
        best = min(best, begin.elapsed_time(end) * 1e-3)
    return best


def model_leg(ckpt, prompts, decode_steps: int, hbm: float, tensor: float, hybrid: bool) -> dict:
    engine = Engine(ckpt, max_context=max(prompts) + 1024, device="cuda:0")
    vocab = ckpt.config.vocab_size
    out = {"prefill": []}
    for n in prompts:
        tokens = (torch.arange(n) * 7919 % vocab).tolist()
        ids = torch.tensor(tokens, device="cuda:0")

        def run():
            engine.reset()
            for a in range(0, n, engine.prefill_chunk_size):
                engine.chunk_prefill.run(ids[a:a + engine.prefill_chunk_size], a, engine.state)
        seconds = timed(run)
        row = {"tokens": n, "ms": round(seconds * 1e3, 2), "tok_s": round(n / seconds)}
        if hybrid:
            row["products_frac"] = round(matmul_flops(engine, n) / seconds / tensor, 3)
        out["prefill"].append(row)
    engine.prefill([1, 2, 3] * 170)
    engine.pending_token = torch.tensor(5, device="cuda:0")
    for _ in range(8):
        engine.decode_step()

    def decode():
        for _ in range(decode_steps):
            engine.graph.replay()
    seconds = timed(decode) / decode_steps
    out["decode"] = {"ms_per_token": round(seconds * 1e3, 4), "tok_s": round(1 / seconds, 1)}
    if hybrid:
        nbytes = step_bytes(engine, engine.state.position)
        out["decode"] |= {"bytes_per_token": int(nbytes), "frac_of_hbm": round(nbytes / seconds / hbm, 3)}
    return out


def fezopel_cases(cases: Cases) -> None:
    cases.products(8192, 8192, 2048)
    cases.products(512, 8192, 2048)
    cases.matvec(12288, 2048)
    cases.matvec(2048, 4096)
    cases.recurrences(2048, 32, 16, 128, 16)
    cases.recurrence_steps(32, 16, 128, 16)
    cases.recurrence_steps(32, 16, 128, 128)
    cases.attention(2048, 16, 2, 256, 1024)
    cases.attention(8192, 16, 2, 256, 4096)
    cases.attention_step(16, 2, 256, 8192)
    cases.residual(2048, 2048, 6)
    cases.residual(1, 2048, 6)


def dokulix_cases(cases: LatentCases) -> None:
    cases.product_forms(2048, 16384, 2048)
    cases.matvec_forms(16384, 2048)
    cases.matvec_forms(2048, 8192)
    cases.attentions(2048, 16, 4, 128, 64, 512, 1024)
    cases.attentions(8192, 16, 4, 128, 64, 512, 4096)
    cases.attention_steps(16, 4, 128, 64, 512, 1024)
    cases.attention_steps(16, 4, 128, 64, 512, 8192)
    cases.stream_norm(2048, 2048)
    cases.stream_norm(1, 2048)


def fezopel_models(device, leg) -> dict:
    models = {}
    for hidden, depth in ((2048, 12), (4096, 12)):
        cfg = synthetic.fezopel_config(depth, 32768, hidden=hidden, heads=hidden // 128, kv_heads=max(2, hidden // 512))
        models[f"fezopel {depth} x {hidden}"] = leg(synthetic.make_fezopel(cfg, 0, device), True)
        torch.cuda.empty_cache()
    return models


def dokulix_models(device, leg) -> dict:
    models = {}
    for hidden, depth, loop in ((2048, 12, None), (4096, 12, None), (2048, 12, LoopConfig(3, 9, 2))):
        cfg = synthetic.dokulix_config(depth, 32768, hidden=hidden, heads=hidden // 128, kv_heads=max(2, hidden // 512), loop=loop)
        name = f"dokulix {depth} x {hidden}" + ("" if loop is None else f", layers {loop.start} - {loop.stop - 1} {loop.times} times")
        models[name] = leg(synthetic.make_dokulix(cfg, 0, device), True)
        torch.cuda.empty_cache()
    return models


def run(args, peaks: dict, clocks) -> None:
    device = torch.device("cuda:0")
    torch.cuda.set_device(device)
    hbm, tensor = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    torch.manual_seed(0)
    clocks.mark_begin()
    own = args.model == "fezopel"
    cases = (Cases if own else LatentCases)(device, peaks["hbm_gbs"], peaks["bf16_tflops"])
    (fezopel_cases if own else dokulix_cases)(cases)
    assert int(cases.status.item()) == 0
    torch.cuda.empty_cache()
    leg = lambda ckpt, hybrid: model_leg(ckpt, (512, 2048, 8192), 64, hbm, tensor, hybrid)
    models = {} if own else dokulix_models(device, leg)
    models |= fezopel_models(device, leg)
    if own:
        like = synthetic.model_config(num_layers=12, vocab_size=32768)
        models["nvfp4 hybrid MoE 12 x 2048"] = leg(synthetic.make_checkpoint(like, seed=0, device=device), False)
    clocks.mark_end()
    first = models[f"{args.model} 12 x 2048"]
    line = {"metric": "decode_tok_s", "model": args.model, "value": first["decode"]["tok_s"], "unit": "tok/s", "higher_is_better": True, "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic (random weights)", "vs_baseline": None, "ms_per_step": first["decode"]["ms_per_token"],
            "config": {"l2": "kernel legs rotate over operands beyond L2 or exceed it; a decode step streams its weights"},
            "models": models, "kernels": cases.rows, "peaks": peaks, "clocks": None, "cpus": os.cpu_count()}
    clocks.__exit__()
    line["clocks"] = clocks.summary()
    print(json.dumps(line), flush=True)
