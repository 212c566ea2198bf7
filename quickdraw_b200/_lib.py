"""ctypes binding of ``libquickdraw_b200.so`` (declarations: ``include/quickdraw_b200.h``) and of
the libraries of the bf16-weight models (``include/quickdraw_b200_hybrid.h``): ``_hybrid`` with what all of them use,
``_recurrent`` and ``_latent`` with the mixers that only some of them have.

Each library is the only execution path of this package: if it cannot be loaded the
import of any operator raises, there is no PyTorch or CPU fallback.
"""

from __future__ import annotations

import ctypes
from ctypes import c_char_p, c_float, c_int, c_longlong, c_void_p
from pathlib import Path

import torch

LIB_PATH = Path(__file__).resolve().parent / "libquickdraw_b200.so"

P, I, F, L = c_void_p, c_int, c_float, c_longlong

SIGNATURES = {
    "qd_version": [],
    "qd_rms_norm": [P, P, P, I, I, F, I, P],
    "qd_add_rms_norm": [P, P, P, P, P, I, F, P],
    "qd_nvfp4_gemv": [P, P, P, P, P, P, I, I, I, I, P],
    "qd_nvfp4_expert_gemv": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "qd_nvfp4_gate_up": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, P],
    "qd_nvfp4_dequantize": [P, P, F, P, L, I, I, I, P],
    "qd_bf16_gemv": [P, P, P, I, I, P],
    "qd_fp8_gemv": [P, P, P, P, P, I, I, I, P],
    "qd_fp8_matmul": [P, P, P, P, P, I, I, I, P, I, P],
    "qd_route_topk": [P, I, I, I, P, P, P],
    "qd_moe_combine": [P, P, P, P, P, I, I, P],
    "qd_swiglu": [P, P, P, I, P],
    "qd_gdn_conv": [P, P, P, P, I, I, P],
    "qd_gdn_recurrence": [P, P, P, P, P, P, P, I, I, I, I, I, P],
    "qd_gdn_gated_norm": [P, P, P, P, I, I, F, P],
    "qd_attn_scratch_floats": [I, I, I, I],
    "qd_attn_decode": [P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, F, I, I, P],
    "qd_attn_decode_static": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, F, I, P],
    "qd_moe_down_combine": [P, P, P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "qd_moe_finish": [P, P, P, I, I, P],
    "qd_model_create": [P, P],
    "qd_model_destroy": [P],
    "qd_model_set_layer": [P, I, P],
    "qd_decode_workspace_bytes": [P],
    "qd_decode_step": [P, P, P, P, I, P, P, P, I, P],
    "qd_program_bytes": [P],
    "qd_program_build": [P, P, P, L],
    "qd_decode_step_persistent": [P, P, P, P, I, P, P, P, P, P, I, P, P],
    "qd_exchange_bytes": [P],
    "qd_set_wait_limit_us": [ctypes.c_uint],
    "qd_set_chained_launches": [I],
    "qd_nvfp4_gemv_bank": [P, P, P, P, P, I, I, I, I, P],
    "qd_nvfp4_matmul": [P, P, P, P, P, I, I, I, I, P, P],
    "qd_nvfp4_matmul_rows_scratch_bytes": [I],
    "qd_nvfp4_matmul_rows": [P, P, P, P, P, P, I, I, I, I, P, I, P],
    "qd_nvfp4_matmul_rows3": [P, P, I, I, I, P, I, I, P, P, P, P, I, P, P, P, P, I, P, P, P, P, I, P],
    "qd_nvfp4_quantize_act": [P, I, I, P, P, P, P, P],
    "qd_nvfp4_matmul_w4a4": [P, P, P, P, P, P, P, I, I, I, I, P, P],
    "qd_nvfp4_grouped_matmul": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, P, P],
    "qd_nvfp4_expert_rows_scratch_bytes": [I, I],
    "qd_nvfp4_expert_rows2": [P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, P, I, P],
    "qd_nvfp4_expert_rows": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, P, I, P],
    "qd_seq_add_rms_norm": [P, P, P, P, P, I, I, F, P],
    "qd_seq_bf16_matmul": [P, P, P, I, I, I, P],
    "qd_seq_bf16_matmul2": [P, P, P, I, P, P, I, I, I, P],
    "qd_seq_gdn_conv": [P, P, P, P, I, I, I, P],
    "qd_seq_gdn_recurrence": [P, P, P, P, P, P, P, I, I, I, I, I, P],
    "qd_seq_gdn_chunk_scratch_bytes": [I, I],
    "qd_seq_gdn_recurrence_chunked": [P, P, P, P, P, P, P, I, I, I, I, I, P, P],
    "qd_seq_attention": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, F, P],
    "qd_seq_route_topk": [P, I, I, I, P, P, P],
    "qd_batch_gdn_conv": [P, P, P, L, P, I, I, I, P],
    "qd_batch_gdn_recurrence": [P, P, P, P, P, P, L, P, I, I, I, I, I, P],
    "qd_batch_attn_decode": [P, P, P, P, P, P, P, L, P, P, P, P, I, I, I, I, I, I, F, F, I, P],
    "qd_batch_attention": [P, P, P, P, P, P, P, L, P, P, P, P, P, I, I, I, I, I, I, F, F, I, P],
    "qd_seq_group_routes": [P, I, I, P, P, P],
    "qd_seq_moe_combine": [P, P, P, P, P, I, I, I, P],
    "qd_seq_moe_combine_norm": [P, P, P, P, P, P, P, P, I, I, I, F, P],
}

# entry points of the bf16-weight models by library (declarations: ``include/quickdraw_b200_hybrid.h``)
HYBRID_LIBRARIES = {
    "hybrid": {
        "qd_set_chained_launches": [I],
        "qd_linear": [P, L, I, P, P, L, I, I, I, I, I, I, P, I, P, F, F, P, P],
        "qd_greedy": [P, I, P, P, P, P],
        "qd_embed_norm": [P, P, I, P, P, P, P, I, I, F, I, P],
        "qd_layer_norm_rows": [P, P, P, P, P, I, I, F, I, P],
        "qd_sublayer_close": [P, P, L, P, P, P, P, P, P, L, P, I, P, P, P, I, I, F, I, P],
        "qd_stream_norm": [P, P, I, P, P, P, P, P, P, F, P, I, I, F, I, P],
        "qd_attention": [P, P],
        "qd_attention_step_floats": [I, I, I],
        "qd_attention_step": [P, P],
    },
    "recurrent": {
        "qd_gla_prepare": [P, P, P, L, P, P, F, P, P, P, P, I, I, I, I, I, P],
        "qd_channel_delta_prepare": [P, P, P, P, L, P, P, P, P, P, P, P, I, P, I, P, P, P, P, P, P, I, I, I, I, I, I, P],
        "qd_linear_recurrence": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, P],
        "qd_head_norm_gate": [P, P, P, L, P, I, I, I, F, I, I, P],
        "qd_gla_step": [P, P, P, P, P, P, I, F, P, P, F, P, P, I, I, I, I, P],
        "qd_channel_delta_step": [P, P, P, P, P, P, P, I, P, P, P, P, P, I, P, I, P, P, I, P, F, P, P, I, I, I, I, I, P],
    },
    "latent": {
        "qd_latent_prepare": [P, P],
        "qd_rotate_half": [P, P, P, I, I, I, I, I, I, P],
        "qd_latent_step_floats": [I, I, I],
        "qd_latent_step": [P, P],
    },
}
HYBRID_LONG_RESULTS = {"qd_attention_step_floats", "qd_latent_step_floats"}
HYBRID_OWNER = {name: target for target, names in HYBRID_LIBRARIES.items() for name in names}


def _structure(name: str, *kinds) -> type:
    """A ctypes structure from (type, field names) pairs."""
    return type(name, (ctypes.Structure,), {"_fields_": [(field, kind) for kind, names in kinds for field in names.split()]})


AttentionArgs = _structure(
    "AttentionArgs", (P, "q k v gate q_norm k_norm freq sink slopes k_cache v_cache k_shared position_ptr q_rows out partial counters"),
    (L, "ld ld_gate ld_k ld_v ld_shared"), (F, "scale eps"),
    (I, "norm rot sink_kind gate_kind mask span capacity position tokens heads kv_heads dim vdim shared_dim splits dtype"))
LatentArgs = _structure(
    "LatentArgs", (P, "q dq dkv gate dq_norm dkv_norm freq uk uv cache position_ptr q_latent absorbed partial out"), (L, "ld ld_cache"),
    (F, "scale eps"), (I, "span capacity position tokens heads dim rot vdim q_rank kv_rank rot_column splits dtype"))
STRUCTURES = {"qd_attention_args": AttentionArgs, "qd_latent_args": LatentArgs}

LONG_RESULTS = {"qd_decode_workspace_bytes", "qd_program_bytes", "qd_exchange_bytes",
                "qd_nvfp4_matmul_rows_scratch_bytes", "qd_seq_gdn_chunk_scratch_bytes",
                "qd_nvfp4_expert_rows_scratch_bytes"}

_lib = None
_hybrid: dict[str, ctypes.CDLL] = {}


class LibraryMissing(RuntimeError):
    pass


def _open(path: Path, target: str, signatures: dict, long_results: set) -> ctypes.CDLL:
    if not path.exists():
        raise LibraryMissing(
            f"{path} not found: build it with `python -m quickdraw_b200.build{target}` "
            "(this package has no fallback path)")
    handle = ctypes.CDLL(str(path))
    for name, argtypes in signatures.items():
        fn = getattr(handle, name, None)
        if fn is None:
            continue
        fn.argtypes = argtypes
        fn.restype = c_longlong if name in long_results else c_int
    handle.qd_error_string.argtypes = [c_int]
    handle.qd_error_string.restype = c_char_p
    return handle


def lib() -> ctypes.CDLL:
    """Load the CUDA library once; raise loudly if it has not been built."""
    global _lib
    if _lib is None:
        _lib = _open(LIB_PATH, "", SIGNATURES, LONG_RESULTS)
    return _lib


def hybrid_path(target: str) -> Path:
    return LIB_PATH.with_name(f"libquickdraw_b200_{target}.so")


def hybrid_lib(target: str = "hybrid") -> ctypes.CDLL:
    """A library of the bf16-weight models, loaded on first use."""
    if target not in _hybrid:
        _hybrid[target] = _open(hybrid_path(target), f" {target}", HYBRID_LIBRARIES[target], HYBRID_LONG_RESULTS)
    return _hybrid[target]


def exported_symbols() -> list[str]:
    return sorted(SIGNATURES) + ["qd_error_string"]


def ptr(t: torch.Tensor | None):
    """Device address of a tensor (or NULL)."""
    return None if t is None else c_void_p(t.data_ptr())


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def stream_of(t: torch.Tensor):
    """The current CUDA stream of the tensor's device as a C handle.  A prompt chunk is some 1 300
    launches: the raw-handle query (a fraction of a microsecond) instead of building a
    ``torch.cuda.Stream`` object per launch (several microseconds) is 3 ms of host time per chunk."""
    if _raw_stream is not None:
        return c_void_p(_raw_stream(t.device.index if t.device.index is not None else torch.cuda.current_device()))
    return c_void_p(torch.cuda.current_stream(t.device).cuda_stream)


def check(code: int, name: str) -> None:
    if code != 0:
        raise RuntimeError(f"{name} failed: {lib().qd_error_string(code).decode()} (code {code})")


def call(name: str, *args) -> None:
    check(getattr(lib(), name)(*args), name)


def call_hybrid(name: str, *args) -> None:
    library = hybrid_lib(HYBRID_OWNER[name])
    code = getattr(library, name)(*args)
    if code != 0:
        raise RuntimeError(f"{name} failed: {library.qd_error_string(code).decode()} (code {code})")


def size_hybrid(name: str, *args) -> int:
    """The result of an entry point that computes a size."""
    return getattr(hybrid_lib(HYBRID_OWNER[name]), name)(*args)
