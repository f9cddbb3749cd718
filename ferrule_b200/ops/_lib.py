"""ctypes binding of libferrule_b200.so.

The library is loaded lazily.  On a machine with a CUDA device a missing or stale
library is an error (ops never fall back to PyTorch silently); on a CPU-only machine
`get_lib()` returns None and callers use the fp32 PyTorch reference path, which is
the oracle the CUDA kernels are tested against.

Mirrors the role of the reference's FFI layer between its device runtime and native
kernels (crates/ferrule-backend/src/cuda/kernels.rs:523-545, cutlass.rs:30-75).
"""
from __future__ import annotations

import ctypes as C
import os
import threading
from typing import Optional

import torch

from .. import _build

FB_OK = 0
_ERR_NAMES = {
    1: "FB_ERR_SHAPE (launcher rejected the arguments)",
    2: "FB_ERR_ALIGN (pointer or stride not 16-byte aligned)",
    3: "FB_ERR_DRIVER (driver entry point missing / tensor map encode failed)",
    4: "FB_ERR_LAUNCH (kernel launch failed)",
    5: "FB_ERR_RUNTIME (CUDA runtime error)",
    6: "FB_ERR_LIMIT (size beyond a fixed capacity)",
}


class NativeLibraryError(RuntimeError):
    pass


class GemmArgs(C.Structure):
    _fields_ = [
        ("w", C.c_void_p), ("x", C.c_void_p), ("out", C.c_void_p),
        ("ldw", C.c_longlong), ("w_group_stride", C.c_longlong), ("ldx", C.c_longlong),
        ("ldo", C.c_longlong),
        ("n_out", C.c_int), ("k", C.c_int), ("groups", C.c_int), ("w_rows_per_group", C.c_int),
        ("x_rows", C.c_int), ("ntok", C.c_int), ("epilogue", C.c_int), ("dual_offset", C.c_int),
        ("out_fp32", C.c_int), ("max_tok_tiles", C.c_int), ("x_group_koff", C.c_int),
        ("out_group_coff", C.c_int), ("force_split", C.c_int),
        ("tile_group", C.c_void_p), ("tile_row0", C.c_void_p), ("tile_rows", C.c_void_p),
        ("num_tok_tiles", C.c_void_p), ("dst_row", C.c_void_p), ("row_scale", C.c_void_p),
        ("act_limit", C.c_float), ("rank", C.c_int), ("world", C.c_int), ("rows_cap", C.c_int),
        ("flag_capacity", C.c_int),
        ("peer_recv", C.c_void_p * 8), ("peer_flags", C.c_void_p * 8),
        ("local_ctr", C.c_void_p), ("residual", C.c_void_p), ("ldr", C.c_longlong),
        ("peer_wait_ns", C.c_ulonglong), ("status", C.c_void_p), ("trace", C.c_void_p),
        ("ar_payload_bf16", C.c_int),
        ("remap_rank", C.c_void_p), ("remap_row", C.c_void_p), ("mc_recv", C.c_void_p),
        ("bias", C.c_void_p), ("act_alpha", C.c_float), ("act_shift", C.c_float),
    ]


class AttnArgs(C.Structure):
    _fields_ = [
        ("q", C.c_void_p), ("kv", C.c_void_p), ("out", C.c_void_p),
        ("block_table", C.c_void_p), ("row_seq", C.c_void_p), ("row_pos", C.c_void_p),
        ("sink", C.c_void_p), ("part_o", C.c_void_p), ("part_ml", C.c_void_p),
        ("status", C.c_void_p),
        ("ldq", C.c_longlong), ("ldo", C.c_longlong), ("pool_rows", C.c_longlong),
        ("rows", C.c_int), ("heads", C.c_int), ("kv_lora", C.c_int), ("rope_dim", C.c_int),
        ("num_seqs", C.c_int), ("max_blocks", C.c_int), ("page_size", C.c_int),
        ("group_rows", C.c_int), ("splits", C.c_int), ("split_tokens", C.c_int),
        ("softmax_scale", C.c_float), ("merge_ctr", C.c_void_p),
        ("selection", C.c_void_p), ("sel_width", C.c_int), ("trace", C.c_void_p),
        ("decode_only", C.c_int),
        ("gate", C.c_void_p), ("ldg", C.c_longlong), ("window", C.c_int),
    ]


class PrefillAttnArgs(C.Structure):
    _fields_ = [
        ("q", C.c_void_p), ("kv", C.c_void_p), ("out", C.c_void_p), ("tiles", C.c_void_p),
        ("block_table", C.c_void_p), ("sink", C.c_void_p), ("status", C.c_void_p),
        ("ldq", C.c_longlong), ("ldo", C.c_longlong), ("pool_rows", C.c_longlong),
        ("n_tiles", C.c_int), ("rows", C.c_int), ("heads", C.c_int), ("kv_lora", C.c_int), ("rope_dim", C.c_int),
        ("num_seqs", C.c_int), ("max_blocks", C.c_int), ("page_size", C.c_int), ("softmax_scale", C.c_float),
        ("gate", C.c_void_p), ("ldg", C.c_longlong), ("window", C.c_int),
    ]


class LayerTailArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("ldx", C.c_longlong), ("mix", C.c_void_p), ("ldm", C.c_longlong),
        ("gate1", C.c_void_p), ("ldg1", C.c_longlong), ("bias1", C.c_void_p),
        ("ffn", C.c_void_p), ("ldf", C.c_longlong), ("slots", C.c_int), ("topk", C.c_int),
        ("gate2", C.c_void_p), ("ldg2", C.c_longlong), ("bias2", C.c_void_p),
        ("norm_w", C.c_void_p), ("norm_stride", C.c_int), ("rows", C.c_int),
        ("h", C.c_void_p), ("ldh", C.c_longlong), ("dim", C.c_int), ("dim_pad", C.c_int), ("eps", C.c_float),
        ("fp32", C.c_int),
    ]


class DeltaArgs(C.Structure):
    _fields_ = [
        ("proj", C.c_void_p), ("ldp", C.c_longlong),
        ("off_q", C.c_int), ("off_k", C.c_int), ("off_v", C.c_int), ("off_b", C.c_int),
        ("ag", C.c_void_p), ("ldag", C.c_longlong), ("off_gate", C.c_int),
        ("off_a", C.c_int), ("off_g", C.c_int), ("gate_silu", C.c_int), ("long_seqs", C.c_int), ("fp32", C.c_int),
        ("conv", C.c_void_p), ("a_neg", C.c_void_p), ("dt_bias", C.c_void_p), ("norm_w", C.c_void_p),
        ("state", C.c_void_p), ("tail", C.c_void_p), ("row_seq", C.c_void_p), ("seq_start", C.c_void_p),
        ("state_in", C.c_void_p), ("state_out", C.c_void_p),
        ("qn", C.c_void_p), ("kn", C.c_void_p), ("v", C.c_void_p), ("decay", C.c_void_p), ("beta", C.c_void_p),
        ("qk", C.c_void_p), ("o", C.c_void_p),
        ("out", C.c_void_p), ("ldo", C.c_longlong), ("status", C.c_void_p),
        ("n_states", C.c_int), ("rows", C.c_int), ("n_seqs", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int),
        ("dim", C.c_int), ("vdim", C.c_int), ("taps", C.c_int), ("eps", C.c_float),
    ]


class StreamArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("ldx", C.c_longlong), ("ids", C.c_void_p), ("positions", C.c_void_p),
        ("table", C.c_void_p), ("pos_table", C.c_void_p), ("ldt", C.c_longlong), ("vocab", C.c_int), ("max_pos", C.c_int),
        ("y", C.c_void_p), ("ldy", C.c_longlong), ("norm_w", C.c_void_p), ("norm_b", C.c_void_p), ("rms", C.c_int),
        ("act", C.c_void_p), ("lda", C.c_longlong), ("conv", C.c_void_p), ("tail", C.c_void_p),
        ("state_in", C.c_void_p), ("state_out", C.c_void_p), ("taps", C.c_int), ("n_states", C.c_int),
        ("h", C.c_void_p), ("ldh", C.c_longlong), ("rows", C.c_int), ("dim", C.c_int), ("dim_pad", C.c_int),
        ("fp32", C.c_int), ("eps", C.c_float), ("status", C.c_void_p),
    ]


class ConvArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("ldx", C.c_longlong), ("w", C.c_void_p), ("bias", C.c_void_p), ("tail", C.c_void_p),
        ("out", C.c_void_p), ("ldo", C.c_longlong), ("row_seq", C.c_void_p), ("seq_start", C.c_void_p),
        ("state_in", C.c_void_p), ("state_out", C.c_void_p), ("rows", C.c_int), ("channels", C.c_int), ("taps", C.c_int),
        ("n_states", C.c_int), ("n_seqs", C.c_int), ("x_fp32", C.c_int), ("out_fp32", C.c_int), ("residual", C.c_int),
        ("silu", C.c_int), ("status", C.c_void_p),
    ]


class ScanArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("ldx", C.c_longlong), ("z", C.c_void_p), ("ldz", C.c_longlong),
        ("bc", C.c_void_p), ("ldbc", C.c_longlong), ("off_b", C.c_int), ("off_c", C.c_int),
        ("dt", C.c_void_p), ("lddt", C.c_longlong), ("dt_bias", C.c_void_p), ("a_log2", C.c_void_p), ("d_skip", C.c_void_p),
        ("states", C.c_void_p), ("seq_start", C.c_void_p), ("state_in", C.c_void_p), ("state_out", C.c_void_p),
        ("out", C.c_void_p), ("ldo", C.c_longlong), ("rows", C.c_int), ("n_seqs", C.c_int), ("inner", C.c_int),
        ("state", C.c_int), ("n_states", C.c_int), ("fp32", C.c_int), ("status", C.c_void_p),
    ]


class GqaArgs(C.Structure):
    _fields_ = [
        ("q", C.c_void_p), ("ldq", C.c_longlong), ("k", C.c_void_p), ("v", C.c_void_p), ("ldkv", C.c_longlong),
        ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("cos_t", C.c_void_p), ("sin_t", C.c_void_p),
        ("max_pos", C.c_int), ("rot_dims", C.c_int), ("positions", C.c_void_p), ("write_slot", C.c_void_p),
        ("pool", C.c_void_p), ("pool_rows", C.c_longlong), ("pool_ld", C.c_longlong),
        ("first_pool", C.c_void_p), ("first_off", C.c_longlong), ("v_mix", C.c_float),
        ("block_table", C.c_void_p), ("row_seq", C.c_void_p), ("row_pos", C.c_void_p),
        ("num_seqs", C.c_int), ("max_blocks", C.c_int), ("page_size", C.c_int), ("chunk", C.c_int),
        ("scale", C.c_float), ("eps", C.c_float), ("out", C.c_void_p), ("ldo", C.c_longlong),
        ("rows", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("dim_pad", C.c_int),
        ("vdim", C.c_int), ("vdim_pad", C.c_int), ("fp32", C.c_int), ("maps", C.c_int), ("key_width", C.c_int),
        ("key_stride", C.c_int), ("v_offset", C.c_int), ("window", C.c_int), ("keep_first", C.c_int),
        ("slopes", C.c_void_p), ("gate", C.c_void_p), ("ldg", C.c_longlong), ("diff_lambda", C.c_float),
        ("diff_scale", C.c_float), ("value_width", C.c_int), ("value_stride", C.c_int), ("softcap", C.c_float),
        ("score_bound", C.c_float), ("pooled", C.c_void_p), ("pooled_rows", C.c_longlong), ("pool_tokens", C.c_int), ("pooled_stride", C.c_int),
        ("slot_div", C.c_int), ("slot_of", C.c_void_p), ("talk", C.c_void_p), ("status", C.c_void_p),
    ]


class SandwichArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("ldx", C.c_longlong), ("y", C.c_void_p), ("ldy", C.c_longlong), ("y_bias", C.c_void_p),
        ("out_w", C.c_void_p), ("ids", C.c_void_p), ("table", C.c_void_p), ("ldt", C.c_longlong), ("vocab", C.c_int),
        ("fresh", C.c_int), ("in_w", C.c_void_p), ("act", C.c_void_p), ("lda", C.c_longlong), ("rows", C.c_int),
        ("dim", C.c_int), ("dim_pad", C.c_int), ("groups", C.c_int), ("fp32", C.c_int), ("eps", C.c_float),
        ("status", C.c_void_p),
    ]


class PreNormArgs(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("x_out", C.c_void_p), ("ldx", C.c_longlong), ("ids", C.c_void_p), ("table", C.c_void_p),
        ("ldt", C.c_longlong), ("vocab", C.c_int), ("scale", C.c_float), ("y", C.c_void_p), ("ldy", C.c_longlong),
        ("ffn", C.c_void_p), ("ldf", C.c_longlong), ("slots", C.c_int), ("topk", C.c_int), ("shared", C.c_void_p),
        ("lds", C.c_longlong), ("shared_gate", C.c_void_p), ("ldsg", C.c_longlong), ("norm_w", C.c_void_p),
        ("act", C.c_void_p), ("lda", C.c_longlong), ("shift", C.c_void_p), ("plane", C.c_void_p), ("row_seq", C.c_void_p),
        ("seq_start", C.c_void_p), ("state_in", C.c_void_p), ("state_out", C.c_void_p), ("n_states", C.c_int),
        ("n_seqs", C.c_int), ("rows", C.c_int), ("dim", C.c_int), ("dim_pad", C.c_int), ("fp32", C.c_int),
        ("eps", C.c_float), ("status", C.c_void_p),
    ]


class HeadScanArgs(C.Structure):
    _fields_ = [
        ("xbc", C.c_void_p), ("ldx", C.c_longlong), ("off_b", C.c_int), ("off_c", C.c_int), ("dt", C.c_void_p),
        ("z", C.c_void_p), ("ldp", C.c_longlong), ("dt_bias", C.c_void_p), ("a_neg", C.c_void_p), ("d_skip", C.c_void_p),
        ("states", C.c_void_p), ("seq_start", C.c_void_p), ("state_in", C.c_void_p), ("state_out", C.c_void_p),
        ("out", C.c_void_p), ("ldo", C.c_longlong), ("rows", C.c_int), ("n_seqs", C.c_int), ("heads", C.c_int),
        ("vdim", C.c_int), ("state", C.c_int), ("groups", C.c_int), ("n_states", C.c_int), ("fp32", C.c_int),
        ("long_seqs", C.c_int), ("by_token", C.c_int), ("status", C.c_void_p),
    ]


class LatentPrepArgs(C.Structure):
    _fields_ = [
        ("cq", C.c_void_p), ("ckv", C.c_void_p), ("ldp", C.c_longlong), ("rank_q", C.c_int), ("rank", C.c_int),
        ("rot", C.c_int), ("row_dim", C.c_int), ("rot_off", C.c_int), ("rows", C.c_int), ("q_w", C.c_void_p),
        ("kv_w", C.c_void_p), ("cos_t", C.c_void_p), ("sin_t", C.c_void_p), ("max_pos", C.c_int), ("fp32", C.c_int),
        ("positions", C.c_void_p), ("write_slot", C.c_void_p), ("pool", C.c_void_p), ("pool_rows", C.c_longlong),
        ("eps", C.c_float), ("status", C.c_void_p),
    ]


class PoolArgs(C.Structure):
    _fields_ = [
        ("pool", C.c_void_p), ("pool_rows", C.c_longlong), ("pool_ld", C.c_longlong), ("pooled", C.c_void_p),
        ("pooled_rows", C.c_longlong), ("positions", C.c_void_p), ("row_seq", C.c_void_p), ("block_table", C.c_void_p),
        ("slot_of", C.c_void_p), ("rows", C.c_int), ("width", C.c_int), ("num_seqs", C.c_int), ("max_blocks", C.c_int),
        ("page_size", C.c_int), ("pool_tokens", C.c_int), ("pooled_stride", C.c_int), ("slot_div", C.c_int),
        ("fp32", C.c_int), ("status", C.c_void_p),
    ]


class HeadPrepArgs(C.Structure):
    _fields_ = [
        ("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ldp", C.c_longlong), ("q_bias", C.c_void_p),
        ("k_bias", C.c_void_p), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("q_mix", C.c_void_p), ("mix", C.c_int),
        ("q_out", C.c_void_p), ("ldqo", C.c_longlong), ("write_slot", C.c_void_p), ("pool", C.c_void_p),
        ("pool_rows", C.c_longlong), ("pool_ld", C.c_longlong), ("rows", C.c_int), ("heads", C.c_int),
        ("kv_heads", C.c_int), ("maps", C.c_int), ("dim", C.c_int), ("dim_pad", C.c_int), ("vdim_pad", C.c_int),
        ("fp32", C.c_int), ("eps", C.c_float), ("status", C.c_void_p), ("cos_t", C.c_void_p), ("sin_t", C.c_void_p),
        ("positions", C.c_void_p), ("half", C.c_int), ("max_pos", C.c_int), ("blocks", C.POINTER(PoolArgs)),
    ]


_lock = threading.Lock()
_lib: Optional[C.CDLL] = None
_tried = False
_component = ""


def use_component(name: str) -> None:
    """For programs that need one part of the library: without a built full library, `get_lib` builds and loads this
    component (`_build.COMPONENTS`) instead of everything.  Call before the first `get_lib`."""
    global _component
    if name and name not in _build.COMPONENTS:
        raise ValueError(f"unknown library component {name!r}")
    _component = name


def _declare(lib: C.CDLL) -> None:
    vp, i, ll, f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
    lib.fb_status_bytes.restype = i
    lib.fb_gemm_bf16.argtypes = [C.POINTER(GemmArgs), vp]
    lib.fb_mla_attention.argtypes = [C.POINTER(AttnArgs), vp]
    lib.fb_mla_prefill_tc.argtypes = [C.POINTER(PrefillAttnArgs), vp]
    lib.fb_mla_prefill_tc.restype = i
    lib.fb_embedding.argtypes = [vp, vp, vp, i, i, i, vp, vp]
    lib.fb_add_rmsnorm.argtypes = [vp, ll, vp, ll, vp, vp, ll, vp, ll, i, i, f, vp]
    lib.fb_mla_prep.argtypes = [vp, ll, i, vp, ll, i, i, i, vp, f, vp, vp, i, vp, vp, vp, ll, vp,
                                ll, i, vp, vp]
    lib.fb_router_topk.argtypes = [vp, ll, vp, vp, vp, i, i, i, i, i, i, i, f, vp, vp, vp, vp]
    lib.fb_moe_plan.argtypes = [vp, vp, i, i, i, i, i, i, vp, vp, vp, vp, vp, vp, i, vp, vp, vp, vp]
    lib.fb_gather_rows.argtypes = [vp, ll, vp, vp, vp, ll, i, i, i, vp, vp]
    lib.fb_moe_reduce.argtypes = [vp, i, i, vp, i, i, vp, ll, vp, ll, vp, ll, i, i, i, vp]
    lib.fb_argmax.argtypes = [vp, ll, i, i, vp, vp, vp]
    lib.fb_topk_logits.argtypes = [vp, ll, i, i, i, vp, vp, vp]
    lib.fb_copy_pages.argtypes = [vp, ll, ll, vp, i, i, i, vp, vp]
    for name in ("fb_gemm_bf16", "fb_mla_attention", "fb_embedding", "fb_add_rmsnorm",
                 "fb_mla_prep", "fb_router_topk", "fb_moe_plan", "fb_gather_rows", "fb_moe_reduce",
                 "fb_argmax", "fb_topk_logits", "fb_copy_pages"):
        getattr(lib, name).restype = i
    # optional groups, declared by their own modules when present
    from . import _lib_ext
    _lib_ext.declare(lib)


def get_lib(required: Optional[bool] = None) -> Optional[C.CDLL]:
    """Return the loaded native library, building it if the tree has sources but no .so.

    required=None means "required iff a CUDA device is present".
    """
    global _lib, _tried
    if required is None:
        required = torch.cuda.is_available()
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is not None:
            return _lib
        if _tried and not required:
            return None
        _tried = True
        path = _build.LIB_PATH
        try:
            if not path.exists():
                if os.environ.get("FERRULE_NO_BUILD"):
                    raise NativeLibraryError(f"{path} is missing and FERRULE_NO_BUILD is set")
                path = _build.build(component=_component)
            lib = C.CDLL(str(path))
            _declare(lib)
            _lib = lib
            return lib
        except Exception as exc:  # noqa: BLE001 - surfaced below
            if required:
                raise NativeLibraryError(
                    f"native library unavailable on a CUDA machine ({exc}); "
                    "run `python -m ferrule_b200._build`") from exc
            return None


def native_available() -> bool:
    return torch.cuda.is_available() and get_lib(required=False) is not None


LAUNCHES = [0]      # native kernel-launching calls that returned FB_OK (one launch each)


def check(rc: int, what: str) -> None:
    if rc != FB_OK:
        raise NativeLibraryError(f"{what}: {_ERR_NAMES.get(rc, rc)}")
    LAUNCHES[0] += 1


def stream_ptr() -> int:
    return torch.cuda.current_stream().cuda_stream


def ptr(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


# ---------------------------------------------------------------------------
# device status word: one per device, checked by the engine between steps
# ---------------------------------------------------------------------------
_status = {}

_STATUS_NAMES = {1: "pipeline barrier timeout", 2: "peer flag timeout", 3: "index out of range",
                 4: "shape/capacity rejected on device"}


def status_tensor(device=None) -> torch.Tensor:
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    if dev.type == "cuda" and dev.index is None:          # "cuda" and "cuda:N" must name the same status word
        dev = torch.device("cuda", torch.cuda.current_device())
    t = _status.get(dev)
    if t is None:
        # words 0..3: status {code, site, detail0, detail1}; 4..5: ns spent waiting on peer flags; 6: waits that spun
        t = torch.zeros(8, dtype=torch.int32, device=dev)
        _status[dev] = t
    return t


def read_status(device=None, reset: bool = True):
    """Synchronising read of the status word -> (code, where, d0, d1)."""
    t = status_tensor(device)
    vals = [int(v) & 0xFFFFFFFF for v in t[:4].tolist()]
    if reset and vals[0] != 0:
        t[:4].zero_()
    return tuple(vals)


def read_peer_wait(device=None, reset: bool = True):
    """(nanoseconds kernels of this device spent spinning on peer flags, number of such waits) since the last reset."""
    t = status_tensor(device)
    w = [int(v) & 0xFFFFFFFF for v in t[4:7].tolist()]
    if reset:
        t[4:7].zero_()
    return (w[1] << 32) | w[0], w[2]


def raise_on_status(device=None) -> None:
    code, where, d0, d1 = read_status(device)
    if code != 0:
        raise NativeLibraryError(
            f"device status: {_STATUS_NAMES.get(code, code)} at site 0x{where:x} (detail {d0}, {d1})")
