"""Python side of the CUDA kernels: loads the library and checks arguments before a launch.

Every function here runs a hand-written sm_100a kernel of ``csrc/`` on the current CUDA
stream.  There is no other implementation behind them: without the library (no nvcc, no
GPU) they raise.  The reference builds its kernels with torch's JIT at import
(layers/ops.py:5-18); here the build is a plain nvcc run at the first call.
"""
from __future__ import annotations

import ctypes
from typing import Optional, Sequence

import torch

from . import build as _build

ATTN_TILE_Q = 16          # query tokens per block of the CUDA-core chunk kernel (csrc/attention_chunk.cu)
ATTN_TILE_SIZES = (8, 16, 32, 64, 128)   # query tokens per block that some attention kernel may ask for
SINK_ATTN_TILE_Q = 16     # query tokens per block of csrc/sink_attention.cu
DECODE_PARTITION = 128    # keys per partition of the decode kernel (csrc/attention_decode.cu)
MAX_HEAD_DIM = 256

_P, _I, _L, _F = ctypes.c_void_p, ctypes.c_int, ctypes.c_int64, ctypes.c_float
_PROTOS = {
    "me_embed": [_P, _P, _I, _P, _I, _I, _I, _P, _P, _I, _F, _I, _L, _P, _P, _I, _P, _I, _L, _P],
    "me_hc_norm": [_P, _L, _I, _P, _I, _P, _P, _P, _P, _F, _P, _I, _P, _I, _I, _P, _P, _P, _P, _I, _P],
    "me_short_conv": [_P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P],
    "me_polynorm": [_P, _I, _L, _P, _F, _P, _I, _L, _I, _I, _P],
    "me_mlstm_scan": [_P, _L, _I, _I, _I, _I, _I, _P, _P, _F, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _F, _I, _P],
    "me_mlstm_out": [_P, _P, _L, _I, _P, _F, _P, _I, _L, _I, _I, _I, _I, _I, _P],
    "me_latent_prep": [_P, _L, _I, _I, _I, _P, _F, _P, _I, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "me_latent_attention": [_P, _P, _I, _P, _P, _I, _P, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "me_heads_to_rows": [_P, _P, _I, _I, _I, _I, _P],
    "me_latent_attention_mma": [_P, _P, _P, _P, _I, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "me_latent_attention_decode": [_P, _P, _P, _P, _I, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _I, _P],
    "me_add_rmsnorm": [_P, _P, _I, _P, _F, _P, _I, _P, _I, _I, _I, _L, _P],
    "me_gemm_skinny": [_P, _L, _P, _P, _I, _L, _P, _I, _I, _I, _I, _P],
    "me_silu_mul": [_P, _P, _I, _I, _I, _P],
    "me_gemm_simt": [_P, _I, _L, _P, _I, _P, _I, _L, _I, _I, _I, _I, _P],
    "me_qk_norm_rope_kv_write": [_P, _I, _L, _I, _I, _I, _I, _P, _P, _F, _P, _I, _P, _P, _P, _I, _P],
    "me_attn_chunk": [_P, _I, _L, _P, _L, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "me_attn_decode": [_P, _I, _L, _P, _L, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P, _I, _P, _I, _P, _I, _P, _L, _I, _I, _F, _P, _P, _P, _I, _I, _I, _P, _P, _I, _I, _F, _F, _F, _I, _P],
    "me_attn_decode_fused": [_P, _L, _P, _L, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P, _F, _P, _P, _P, _P, _P,
                             _I, _I, _I, _P, _P],
    "me_gemm_decode": [_I, _P, _L, _P, _I, _F, _P, _P, _I, _L, _P, _P, _P, _P, _I, _I, _I, _P, ctypes.c_uint64, _F, _F, _F, _P],
    "me_gemm_stream": [_I, _P, _P, _I, _F, _P, _P, _I, _L, _P, _P, _P, _P, _I, _I, _I, _P, _P, _P, _F, _F, _F, _P],
    "me_gemm_tcgen05": [_P, _P, _P, _I, _L, _I, _I, _I, _I, _I, _I, _L, _F, _F, _F, _P, _P],
    "me_gemm_tcgen05_persistent": [_P, _P, _P, _I, _L, _I, _I, _I, _I, _I, _F, _F, _F, _P, _P],
    "me_gemm_tcgen05_shared": [_P, _P, _P, _I, _L, _I, _I, _I, _I, _I, _P, _P, _P, _P],
    "me_attn_prefill_tcgen05": [_P, _P, _P, _L, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _I, _P, _L, _P, _I, _I, _F, _P, _P, _P, _I, _I, _P, _P, _I, _I, _F, _F, _F, _I, _P],
    "me_tma_encode_2d": [_P, _P, ctypes.c_uint64, ctypes.c_uint64, ctypes.c_uint64, ctypes.c_uint32, ctypes.c_uint32, _I],
    "me_attn_prefill": [_P, _L, _P, _L, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "me_sample": [_P, _L, _P, _P, _P, _P, _I, _I, _P, _P, _P],
    "me_test_wait_expires": [_P, _I, _P, _P],
    "me_sandwich_norm": [_P, _P, _I, _P, _F, _P, _F, _P, _I, _P, _I, _I, _I, _P],
    "me_clamped_glu": [_P, _I, _L, _P, _I, _L, _I, _I, _F, _F, _F, _P],
    "me_conv_rope_kv": [_P, _L, _P, _P, _P, _I, _P, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P, _P],
    "me_rope_table": [_P, _P, _I, _I, _P, _P],
    "me_sink_attn": [_P, _I, _L, _P, _L, _P, _L, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _I, _I, _P, _F, _I, _I, _P, _P, _I, _I, _P, _P, _I, _P],
    "me_parallel_norm": [_P, _P, _P, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _P, _I, _I, _F, _P, _P, _I, _I, _P, _I, _F, _P],
    "me_attn_prep": [_P, _L, _P, _P, _P, _I, _F, _P, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P, _I, _F, _F, _F, _F, _P],
    "me_diff_combine": [_P, _I, _L, _P, _I, _L, _I, _I, _I, _I, _F, _F, _F, _P],
    "me_gla_decay": [_P, _L, _I, _I, _P, _I, _P, _F, _P, _I, _I, _P],
    "me_gla_scan": [_P, _L, _I, _I, _I, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _F, _P, _I, _I, _P, _P, _P, _P, _P],
    "me_stream_norm": [_P, _P, _P, _P, _I, _P, _P, _P, _F, _F, _F, _P, _P, _P, _F, _P, _I, _L, _P, _I, _I, _P],
    "me_conv_silu": [_P, _L, _P, _P, _P, _P, _I, _I, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "me_head_decay_scan": [_P, _P, _P, _I, _L, _L, _L, _I, _I, _I, _I, _F, _P, _L, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _P, _I, _P, _P, _I, _P],
    "me_gated_group_norm": [_P, _L, _P, _I, _L, _P, _I, _F, _P, _I, _L, _I, _I, _I, _P],
    "me_activation": [_P, _I, _L, _P, _I, _L, _I, _I, _I, _P],
    "me_soft_cap": [_P, _L, _F, _F, _P],
    "me_add_row_vector": [_P, _I, _I, _I, _P, _P],
    "me_moe_route": [_P, _P, _I, _I, _I, _P, _P, _P],
    "me_moe_route_grouped": [_P, _L, _P, _I, _I, _I, _I, _I, _I, _F, _P, _P, _P],
    "me_moe_route_grouped_sort": [_P, _L, _P, _I, _I, _I, _I, _I, _I, _F, _P, _P, _P, _P, _P, _P, _P],
    "me_group_norm": [_P, _P, _I, _L, _P, _I, _F, _P, _I, _P, _I, _I, _P],
    "me_pool_kv": [_P, _P, _I, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "me_moe_sort": [_P, _I, _I, _I, _P, _P, _P, _P, _P],
    "me_moe_route_sort": [_P, _P, _I, _I, _I, _P, _P, _P, _P, _P, _P, _P],
    "me_moe_gemm": [_P, _I, _L, _P, _I, _P, _I, _L, _P, _I, _P, _I, _L, _I, _I, _I, _I, _F, _F, _F, _I, _P],
    "me_moe_gather": [_P, _I, _L, _P, _I, _P, _I, _I, _P],
    "me_gemm_tcgen05_grouped": [_P, _P, _P, _I, _L, _P, _I, _I, _I, _I, _I, _I, _F, _F, _F, _I, _P, _P],
    "me_moe_combine": [_P, _L, _P, _P, _I, _P, _I, _L, _P, _L, _P, _I, _L, _I, _I, _P],
    "me_token_side_gate": [_P, _I, _L, _P, _P, _P, _I, _L, _I, _I, _I, _P, _I, _I, _P],
}
_DT = {torch.float32: 0, torch.bfloat16: 1}

_lib: Optional[ctypes.CDLL] = None
launches = 0              # kernels launched through this module (counted for the benchmark)


class KernelError(RuntimeError):
    pass


def require_extension() -> ctypes.CDLL:
    """The loaded kernel library; builds it at the first call; raises if that is impossible."""
    global _lib
    if _lib is not None:
        return _lib
    if not torch.cuda.is_available():
        raise KernelError("mini_engine_b200 needs a CUDA device: its kernels have no CPU path")
    path = _build.library_path()
    lib = ctypes.CDLL(path)
    lib.me_last_error.restype = ctypes.c_char_p
    for name, args in _PROTOS.items():
        fn = getattr(lib, name)
        fn.argtypes = args
        fn.restype = ctypes.c_int
    if (lib.me_attn_chunk_tile_q() != ATTN_TILE_Q or lib.me_attn_decode_partition() != DECODE_PARTITION
            or lib.me_sink_attn_tile_q() != SINK_ATTN_TILE_Q or lib.me_gla_chunk_len() != GLA_CHUNK):
        raise KernelError("the kernel library and ops/__init__.py disagree on tile sizes")
    lib.me_attn_prefill_heads_per_block.argtypes = [_I, _I, _I]
    lib.me_attn_prefill_tcgen05_heads_per_block.argtypes = [_I, _I, _I, _I]
    lib.me_sample_chunks.argtypes = [_I]
    lib.me_gemm_tcgen05_splits.argtypes = [_I, _I]
    lib.me_gemm_decode_sumsq_parts.argtypes = [_I]
    lib.me_gemm_stream_sumsq_parts.argtypes = [_I, _I]
    lib.me_gemm_stream_x_box_rows.argtypes = [_I]
    lib.me_gemm_stream_w_box_rows.argtypes = [_I]
    lib.me_attn_decode_fused_takes.argtypes = [_I, _I]
    lib.me_gemm_skinny_splits.argtypes = [_I]
    lib.me_latent_attention_mma_takes.argtypes = [_I, _I]
    lib.me_latent_attention_mma_heads_per_block.argtypes = [_I]
    _lib = lib
    return lib


def set_programmatic_launch(on: bool) -> None:
    """Switch programmatic dependent launch (a kernel may start, and fetch weights, while its predecessor
    still runs) on or off for all later launches; it is on by default."""
    (_lib or require_extension()).me_set_pdl(1 if on else 0)


def library_file() -> str:
    require_extension()
    return _lib._name


_fns: dict = {}
_last_call = None         # (entry point, arguments) of the launch before

# Per-kernel timing for the benchmark's roofline table: while ``timeline`` is a list, every launch made through
# this module is bracketed by two CUDA events and recorded as (tag, entry point, start, end).  ``tag`` is set by
# the caller that knows what the launch is for (a Linear part sets it to its output's name).  An event between
# two launches keeps the second from starting under the first (programmatic dependent launch), so these are the
# times of kernels run one after the other, not shares of a step replayed from a graph.
timeline: Optional[list] = None
tag = ""


class _Timed:
    def __init__(self, name: str):
        self.name = name

    def __enter__(self):
        if timeline is not None:
            self.e0, self.e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            self.e0.record()
        return self

    def __exit__(self, *exc):
        if timeline is not None:
            self.e1.record()
            timeline.append((tag, self.name, self.e0, self.e1))


def _call(name: str, *args) -> None:
    global launches, _last_call
    fn = _fns.get(name)
    if fn is None:
        fn = _fns[name] = getattr(_lib or require_extension(), name)
    if timeline is not None:
        with _Timed(name):
            rc = fn(*args)
    else:
        rc = fn(*args)
    if rc != 0:
        raise KernelError(_lib.me_last_error().decode())
    launches += 1
    _last_call = (fn, args)


# The same product or norm comes back step after step with the same tensors (the work buffers of a step are the
# same storage every time): a wrapper that finds its key here, with the same addresses, shapes and strides as when
# it was made, launches at once with the arguments of that time (and the stream of now) instead of checking and
# deciding everything again.  An eager step spends more host time on that than on the launches themselves.
_repeats: dict = {}
remember_launches = True  # False: every wrapper runs in full every time (a switch for comparisons)


def _repeat(key, sig) -> bool:
    global launches
    hit = _repeats.get(key) if remember_launches and timeline is None else None
    if hit is None or hit[0] != sig:
        return False
    if hit[1](*hit[2], _stream()) != 0:
        raise KernelError(_lib.me_last_error().decode())
    launches += 1
    return True


def _remember(key, sig, launches_before: int) -> None:
    """After a wrapper has run in full: keep its launch if it was exactly one, with the stream as last argument."""
    if launches == launches_before + 1 and _last_call is not None and _last_call[1][-1] == _stream():
        if len(_repeats) > 16384:
            _repeats.clear()
        _repeats[key] = (sig, _last_call[0], _last_call[1][:-1])


def forget_tensors() -> None:
    """Drop everything remembered about tensors seen so far (launch arguments, tensor maps): for a process that
    frees one engine and builds another."""
    _repeats.clear()
    _tensor_maps.clear()


_device_index: Optional[int] = None


def _stream() -> int:
    """The current stream's handle (a launch a few microseconds apart cannot afford torch's Stream object)."""
    global _device_index
    if _device_index is None:
        _device_index = torch.cuda.current_device()
    return torch._C._cuda_getCurrentRawStream(_device_index)


def _dt(t: torch.Tensor) -> int:
    try:
        return _DT[t.dtype]
    except KeyError:
        raise KernelError(f"dtype {t.dtype} is not supported by the kernels (float32 and bfloat16 are)") from None


def _ptr(t: Optional[torch.Tensor]) -> int:
    return 0 if t is None else t.data_ptr()


def _need(cond: bool, msg: str) -> None:
    if not cond:
        raise KernelError(msg)


_sm_count = 0


def sm_count() -> int:
    """Multiprocessors of the current device."""
    global _sm_count
    if not _sm_count:
        _sm_count = int((_lib or require_extension()).me_device_sm_count())
    return _sm_count


def wait_expires_selftest(err: torch.Tensor, limit: int = 4096) -> int:
    """Runs the kernel of csrc/selftest.cu: a bounded wait on a barrier that nothing completes.  It sets flag 1 of
    ``err`` (int32[4] on the device) as the tensor-map kernels do when a wait runs out; returns the polls made."""
    _need(err.dtype == torch.int32 and err.numel() >= 4 and err.is_cuda, "wait_expires_selftest: err must be int32[4] on the device")
    polls = torch.zeros(1, dtype=torch.int32, device=err.device)
    _call("me_test_wait_expires", err.data_ptr(), int(limit), polls.data_ptr(), _stream())
    return int(polls.item())


def check_attention_sizes(head_dim: int, num_heads: int, num_kv_heads: int) -> None:
    """What the attention kernels take; anything else is refused here, before any launch."""
    if head_dim % 16 or not 16 <= head_dim <= MAX_HEAD_DIM:
        raise ValueError(f"head_dim {head_dim} is not supported: the attention kernels take multiples "
                         f"of 16 from 16 to {MAX_HEAD_DIM}")
    if num_heads < 1 or num_kv_heads < 1 or num_heads % num_kv_heads:
        raise ValueError(f"{num_heads} heads with {num_kv_heads} key/value heads is not supported")


# ---- element-wise and normalisation ----------------------------------------------------
def embed(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor, err: torch.Tensor,
          feedback: Optional[torch.Tensor] = None, scale: float = 1.0, position_rows: Optional[tuple] = None,
          copy: Optional[torch.Tensor] = None) -> None:
    """Rows of ``table`` times ``scale`` into the float32 ``out`` [T, H], or into every stream of ``out`` [S, T, H].
    ``position_rows`` = (table [P, H] of the same dtype, int32 positions [T]): the row of a token's position is added.  ``copy`` [T, H]
    (any dtype, rows may lie apart) takes the same rows once more.
    An id ~j (negative) stands for ``feedback[j]`` (int32 on the device: the tokens the step before drew); ids
    outside the vocabulary set flag 0 of ``err``."""
    _need(ids.dtype == torch.int32 and ids.is_contiguous(), "embed: token ids must be contiguous int32")
    _need(feedback is None or (feedback.dtype == torch.int32 and feedback.is_contiguous()), "embed: feedback must be int32")
    _need(out.dtype == torch.float32 and out.is_contiguous() and table.is_contiguous(), "embed: bad tensors")
    T, (V, H) = ids.shape[0], table.shape
    copies = out.shape[0] if out.dim() == 3 else 1
    _need(tuple(out.shape[-2:]) == (T, H) and out.dim() in (2, 3), "embed: output shape")
    ptable, positions = position_rows if position_rows is not None else (None, None)
    _need(ptable is None or (ptable.is_contiguous() and ptable.dtype == table.dtype and ptable.dim() == 2 and ptable.shape[1] == H
                             and positions.dtype == torch.int32 and positions.is_contiguous() and positions.numel() == T),
          "embed: the table over positions is [positions, H] of the table's dtype, with an int32 position a token")
    _need(copy is None or (tuple(copy.shape) == (T, H) and copy.stride(1) == 1), "embed: the copy is [T, H]")
    _call("me_embed", ids.data_ptr(), table.data_ptr(), _dt(table), out.data_ptr(), T, H, V, err.data_ptr(), _ptr(feedback),
          feedback.numel() if feedback is not None else 0, float(scale), copies, T * H, _ptr(ptable), _ptr(positions),
          ptable.shape[0] if ptable is not None else 0, _ptr(copy), _dt(copy) if copy is not None else 0,
          copy.stride(0) if copy is not None else H, _stream())


def add_rmsnorm(residual: torch.Tensor, delta: Optional[torch.Tensor], weight: torch.Tensor, eps: float,
                out: torch.Tensor, rows: Optional[torch.Tensor] = None) -> None:
    """``residual += delta`` (float32, in place), ``out = rmsnorm(residual) * weight``; with ``rows``
    only those rows are read and ``residual`` is not written.  A 3-D ``delta`` [splits, T, H] holds the
    partial results of a split-K product; they are added in order."""
    key = ("add_rmsnorm", id(residual), id(delta), id(weight), id(out), id(rows))
    sig = (residual.data_ptr(), _ptr(delta), weight.data_ptr(), out.data_ptr(), _ptr(rows), residual.shape, residual.stride(),
           residual.dtype, None if delta is None else (delta.shape, delta.stride(), delta.dtype), weight.shape, weight.dtype,
           out.shape, out.stride(), out.dtype, None if rows is None else (rows.shape, rows.stride(), rows.dtype), eps)
    if _repeat(key, sig):
        return
    before = launches
    H = residual.shape[1]
    _need(residual.dtype == torch.float32 and residual.is_contiguous(), "add_rmsnorm: residual must be float32")
    _need(weight.dtype == torch.float32 and weight.shape == (H,), "add_rmsnorm: weight must be float32 [H]")
    n = residual.shape[0] if rows is None else rows.shape[0]
    _need(out.is_contiguous() and tuple(out.shape) == (n, H), "add_rmsnorm: output shape")
    splits, stride = 1, 0
    if delta is not None:
        if delta.dim() == 3:                      # partial results of a split-K product: [splits, T, H]
            splits, stride = delta.shape[0], delta.stride(0)
            _need(delta.is_contiguous() and tuple(delta.shape[1:]) == tuple(residual.shape), "add_rmsnorm: delta shape")
        else:
            _need(delta.is_contiguous() and delta.shape == residual.shape, "add_rmsnorm: delta shape")
    if rows is not None:
        _need(rows.dtype == torch.int32 and rows.is_contiguous(), "add_rmsnorm: rows must be int32")
    _call("me_add_rmsnorm", residual.data_ptr(), _ptr(delta), _dt(delta) if delta is not None else 0,
          weight.data_ptr(), float(eps), out.data_ptr(), _dt(out), _ptr(rows), n, H, splits, stride, _stream())
    _remember(key, sig, before)


def silu_mul(x: torch.Tensor, out: torch.Tensor) -> None:
    T, I2 = x.shape
    _need(I2 % 2 == 0 and tuple(out.shape) == (T, I2 // 2) and x.dtype == out.dtype, "silu_mul: shapes")
    _need(x.is_contiguous() and out.is_contiguous(), "silu_mul: contiguous tensors")
    _call("me_silu_mul", x.data_ptr(), out.data_ptr(), _dt(x), T, I2 // 2, _stream())


# ---- matrix products ----------------------------------------------------------------------
library_calls = 0         # cuBLAS products issued through torch (not counted as this package's kernels)


SKINNY_MAX_ROWS = 16      # rows up to which bfloat16 products run csrc/gemm_skinny.cu


def skinny_splits(M: int, K: int, x: torch.Tensor, weight: torch.Tensor) -> int:
    """How many float32 partial results the small-batch kernel would leave for this product
    (0: the kernel does not take it; 1: it writes the result itself)."""
    if not (x.is_cuda and x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and 0 < M <= SKINNY_MAX_ROWS
            and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and weight.data_ptr() % 16 == 0):
        return 0
    return (_lib or require_extension()).me_gemm_skinny_splits(K)


def linear_partials(x: torch.Tensor, weight: torch.Tensor, workspace, name: str,
                    err: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """``x @ weight.T`` as float32 partial results [splits, M, N] of a split-K product, for a consumer that
    adds them (``add_rmsnorm``); None when the product is not one that is split: the small-batch kernel splits long
    rows of few requests, the tcgen05 kernel products of a few hundred rows whose tiles would leave most SMs idle.
    ``err``: the int32[4] error word of the step (the tcgen05 kernel reports a wait that ran out there); without it
    the tcgen05 kernel is not used."""
    M, K = x.shape
    N = weight.shape[0]
    splits = skinny_splits(M, K, x, weight)
    if splits >= 2:
        part = workspace(name, (splits, M, N), torch.float32)
        _call("me_gemm_skinny", x.data_ptr(), x.stride(0), weight.data_ptr(), 0, 0, 0, part.data_ptr(), M, N, K, 0, _stream())
        return part
    if err is not None and use_tcgen05_gemm and tcgen05_takes(x, weight) and weight.is_contiguous():
        bn, parts = tcgen05_split_plan(M, N, K)
        if parts >= 2:
            part = workspace(name, (parts, M, N), torch.float32)
            linear_tcgen05(x, weight, part, "none", err, tile_n=bn, splits=parts)
            return part
    return None


DECODE_MAX_K = 3072       # largest K of csrc/gemm_decode.cu (one block covers all of K); beyond: csrc/gemm_stream.cu
# Which of the two kernels a decode product runs: "auto" (gemm_decode up to DECODE_MAX_K, gemm_stream beyond),
# "stream" (gemm_stream for every K) or "decode" (gemm_decode only; larger K is then not taken).  A switch for comparisons.
decode_kernel = "auto"


def _decode_uses_stream(K: int) -> bool:
    return decode_kernel == "stream" or (decode_kernel == "auto" and K > DECODE_MAX_K)


# Which products over a K beyond DECODE_MAX_K run csrc/gemm_stream.cu: "all", or "residual" (only those that add into
# the residual stream; the others go to the library).  A switch for comparisons.
stream_products = "all"
# Weights from this many elements on (32 MB of bfloat16: the LM head) go through csrc/gemm_stream.cu in ``linear`` too
# when the batch has up to 16 rows: a product that long is all stream, and that kernel streams fastest.
STREAM_MIN_WEIGHT_ELEMENTS = 1 << 24


def _decode_operands_ok(M: int, K: int, weight: torch.Tensor) -> bool:
    return (weight.is_cuda and weight.dtype == torch.bfloat16 and 0 < M <= SKINNY_MAX_ROWS and K % 8 == 0
            and weight.data_ptr() % 16 == 0)


def decode_linear_takes(M: int, K: int, weight: torch.Tensor, adds_to_residual: bool = True) -> bool:
    """Whether a decode product with norm / residual folded in (csrc/gemm_decode.cu, csrc/gemm_stream.cu: up to 16
    rows) takes the shape; ``adds_to_residual``: the product is one whose result is added to the residual stream."""
    if not _decode_operands_ok(M, K, weight):
        return False
    if _decode_uses_stream(K):
        return decode_kernel == "stream" or stream_products == "all" or adds_to_residual
    return K <= DECODE_MAX_K


_stream_ws: dict = {}


def _stream_work_buffers(device) -> tuple[torch.Tensor, torch.Tensor]:
    """What csrc/gemm_stream.cu needs beside its operands: room for the sums a block leaves to the block that finishes its
    group of rows, and a flag a block (zero between launches).  One pair a device: launches in one stream never overlap."""
    ws = _stream_ws.get(device)
    if ws is None:
        lib = _lib or require_extension()
        ws = _stream_ws[device] = (torch.empty(lib.me_gemm_stream_partial_floats(), dtype=torch.float32, device=device),
                                   torch.zeros(lib.me_gemm_stream_flag_ints(), dtype=torch.int32, device=device))
    return ws


_shared_ws: dict = {}


def _tcgen05_shared_buffers(device) -> tuple[torch.Tensor, torch.Tensor]:
    """The same for the work-sharing form of csrc/gemm_tcgen05.cu: a 128 x 256 tile of float32 sums a block, four flags a block."""
    ws = _shared_ws.get(device)
    if ws is None:
        lib = _lib or require_extension()
        ws = _shared_ws[device] = (torch.empty(lib.me_gemm_tcgen05_shared_partial_floats(), dtype=torch.float32, device=device),
                                   torch.zeros(lib.me_gemm_tcgen05_shared_flag_ints(), dtype=torch.int32, device=device))
    return ws


def reset_stream_work_buffers() -> None:
    """Clear the flags of the work buffers of csrc/gemm_stream.cu and of the work-sharing tcgen05 product.  Every launch
    leaves them zero, except one whose bounded wait ran out (flag 1 of the error word): the caller that reports that
    error calls this, so that a later launch does not take a stale flag for a neighbour's finished sums."""
    for _, flags in list(_stream_ws.values()) + list(_shared_ws.values()):
        flags.zero_()


def decode_linear_sumsq_parts(N: int, K: int = 0, stream: Optional[bool] = None) -> int:
    """Parts in which the residual epilogue of ``decode_linear`` writes sums of squares, for N columns over K
    (``stream``: by which of the two kernels; None: the one that ``decode_kernel`` picks for K)."""
    lib = _lib or require_extension()
    stream = _decode_uses_stream(K) if stream is None else stream
    return lib.me_gemm_stream_sumsq_parts(N, K) if stream else lib.me_gemm_decode_sumsq_parts(N)


def decode_linear(weight: torch.Tensor, x: torch.Tensor, *, out: Optional[torch.Tensor] = None, epilogue: str = "none",
                  row_scale=None, residual_out: Optional[torch.Tensor] = None, sumsq_out: Optional[torch.Tensor] = None,
                  next_norm=None, fetch_ahead: Optional[torch.Tensor] = None, err: Optional[torch.Tensor] = None,
                  kernel: Optional[str] = None, glu: Optional[tuple[float, float, float]] = None) -> None:
    """One decode product with its neighbours folded in (csrc/gemm_decode.cu, csrc/gemm_stream.cu; ``kernel``:
    "stream" asks for the latter whatever ``decode_kernel`` says).

    ``x``: bfloat16 [M, K].  ``row_scale`` = (sums of squares float32 [parts, M], eps): x is a residual times a
    norm's weight, and the float32 results of row m are multiplied by rsqrt(sum / K + eps), which completes that
    RMSNorm.  Output: ``out`` (epilogue "none" or "silu_mul") or ``residual_out`` (float32 [M, N], epilogue
    "residual": residual_out += x W^T; ``sumsq_out`` [decode_linear_sumsq_parts(N), M] gets the new residual's sums
    of squares per strip of columns, and with ``next_norm`` = (weight float32 [N], xw bfloat16 [M, N]) xw gets the new
    residual times that weight).  ``fetch_ahead``: a tensor that a later kernel reads (the next product's weight);
    this kernel asks it into L2.  ``epilogue`` may also be a key of ``ACTIVATIONS``: that function of the results.  ``glu`` = (limit, alpha, shift) with "silu_mul": the gated epilogue in its general form,
    g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit) when limit > 0."""
    epi = 3 + ACTIVATIONS[epilogue] if epilogue in ACTIVATIONS else {"none": 0, "silu_mul": 1, "residual": 2}[epilogue]
    _need(glu is None or epi == 1, "decode_linear: the gate's parameters go with the gated epilogue")
    glu_params = tuple(float(v) for v in (glu or (0.0, 1.0, 0.0)))
    M, K = x.shape
    _need(x.dtype == torch.bfloat16 and x.stride(1) == 1 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0, "decode_linear: x")
    stream = kernel == "stream" or _decode_uses_stream(K)
    _need((stream or K <= DECODE_MAX_K) and _decode_operands_ok(M, K, weight) and weight.shape[1] == K
          and weight.is_contiguous(), "decode_linear: shape not taken")
    sumsq, eps = row_scale if row_scale is not None else (None, 0.0)
    if sumsq is not None:
        _need(sumsq.dtype == torch.float32 and sumsq.is_contiguous() and sumsq.dim() == 2 and sumsq.shape[1] == M,
              "decode_linear: sums of squares")
    N = weight.shape[0] // 2 if epi == 1 else weight.shape[0]
    nw, xw = next_norm if next_norm is not None else (None, None)
    if epi == 2:
        _need(residual_out.dtype == torch.float32 and residual_out.is_contiguous() and tuple(residual_out.shape) == (M, N)
              and sumsq_out.dtype == torch.float32 and sumsq_out.is_contiguous()
              and tuple(sumsq_out.shape) == (decode_linear_sumsq_parts(N, K, stream), M), "decode_linear: residual output")
        if nw is not None:
            _need(nw.dtype == torch.float32 and tuple(nw.shape) == (N,) and nw.is_contiguous() and xw.dtype == torch.bfloat16
                  and tuple(xw.shape) == (M, N) and xw.is_contiguous(), "decode_linear: pre-weighted output")
        yp, ydt, ldy = 0, 0, 0
    else:
        _need(next_norm is None, "decode_linear: the pre-weighted output belongs to the residual epilogue")
        _need(tuple(out.shape) == (M, N) and out.stride(1) == 1, "decode_linear: output shape")
        yp, ydt, ldy = out.data_ptr(), _dt(out), out.stride(0)
    if stream:
        _need(err is not None, "decode_linear: the streaming kernel needs the step's error word (err=)")
        lib = _lib or require_extension()
        partials, flags = _stream_work_buffers(x.device)
        _call("me_gemm_stream", epi, matrix_tensor_map(x, lib.me_gemm_stream_x_box_rows(M)).ptr, _ptr(sumsq),
              sumsq.shape[0] if sumsq is not None else 0, float(eps), matrix_tensor_map(weight, lib.me_gemm_stream_w_box_rows(epi)).ptr, yp, ydt, ldy,
              _ptr(residual_out), _ptr(sumsq_out), _ptr(nw), _ptr(xw), M, N, K, partials.data_ptr(), flags.data_ptr(),
              err.data_ptr(), *glu_params, _stream())
        return
    _call("me_gemm_decode", epi, x.data_ptr(), x.stride(0), _ptr(sumsq), sumsq.shape[0] if sumsq is not None else 0, float(eps),
          weight.data_ptr(), yp, ydt, ldy, _ptr(residual_out), _ptr(sumsq_out), _ptr(nw), _ptr(xw), M, N, K,
          _ptr(fetch_ahead), fetch_ahead.numel() * fetch_ahead.element_size() if fetch_ahead is not None else 0, *glu_params,
          _stream())


TCGEN05_MIN_ROWS = 128    # rows from which bfloat16 products run csrc/gemm_tcgen05.cu whatever the weight (fewer: cuBLAS) ...
# ... and from 48 rows on where the weight is small (up to 8 M elements: every product of a layer at the 0.6B sizes).  There a
# decode step of 64 requests takes 2.39 ms against 2.44 with the library's products and a SiLU kernel, one of 96 requests 3.36
# against 3.50 (32 requests: level); at the 8B and 32B sizes, where such a product streams 30 to 260 MB of weights over a
# half-empty tile of rows, the library is 5 to 12% ahead and keeps them.
TCGEN05_SMALL_MIN_ROWS = 48
TCGEN05_SMALL_MAX_WEIGHT_ELEMENTS = 8 << 20
use_tcgen05_gemm = True   # False: such products go to cuBLAS instead (a switch for comparisons)


def tcgen05_min_rows(weight_elements: int) -> int:
    """Rows from which a product with a weight of that many elements runs the tcgen05 kernels."""
    return min(TCGEN05_MIN_ROWS, TCGEN05_SMALL_MIN_ROWS) if weight_elements <= TCGEN05_SMALL_MAX_WEIGHT_ELEMENTS else TCGEN05_MIN_ROWS


def matrix_tensor_map(t: torch.Tensor, box_rows: int) -> "TensorMap":
    """The tensor map of a row-major bfloat16 matrix [rows, cols] (row pitch ``t.stride(0)``) with boxes of
    ``box_rows`` x 64 columns and the 128-byte swizzle; cached by address and shape."""
    key = (t.data_ptr(), t.shape[0], t.shape[1], t.stride(0), box_rows)
    tm = _tensor_maps.get(key)
    if tm is None:
        if len(_tensor_maps) > 8192:
            _tensor_maps.clear()
            _repeats.clear()          # remembered launches hold the addresses of the maps just dropped
        tm = TensorMap()
        lib = _lib or require_extension()
        if lib.me_tma_encode_2d(tm.ptr, t.data_ptr(), t.shape[0], t.shape[1], t.stride(0) * 2, box_rows, 64, 128) != 0:
            raise KernelError(lib.me_last_error().decode())
        _tensor_maps[key] = tm
    return tm


def tcgen05_takes(x: torch.Tensor, weight: torch.Tensor) -> bool:
    M, K = x.shape
    return (x.is_cuda and x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and M >= tcgen05_min_rows(weight.numel())
            and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and weight.data_ptr() % 16 == 0)


tcgen05_persistent = "auto"     # the persistent form of the tcgen05 product: "auto", True or False (for comparisons)


def tcgen05_persistent_pays(M: int, N: int, K: int, epi: int) -> bool:
    """Whether a product of M rows and N output columns runs the persistent form of the tcgen05 kernel (one block an
    SM walking 128 x 256 tiles with two accumulators): from two tiles an SM on (a little earlier where K is short and a
    tile's fixed part weighs more: q|k|v of 2,048 rows at the 0.6B sizes).  There the loads of the next tile and
    the epilogue of the last one run beside a tile's products, which is worth a fifth to a third of gate|up at every
    size measured and of q|k|v at 2,048 rows; with fewer tiles (o_proj, down_proj up to a few thousand rows) the form
    with two blocks an SM is level or ahead."""
    out_cols = 128 if epi else 256
    tiles = ((M + 127) // 128) * ((N + out_cols - 1) // out_cols)
    return tiles >= 2 * sm_count() or (K <= 1024 and 10 * tiles >= 17 * sm_count())


tcgen05_share = "auto"          # the work-sharing form of the tcgen05 product: "auto" or False (for comparisons)


def tcgen05_share_pays(M: int, N: int, K: int, epi: int) -> bool:
    """Whether a product of M rows and N output columns runs the work-sharing form of the tcgen05 kernel (the last
    rounds' stages cut into one equal range an SM, partial sums added by the tile's owner).  It pays where whole tiles
    leave SMs idle: a last round that is less than half full (1.1 or 2.2 tiles of 128 x 256 an SM: q|k|v of 1,024 rows at
    the 8B sizes 52 against 66 us, o_proj of 1,024 rows at the 32B sizes 79 against 124), or fewer tiles than SMs with a
    long K and up to 512 rows (q|k|v of 256 rows at the 32B sizes 55 against 75 us, down_proj of 512 rows at the 8B sizes
    74 against 90).  It does not pay with the SiLU epilogue (many tiles anyway), nor where the blocks that share a tile of
    W, now at different places along K, push each other's part of it out of L2: down_proj of 1,024 rows at the 8B sizes
    (eight tiles to a tile of W, 128 tiles for 148 SMs) took 124 against 90 us and read 670 MB from DRAM for operands of
    126 MB; hence the bound on the rows there, and on the operands' bytes where there are more tiles than SMs (wins were
    measured up to 117 MB: q|k|v of 512 and 1,024 rows at the 32B sizes 61 against 97 and 117 against 134 us)."""
    if epi:
        return False
    sms = sm_count()
    tiles = ((M + 127) // 128) * ((N + 255) // 256)
    if tiles >= sms:
        # (K: handing a tile's sums over costs 3 to 5 us, a tile of K = 1,024 takes 5: at the 0.6B sizes it never paid)
        rounds = -(-tiles // sms)
        return K >= 4096 and tiles <= 0.75 * rounds * sms and (M + N) * K * 2 <= 128 << 20
    return 5 * tiles >= sms and K >= 5120 and M <= 512


def tcgen05_one_round_width(M: int, N: int) -> int:
    """The tile width (256 or 128) at which a product of M rows and N columns has about one tile an SM, or 0."""
    sms, m_tiles = sm_count(), (M + 127) // 128
    if 0.85 * sms <= m_tiles * ((N + 255) // 256) <= sms:
        return 256
    if 0.8 * sms <= m_tiles * ((N + 127) // 128) < 2 * sms:
        return 128
    return 0


def linear_tcgen05(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, epilogue: str, err: torch.Tensor,
                   tile_n: Optional[int] = None, splits: int = 1, persistent: Optional[bool] = None,
                   share: Optional[bool] = None, glu: Optional[tuple[float, float, float]] = None) -> None:
    """The tcgen05 product of csrc/gemm_tcgen05.cu: TMA -> swizzled shared memory -> tcgen05.mma -> tensor memory.

    ``glu`` = (limit, alpha, shift) with the "silu_mul" epilogue: the gated epilogue in its general form,
    g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit) when limit > 0.  ``epilogue`` may also
    be a key of ``ACTIVATIONS``: that function of the results (bfloat16).

    With ``splits`` > 1 ``out`` is float32 [tcgen05_splits(K, splits), M, N]: partial results over parts of K.
    ``share``: the form that cuts the stages of all tiles into one equal range an SM (``tile_n`` 128 or 256)."""
    M, K = x.shape
    act = 2 + ACTIVATIONS[epilogue] if epilogue in ACTIVATIONS else 0       # (as for no epilogue, but for the call itself)
    epi = 0 if act else {"none": 0, "silu_mul": 1}[epilogue]
    _need(not act or (splits == 1 and out.dtype == torch.bfloat16), "linear_tcgen05: an activation goes with whole sums and bfloat16 results")
    _need(glu is None or epi == 1, "linear_tcgen05: the gate's parameters go with the gated epilogue")
    glu_params = tuple(float(v) for v in (glu or (0.0, 1.0, 0.0)))
    N = weight.shape[0] // 2 if epi else weight.shape[0]
    if share is None and tile_n is None and persistent is None and splits == 1 and tcgen05_share == "auto" and tcgen05_takes(x, weight):
        share = tcgen05_share_pays(M, N, K, epi)
    if share and (glu is not None or act):
        share = False                 # (the work-sharing form has no gated epilogue in its general form and no activation)
    if share:
        bn = tile_n or 256
        _need(tcgen05_takes(x, weight) and splits == 1 and bn in (128, 256), "linear_tcgen05: operands not taken by the work-sharing form")
        partials, flags = _tcgen05_shared_buffers(x.device)
        _call("me_gemm_tcgen05_shared", matrix_tensor_map(x, 128).ptr, matrix_tensor_map(weight, bn // 2 if epi else bn).ptr,
              out.data_ptr(), _dt(out), out.stride(0), M, N, K, epi, bn, partials.data_ptr(), flags.data_ptr(), err.data_ptr(), _stream())
        return
    if tile_n is None:
        # The widest accumulator that still leaves enough tiles: about two an SM where a tile is short (K up to 3,072),
        # one for every other SM where it is long (measured at the 8B and 32B sizes: with 512 rows the 256-wide tile is a
        # third faster than the 64-wide one that two tiles an SM would ask for).  The SiLU epilogue (half as many output
        # columns per tile) does best at 128 while both the rows and K are few, and again where the output is so large
        # (a quarter of a GB and more) that the wide tiles' order through it stops fitting L2.
        m_tiles = (M + 127) // 128
        if persistent is None and tcgen05_persistent == "auto" and splits == 1 and tcgen05_persistent_pays(M, N, K, epi):
            tile_n, persistent = 256, True
        elif persistent is None and tcgen05_persistent == "auto" and splits == 1 and not epi and K <= 3072 and (
                tcgen05_one_round_width(M, N)):
            # about one tile an SM and a short K (o_proj and down_proj of 2,048 and 4,096 rows at the 0.6B sizes): a block that
            # has the SM to itself, with the persistent form's deeper ring, beats two blocks an SM on narrower tiles (10.0 and
            # 13.2 us against 11.4 and 15.3 at 2,048 rows, 14.6 and 19.2 against 15.1 and 21.0 at 4,096)
            tile_n, persistent = tcgen05_one_round_width(M, N), True
        elif epi:
            tile_n = 256 if (M >= 4096 or K >= 4096) and m_tiles * ((N + 127) // 128) <= 10000 else 128
        else:
            need = 200 if K < 4096 else 64
            tile_n = next((bn for bn in (256, 128) if m_tiles * ((N + bn - 1) // bn) >= need), 64)
    bn = tile_n
    _need(tcgen05_takes(x, weight) or M < tcgen05_min_rows(weight.numel()), "linear_tcgen05: operands not taken")
    box_w = bn // 2 if epi else bn
    if splits > 1:
        _need(out.dim() == 3 and out.shape[0] == tcgen05_splits(K, splits) and out.dtype == torch.float32 and out.is_contiguous(),
              "linear_tcgen05: partial results must be float32 [splits, M, N]")
        ldc, split_stride = out.stride(1), out.stride(0)
    else:
        ldc, split_stride = out.stride(0), 0
    if persistent is None:
        persistent = tcgen05_persistent
    if persistent == "auto":
        persistent = False
    if persistent and splits == 1 and bn >= 128:
        _call("me_gemm_tcgen05_persistent", matrix_tensor_map(x, 128).ptr, matrix_tensor_map(weight, box_w).ptr, out.data_ptr(),
              _dt(out), ldc, M, N, K, act or epi, bn, *glu_params, err.data_ptr(), _stream())
        return
    _call("me_gemm_tcgen05", matrix_tensor_map(x, 128).ptr, matrix_tensor_map(weight, box_w).ptr, out.data_ptr(), _dt(out),
          ldc, M, N, K, act or epi, bn, splits, split_stride, *glu_params, err.data_ptr(), _stream())


def tcgen05_splits(K: int, splits: int) -> int:
    """Partial results that ``linear_tcgen05`` writes when asked to split K ``splits`` ways (whole blocks of 64)."""
    return (_lib or require_extension()).me_gemm_tcgen05_splits(K, splits)


TCGEN05_SPLIT_MAX_ROWS = 1024      # rows up to which a product with few tiles is split along K


def tcgen05_split_plan(M: int, N: int, K: int) -> tuple[int, int]:
    """(tile width, parts of K) for a product of ``M`` rows whose consumer adds float32 partial results, or (0, 1).

    A product of a few hundred rows by a thousand columns has a handful of tiles for 148 SMs; shared out along K
    four ways it ran 25 to 40% faster (o_proj and down_proj of the 0.6B shape at 512 and 1,024 rows), at 2,048 rows
    no faster once the partial results are added."""
    if not (tcgen05_min_rows(N * K) <= M <= TCGEN05_SPLIT_MAX_ROWS):
        return 0, 1
    m_tiles = (M + 127) // 128
    bn = 64 if m_tiles * ((N + 127) // 128) * 4 < 128 else 128
    tiles = m_tiles * ((N + bn - 1) // bn)
    want = max(1, min(4, 256 // max(tiles, 1), K // 512))
    parts = tcgen05_splits(K, want)
    return (bn, parts) if parts >= 2 and tcgen05_splits(K, parts) == parts else (0, 1)


def linear_activation_takes(x: torch.Tensor, weight: torch.Tensor, out: Optional[torch.Tensor], err: Optional[torch.Tensor]) -> bool:
    """Whether ``linear`` takes a key of ``ACTIVATIONS`` as epilogue for these operands: the tcgen05 kernels do."""
    return (err is not None and use_tcgen05_gemm and skinny_splits(x.shape[0], x.shape[1], x, weight) == 0 and tcgen05_takes(x, weight)
            and (out is None or out.dtype == torch.bfloat16))


def linear(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, epilogue: str = "none",
           workspace=None, err: Optional[torch.Tensor] = None) -> None:
    """``out = x @ weight.T`` with float32 accumulation; ``epilogue="silu_mul"`` takes a weight of
    rows gate | up and writes ``silu(x Wg^T) * (x Wu^T)``.

    float32 operands (and any mix of dtypes) run the CUDA-core kernel of csrc/gemm_simt.cu: plain
    FMA, no reduced-precision matrix mode.  bfloat16 x bfloat16 products of up to 16 rows run csrc/gemm_stream.cu
    where the weight has 32 MB and more (the vocabulary product of a decode step) and csrc/gemm_skinny.cu else
    (the layers' own products in decode do not come here: ``decode_linear``); 128 rows and more, and 48 rows and more
    where the weight is small (``tcgen05_min_rows``), run the tcgen05 kernels of csrc/gemm_tcgen05.cu; the rows between,
    and shapes those refuse (K no multiple of 8), go to cuBLAS, as all the
    reference's products do through ``F.linear`` (layers/linear.py:26,45), with SiLU-and-multiply as a kernel of ours
    behind it.

    ``err``: the int32[4] error word of the step; the tcgen05 kernel sets flag 1 there when one of its bounded
    waits runs out.  Without it products of 128 rows and more go to cuBLAS."""
    global library_calls
    key = ("linear", id(x), id(weight), id(out), epilogue)
    sig = (x.data_ptr(), weight.data_ptr(), out.data_ptr(), _ptr(err), x.shape, x.stride(), x.dtype, weight.shape,
           weight.stride(), weight.dtype, out.shape, out.stride(), out.dtype, use_tcgen05_gemm)
    if _repeat(key, sig):
        return
    before = launches
    M, K = x.shape
    _need(weight.dim() == 2 and weight.shape[1] == K and weight.is_contiguous(), "linear: weight shape")
    _need(x.stride(1) == 1 and out.stride(1) == 1, "linear: rows must be contiguous")
    if epilogue in ACTIVATIONS:
        _need(linear_activation_takes(x, weight, out, err), "linear: no kernel of this shape applies an activation to its results")
        linear_tcgen05(x, weight, out, epilogue, err)
        _remember(key, sig, before)
        return
    epi = {"none": 0, "silu_mul": 1}[epilogue]
    N = weight.shape[0] // 2 if epi else weight.shape[0]
    _need(tuple(out.shape) == (M, N), f"linear: output is {tuple(out.shape)}, expected {(M, N)}")
    if M == 0:
        return
    if (err is not None and epi == 0 and weight.numel() >= STREAM_MIN_WEIGHT_ELEMENTS and skinny_splits(M, K, x, weight) > 0
            and out.dtype in (torch.bfloat16, torch.float32)):
        decode_linear(weight, x, out=out, err=err, kernel="stream")
        _remember(key, sig, before)
        return
    if skinny_splits(M, K, x, weight) == 1 and (epi == 0 or out.dtype == torch.bfloat16):
        _call("me_gemm_skinny", x.data_ptr(), x.stride(0), weight.data_ptr(), out.data_ptr(), _dt(out), out.stride(0),
              0, M, N, K, epi, _stream())
        _remember(key, sig, before)
        return
    if err is not None and use_tcgen05_gemm and tcgen05_takes(x, weight) and (epi == 0 or out.dtype == torch.bfloat16):
        linear_tcgen05(x, weight, out, epilogue, err)
        _remember(key, sig, before)
        return
    if x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and x.is_cuda:
        if epi == 0 and out.dtype == torch.bfloat16:
            with _Timed("library_mm"):
                torch.mm(x, weight.t(), out=out)
            library_calls += 1
            return
        if epi == 0 and out.dtype == torch.float32:
            with _Timed("library_mm"):
                torch.mm(x, weight.t(), out_dtype=torch.float32, out=out)
            library_calls += 1
            return
        if epi == 1 and out.dtype == torch.bfloat16 and workspace is not None:
            tmp = workspace("linear_gate_up", (M, 2 * N), torch.bfloat16)
            with _Timed("library_mm"):
                torch.mm(x, weight.t(), out=tmp)
            library_calls += 1
            silu_mul(tmp, out)
            return
    _call("me_gemm_simt", x.data_ptr(), _dt(x), x.stride(0), weight.data_ptr(), _dt(weight),
          out.data_ptr(), _dt(out), out.stride(0), M, N, K, epi, _stream())


# ---- attention ------------------------------------------------------------------------------
ROTARY_LAYOUTS = ("half_split",)     # what the kernels rotate: element i with element i + rotary_dim / 2, i < rotary_dim / 2


def check_rotary(cos_sin: Optional[torch.Tensor], head_dim: int, rotary_dim: Optional[int], layout: str) -> int:
    """The rotary contract between a position encoding and the kernels: a float32 table [positions, rotary_dim]
    (cosines of the rotary_dim / 2 frequencies, then their sines), ``rotary_dim`` even and at most ``head_dim``
    (elements from rotary_dim on are left unrotated), and a layout the kernels know by name.  Returns rotary_dim."""
    if layout not in ROTARY_LAYOUTS:
        raise KernelError(f"rotary layout {layout!r} is not supported by the kernels (they take: {', '.join(ROTARY_LAYOUTS)}); "
                          "another pairing of elements needs another kernel branch")
    if cos_sin is None:
        return head_dim
    rd = head_dim if rotary_dim is None else int(rotary_dim)
    _need(rd % 2 == 0 and 2 <= rd <= head_dim, f"rotary_dim {rd} must be even and at most head_dim {head_dim}")
    _need(cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.dim() == 2 and cos_sin.shape[1] == rd,
          f"the rotary table must be float32 [positions, rotary_dim = {rd}]")
    return rd


def qk_norm_rope_kv_write(qkv: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
                          q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor], eps: float,
                          cos_sin: Optional[torch.Tensor], positions: torch.Tensor,
                          slot_mapping: Optional[torch.Tensor], pool: torch.Tensor, page_size: int,
                          rotary_dim: Optional[int] = None, layout: str = "half_split") -> None:
    """In place on the packed rows q|k|v: RMSNorm of every q and k head, rotary embedding of the first
    ``rotary_dim`` elements of each (default: all of them), and the write of k and v to ``pool``
    [pages, 2, kv_heads, page_size, head_dim] at ``slot_mapping``."""
    T = qkv.shape[0]
    _need(qkv.stride(1) == 1 and qkv.shape[1] == (num_heads + 2 * num_kv_heads) * head_dim, "qk_norm_rope: qkv shape")
    _need(pool.dtype == qkv.dtype and pool.is_contiguous()
          and tuple(pool.shape[1:]) == (2, num_kv_heads, page_size, head_dim), "qk_norm_rope: pool shape")
    for w in (q_weight, k_weight):
        if w is not None:
            _need(w.dtype == torch.float32 and w.shape == (head_dim,), "qk_norm_rope: norm weights are float32 [head_dim]")
    rd = check_rotary(cos_sin, head_dim, rotary_dim, layout)
    _need(positions.dtype == torch.int32 and positions.shape[0] == T, "qk_norm_rope: positions")
    if slot_mapping is not None:
        _need(slot_mapping.dtype == torch.int32 and slot_mapping.shape[0] == T, "qk_norm_rope: slot mapping")
    _call("me_qk_norm_rope_kv_write", qkv.data_ptr(), _dt(qkv), qkv.stride(0), T, num_heads, num_kv_heads,
          head_dim, _ptr(q_weight), _ptr(k_weight), float(eps), _ptr(cos_sin), rd, positions.data_ptr(),
          _ptr(slot_mapping), pool.data_ptr(), page_size, _stream())


def attention_chunks(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta,
                     scale, window, tiles=None, num_tiles=None) -> None:
    """The CUDA-core chunk kernel over query tiles of 16 tokens (requests that bring several tokens)."""
    if tiles is None:
        tiles, num_tiles = meta.tile_lists[ATTN_TILE_Q]
    _call("me_attn_chunk", qkv.data_ptr(), _dt(qkv), qkv.stride(0), out.data_ptr(), out.stride(0),
          pool.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(),
          meta.context_lens.data_ptr(), tiles.data_ptr(), num_tiles, num_heads, num_kv_heads, head_dim,
          page_size, float(scale), int(window or 0), _stream())


def prefill_heads_per_block(num_heads: int, num_kv_heads: int, head_dim: int) -> int:
    """How many heads of a group share a block of the tensor-core prefill kernel; 0 if it refuses the shape."""
    return (_lib or require_extension()).me_attn_prefill_heads_per_block(num_heads, num_kv_heads, head_dim)


def attention_prefill(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta,
                      scale, window, tiles=None, num_tiles=None) -> None:
    """The tensor-core prefill kernel (bfloat16, head_dim 64 or 128) over tiles of 64 / heads-per-block tokens."""
    gp = prefill_heads_per_block(num_heads, num_kv_heads, head_dim)
    _need(gp > 0 and qkv.dtype == torch.bfloat16, "attention_prefill: shape or dtype not taken by the tensor-core kernel")
    if tiles is None:
        tiles, num_tiles = meta.tile_lists[64 // gp]
    _call("me_attn_prefill", qkv.data_ptr(), qkv.stride(0), out.data_ptr(), out.stride(0), pool.data_ptr(),
          block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(),
          tiles.data_ptr(), num_tiles, num_heads, num_kv_heads, head_dim, page_size, float(scale),
          int(window or 0), _stream())


DECODE_KINDS = {"auto": 0, "cuda_cores": 1, "tensor_cores": 3, "tensor_cores_tma": 4}

_tensor_maps: dict = {}


class TensorMap:
    """A CUtensorMap (128 bytes, 64-byte aligned) kept alive on the host for kernels that take it by value."""

    def __init__(self):
        self._raw = ctypes.create_string_buffer(128 + 64)
        self.ptr = (ctypes.addressof(self._raw) + 63) & ~63


def kv_tensor_map(pool: torch.Tensor, page_size: int) -> Optional[TensorMap]:
    """The tensor map of one cache slot [pages, 2, kv_heads, page_size, head_dim] (bfloat16) as the 2-D tensor
    [pages * 2 * kv_heads * page_size, head_dim] with boxes of one page x 64 columns, 128-byte swizzle;
    None where the tensor-map kernels do not apply."""
    hd = pool.shape[-1]
    if pool.dtype != torch.bfloat16 or hd not in (64, 128) or page_size < 8 or DECODE_PARTITION % page_size:
        return None
    key = (pool.data_ptr(), tuple(pool.shape))
    tm = _tensor_maps.get(key)
    if tm is None:
        tm = TensorMap()
        rows = pool.shape[0] * 2 * pool.shape[2] * page_size
        lib = _lib or require_extension()
        if lib.me_tma_encode_2d(tm.ptr, pool.data_ptr(), rows, hd, hd * 2, page_size, 64, 128) != 0:
            raise KernelError(lib.me_last_error().decode())
        _tensor_maps[key] = tm
    return tm


def prefill_tcgen05_heads_per_block(num_heads: int, num_kv_heads: int, head_dim: int, page_size: int) -> int:
    """How many heads of a group share a block of the tcgen05 prefill kernel; 0 if it refuses the shape."""
    return (_lib or require_extension()).me_attn_prefill_tcgen05_heads_per_block(num_heads, num_kv_heads, head_dim, page_size)


def attention_prefill_tcgen05(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta,
                              scale, window, tiles=None, num_tiles=None, key_tile: int = 0, sink: bool = False,
                              gate: Optional[torch.Tensor] = None, keep_first: int = 0, chunk: int = 0, softcap: float = 0.0,
                              sinks: Optional[torch.Tensor] = None, pooled: Optional[tuple] = None, bias: Optional[tuple] = None,
                              out_dim: int = 0, pairs: Optional[tuple[float, float, float]] = None, gate_heads: bool = False) -> None:
    """The tcgen05 / tensor-memory prefill kernel (bfloat16, head_dim 64 or 128, page sizes dividing 128) over
    tiles of 128 / heads-per-block tokens; Q, K and V arrive by tensor-map loads.  ``sink``: one more term, exp(0), in
    the softmax's denominator; ``gate``: float32 rows of pre-activations whose sigmoid multiplies the output.
    ``keep_first``: the window also shows the keys j < keep_first; ``chunk`` (instead of a window): the keys of the query's
    own chunk; ``softcap`` c: scores become c tanh(s / c) after the scale; ``sinks`` (float32 [heads]): the extra term is
    exp(sinks[head]); ``pooled`` = (cache, block tables, P): the blocks of P tokens in front of the window, one row each in a
    second cache of the same layout; ``bias`` = (r1, r2), float32 [heads] each: r1 ln(1 + r2 (p - j)) is taken off the scaled score
    of a key at distance p - j; ``out_dim`` (0: all): how many elements of every head leave, ``out`` then holds
    heads * out_dim columns; ``pairs`` = (lambda, gain, eps): heads 2h and 2h + 1 leave joined as ``diff_combine`` joins them;
    ``gate_heads``: the gate has one pre-activation a head (all of these in the kernel with the key tile of 128 only)."""
    gp = prefill_tcgen05_heads_per_block(num_heads, num_kv_heads, head_dim, page_size)
    _need(gp > 0 and qkv.dtype == torch.bfloat16 and qkv.is_contiguous() and qkv.data_ptr() % 16 == 0,
          "attention_prefill_tcgen05: shape or dtype not taken by the kernel")
    tq = 128 // gp
    if tiles is None:
        tiles, num_tiles = meta.tile_lists[tq]
    _call("me_attn_prefill_tcgen05", matrix_tensor_map(qkv, tq).ptr, kv_tensor_map(pool, page_size).ptr, out.data_ptr(),
          out.stride(0), block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(),
          meta.context_lens.data_ptr(), tiles.data_ptr(), num_tiles, num_heads, num_kv_heads, head_dim, page_size,
          float(scale), int(window or 0), key_tile, 1 if sink else 0, _ptr(gate), gate.stride(0) if gate is not None else 0,
          meta.error_flag.data_ptr(), int(keep_first or 0), int(chunk or 0), float(softcap or 0.0), _ptr(sinks),
          kv_tensor_map(pooled[0], page_size).ptr if pooled else 0, pooled[1].data_ptr() if pooled else 0,
          pooled[1].stride(0) if pooled else 0, int(pooled[2]) if pooled else 0, _ptr(bias[0]) if bias else 0, _ptr(bias[1]) if bias else 0,
          int(out_dim), 1 if pairs else 0, *(float(v) for v in (pairs or (0.0, 0.0, 0.0))), 1 if gate_heads else 0, _stream())


use_tcgen05_attention = True   # False: portions of prompts use the mma.sync kernel instead (a switch for comparisons)


def attention_decode(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta,
                     scale, window, kind: str = "auto", sink: bool = False, gate: Optional[torch.Tensor] = None,
                     keep_first: int = 0, chunk: int = 0, softcap: float = 0.0, sinks: Optional[torch.Tensor] = None,
                     pooled: Optional[tuple] = None, bias: Optional[tuple] = None, out_dim: int = 0,
                     pairs: Optional[tuple[float, float, float]] = None, gate_heads: bool = False) -> None:
    """The split-K decode kernel and its merge over requests [0, meta.num_decodes).  ``sink``: one more term, exp(0), in
    the softmax's denominator (added once, in the merge); ``gate``: float32 rows of pre-activations whose sigmoid
    multiplies the output.  ``sinks`` (float32 [heads]): the term is exp(sinks[head]).  ``keep_first``, ``chunk`` and
    ``softcap``, ``bias`` and ``out_dim`` as for ``attention_prefill_tcgen05`` (the partition kernel fed by tensor-map loads only).
    ``pairs`` = (lambda, gain, eps): the merge joins heads 2h and 2h + 1 as ``diff_combine`` does and ``out`` holds half as many heads.
    ``gate_heads``: the gate has one pre-activation a head.

    ``kind`` picks the partition kernel: "auto" (for bfloat16 with head_dim 64 or 128 the tensor cores, fed by
    tensor-map loads where the page size divides 128, else by cp.async; otherwise the CUDA cores), or one
    of them by name (tests run each)."""
    D = meta.num_decodes
    parts = max(1, (meta.max_context_len + DECODE_PARTITION - 1) // DECODE_PARTITION)
    room = max(parts, (getattr(meta, "scratch_context_len", 0) + DECODE_PARTITION - 1) // DECODE_PARTITION)
    pool_parts = 0
    if pooled is not None:
        # ``pooled`` = (cache, block tables, P): a second launch over the cache of pooled blocks fills the last slots of a head
        rows = lambda n: ((n + int(pooled[2]) - 1) // int(pooled[2]) + DECODE_PARTITION - 1) // DECODE_PARTITION
        pool_parts = max(1, rows(meta.max_context_len))
        parts, room = parts + pool_parts, room + max(pool_parts, rows(getattr(meta, "scratch_context_len", 0)))
    tmp_out = meta.workspace("decode_tmp_out", (D * num_heads * room * head_dim,), torch.float32)
    tmp_ml = meta.workspace("decode_tmp_ml", (2, D * num_heads * room), torch.float32)
    tm = kv_tensor_map(pool, page_size) if kind in ("auto", "tensor_cores_tma") else None
    _call("me_attn_decode", qkv.data_ptr(), _dt(qkv), qkv.stride(0), out.data_ptr(), out.stride(0),
          pool.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(),
          meta.context_lens.data_ptr(), D, num_heads, num_kv_heads, head_dim, page_size, float(scale),
          int(window or 0), tmp_out.data_ptr(), tmp_ml[0].data_ptr(), tmp_ml[1].data_ptr(), parts,
          _ptr(meta.error_flag), DECODE_KINDS[kind], tm.ptr if tm is not None else 0, 1 if sink else 0, _ptr(gate),
          gate.stride(0) if gate is not None else 0, int(keep_first or 0), int(chunk or 0), float(softcap or 0.0), _ptr(sinks),
          kv_tensor_map(pooled[0], page_size).ptr if pooled else 0, pooled[1].data_ptr() if pooled else 0,
          pooled[1].stride(0) if pooled else 0, int(pooled[2]) if pooled else 0, pool_parts, _ptr(bias[0]) if bias else 0,
          _ptr(bias[1]) if bias else 0, int(out_dim), 1 if pairs else 0, *(float(v) for v in (pairs or (0.0, 0.0, 0.0))), 1 if gate_heads else 0,
          _stream())
    global launches
    launches += 2 if pooled else 1          # partition kernel(s) + merge kernel


def decode_fused_takes(qkv: torch.Tensor, head_dim: int, pool: torch.Tensor, page_size: int, meta,
                       rotary_dim: Optional[int] = None) -> bool:
    """Whether ``attention_decode_fused`` takes the step: bfloat16, head size 64 or 128, pages of 8 to 128 tokens
    that divide 128, a tensor map over the cache, and a rotation over the whole head (or none)."""
    lib = _lib or require_extension()
    return (qkv.is_cuda and (rotary_dim is None or rotary_dim == head_dim) and qkv.dtype == torch.bfloat16 and pool.dtype == torch.bfloat16 and meta.error_flag is not None
            and bool(lib.me_attn_decode_fused_takes(head_dim, page_size)) and (qkv.stride(0) * 2) % 16 == 0
            and kv_tensor_map(pool, page_size) is not None)


# The form of the decode partition kernel: "one_tile" (K and V pass through the same shared-memory tile, five blocks
# an SM), "two_tiles" (a tile each, three blocks an SM) or "tile_and_half" (half a tile for V beside K's, four blocks).
DECODE_FORMS = {"one_tile": 0, "two_tiles": 2, "tile_and_half": 3}
# "auto": by the number of partitions with keys.  Up to what three blocks an SM hold at once, two tiles (all loads in
# flight together); beyond, one tile (more blocks an SM).  In a step of the 0.6B shape at 1,024 tokens of context:
# batch 4, 0.770 ms against 0.815 with one tile; batch 8, 0.885 with one tile against 0.898 with two and 0.938 with a
# tile and a half; batch 16, 1.199 against 1.221 and 1.252; batch 64, 2.50 against 2.89 and 3.08.
decode_form = "auto"


decode_tiles = "auto"     # tiles of 128 keys that a block of the "one_tile" form walks: "auto" or a number (for comparisons)


def decode_tiles_for(rows: int, key_tiles: int) -> int:
    """How many tiles of 128 keys a block of the fused decode kernel's "one_tile" form walks, for ``rows`` = requests x
    key/value heads (x strips of 16 query heads) and contexts of ``key_tiles`` tiles: the largest power of two (up to 32)
    that still leaves two partitions a request and as many blocks as the device holds at once (four of the tiled
    kernel share an SM).  Measured on batches of 16 to 256 at contexts of 1,100 to 4,100 with 2 and 8 query heads a
    group: the best count was this one in every case (one partition for the whole context was 2 to 4% behind two)."""
    want = 4 * sm_count()
    tiles = 1
    while tiles < 32 and 2 * tiles < key_tiles and rows * -(-key_tiles // (2 * tiles)) >= want:
        tiles *= 2
    if tiles < 4 and key_tiles > 32:
        # Few requests with long contexts: single tiles would make dozens of partitions a head, whose partial results and
        # merge (more than 16 partitions take the merge kernel several trips to memory) cost more than the blocks that
        # four tiles a block leave idle.  Measured at 1 to 8 requests of 8,192 tokens and 1 of 30,000: 18 to 48% faster.
        tiles = 4 if rows * -(-key_tiles // 4) >= 100 else 2
    return tiles


def decode_forms_for(page_size: int) -> list[str]:
    """The forms of the fused decode kernel that take pages of ``page_size`` tokens (for a caller that times them)."""
    return [f for f in DECODE_FORMS if f != "tile_and_half" or (DECODE_PARTITION // 2) % page_size == 0]


def attention_decode_fused(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta, scale, window,
                           q_weight, k_weight, eps, cos_sin, slot_mapping, form: Optional[str] = None,
                           tiles: Optional[int] = None) -> None:
    """Decode attention over requests [0, meta.num_decodes) straight from the q|k|v product's rows: the kernel
    applies the q/k norm and the rotary embedding to q and to the newest key itself and writes that key and the
    newest value into the cache (``slot_mapping``; None if another layer wrote them), so the step needs no
    ``qk_norm_rope_kv_write`` for these rows.  The token's position is its request's context length minus one.
    Other arguments as for that function and ``attention_decode``.  ``form``: one of ``DECODE_FORMS`` (default
    ``decode_form``).  ``tiles``: how many tiles of 128 keys a block of the "one_tile" form walks (default
    ``decode_tiles``; "auto": by how many blocks there would be)."""
    form = form or decode_form
    typical = getattr(meta, "typical_context_len", 0) or meta.max_context_len
    rows = meta.num_decodes * num_kv_heads * ((num_heads // num_kv_heads + 15) // 16)
    key_tiles = (typical + DECODE_PARTITION - 1) // DECODE_PARTITION
    blocks = rows * key_tiles
    tiles = decode_tiles if tiles is None else tiles
    if form == "auto":
        resident = 3 * sm_count()                   # blocks of the two-tile form that the device holds at once
        form = "two_tiles" if blocks <= resident else "one_tile"
        if tiles == "auto" and decode_tiles_for(rows, key_tiles) > 1:
            form = "one_tile"                       # (the form whose blocks can walk several tiles)
    if form != "one_tile":
        tiles = 1
    elif tiles == "auto":
        tiles = decode_tiles_for(rows, key_tiles)
    D = meta.num_decodes
    part_keys = DECODE_PARTITION * tiles
    parts = max(1, (meta.max_context_len + part_keys - 1) // part_keys)
    room = max(parts, (getattr(meta, "scratch_context_len", 0) + part_keys - 1) // part_keys)
    tmp_out = meta.workspace("decode_tmp_out", (D * num_heads * room * head_dim,), torch.float32)
    tmp_ml = meta.workspace("decode_tmp_ml", (2, D * num_heads * room), torch.float32)
    tm = kv_tensor_map(pool, page_size)
    _need(tm is not None and tuple(pool.shape[1:]) == (2, num_kv_heads, page_size, head_dim) and pool.is_contiguous(),
          "attention_decode_fused: cache slot")
    for w in (q_weight, k_weight):
        _need(w is None or (w.dtype == torch.float32 and tuple(w.shape) == (head_dim,)), "attention_decode_fused: norm weights")
    _need(check_rotary(cos_sin, head_dim, None, "half_split") == head_dim, "attention_decode_fused: the rotation covers the whole head")
    _need(slot_mapping is None or slot_mapping.dtype == torch.int32, "attention_decode_fused: slots are int32")
    _call("me_attn_decode_fused", qkv.data_ptr(), qkv.stride(0), out.data_ptr(), out.stride(0), pool.data_ptr(), tm.ptr,
          block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), D,
          num_heads, num_kv_heads, head_dim, page_size, float(scale), int(window or 0), _ptr(q_weight), _ptr(k_weight),
          float(eps), _ptr(cos_sin), _ptr(slot_mapping), tmp_out.data_ptr(), tmp_ml[0].data_ptr(),
          tmp_ml[1].data_ptr(), parts, DECODE_FORMS[form], int(tiles), meta.error_flag.data_ptr(), _stream())
    global launches
    launches += 1          # partition kernel + merge kernel


def paged_attention(qkv: torch.Tensor, out: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
                    pool: torch.Tensor, page_size: int, block_tables: torch.Tensor, meta, scale: float,
                    window: Optional[int], decodes: bool = True) -> None:
    """Attention of one step over the paged cache: requests that bring one token go to the decode
    kernel (unless ``decodes`` is False: the caller has run them), portions of prompts to the chunk kernel;
    both write their rows of ``out`` (the split of layers/attention.py:64-76)."""
    check_attention_sizes(head_dim, num_heads, num_kv_heads)
    _need(qkv.stride(1) == 1 and out.stride(1) == 1 and out.shape[1] == num_heads * head_dim, "paged_attention: shapes")
    _need(pool.dtype == qkv.dtype == out.dtype and pool.is_contiguous(), "paged_attention: dtypes")
    _need(block_tables.dtype == torch.int32 and block_tables.stride(1) == 1, "paged_attention: block tables")
    if decodes and meta.num_decodes > 0:
        attention_decode(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta, scale, window)
    if meta.num_tiles > 0:
        fn = attention_chunks
        if qkv.dtype == torch.bfloat16:
            if (use_tcgen05_attention and meta.error_flag is not None and qkv.is_contiguous()
                    and prefill_tcgen05_heads_per_block(num_heads, num_kv_heads, head_dim, page_size) > 0):
                fn = attention_prefill_tcgen05
            elif prefill_heads_per_block(num_heads, num_kv_heads, head_dim) > 0:
                fn = attention_prefill
        fn(qkv, out, num_heads, num_kv_heads, head_dim, pool, page_size, block_tables, meta, scale, window)


# ---- sampling -------------------------------------------------------------------------------
def sample(logits: torch.Tensor, temperatures: torch.Tensor, seeds: torch.Tensor, positions: torch.Tensor,
           out: torch.Tensor, workspace=None) -> None:
    """Greedy (temperature 0) or exponential-race draw per row; two passes over pieces of the vocabulary."""
    global launches
    S, V = logits.shape
    _need(logits.dtype == torch.float32 and logits.stride(1) == 1, "sample: logits must be float32 rows")
    _need(temperatures.dtype == torch.float32 and seeds.dtype == torch.int32 and positions.dtype == torch.int32
          and out.dtype == torch.int32, "sample: dtypes")
    _need(temperatures.shape[0] == S and seeds.shape[0] == S and positions.shape[0] == S and out.shape[0] == S, "sample: sizes")
    chunks = (_lib or require_extension()).me_sample_chunks(V)
    if workspace is None:
        part = torch.empty(2, S * chunks, dtype=torch.float32, device=logits.device)
    else:
        part = workspace("sample_partials", (2, S * chunks), torch.float32)
    _call("me_sample", logits.data_ptr(), logits.stride(0), temperatures.data_ptr(), seeds.data_ptr(),
          positions.data_ptr(), out.data_ptr(), S, V, part[0].data_ptr(), part[1].data_ptr(), _stream())
    launches += 1


# ---- several residual streams, layer norm, short convolutions, PolyNorm ----------------------------
def hc_norm(streams: torch.Tensor, *, update=None, mix_in: Optional[torch.Tensor] = None,
            norm_weight: Optional[torch.Tensor] = None, eps: float = 0.0, out: Optional[torch.Tensor] = None,
            rows: Optional[torch.Tensor] = None, conv=None) -> None:
    """One pass over the residual streams ``streams`` [S, T, W] (float32): apply the pending ``update`` = (y [T, W],
    mix [S, S] indexed [from, to], out weights [S]): x_r <- sum_s mix[s, r] x_s + out[r] y; then, with ``norm_weight``,
    write the layer norm of u = sum_s mix_in[s] x_s (every stream once without ``mix_in``) to ``out``.  With ``rows``
    only those tokens are read and the streams stay as they are.  ``conv`` = (weight [W, taps], state [slots, taps-1, W] or
    None, state slots, context lengths), for steps in which every request brings one token (token t is request t): the
    output is then h + conv(h) as ``short_conv`` computes it, and the state moves on, in the same kernel."""
    _need(streams.dim() == 3 and streams.dtype == torch.float32 and streams.is_contiguous(), "hc_norm: streams must be float32 [S, T, W]")
    S, T, W = streams.shape
    y = mix = outw = None
    if update is not None:
        y, mix, outw = update
        _need(tuple(y.shape) == (T, W) and y.is_contiguous(), "hc_norm: the update's y must be [T, W]")
        _need(mix.dtype == torch.float32 and tuple(mix.shape) == (S, S) and mix.is_contiguous()
              and outw.dtype == torch.float32 and outw.numel() == S, "hc_norm: mix must be float32 [S, S], out weights [S]")
    _need(mix_in is None or (mix_in.dtype == torch.float32 and mix_in.numel() == S), "hc_norm: in weights must be float32 [S]")
    n = T if rows is None else rows.shape[0]
    if norm_weight is not None:
        _need(norm_weight.dtype == torch.float32 and norm_weight.numel() == W, "hc_norm: norm weight must be float32 [W]")
        _need(out is not None and out.is_contiguous() and tuple(out.shape) == (n, W), "hc_norm: output shape")
    _need(rows is None or rows.dtype == torch.int32, "hc_norm: rows must be int32")
    cw = cs = slots = lens = None
    taps = 0
    if conv is not None:
        cw, cs, slots, lens = conv
        taps = cw.shape[1]
        _need(rows is None and norm_weight is not None and cw.dtype == torch.float32 and cw.is_contiguous() and cw.shape[0] == W
              and slots.numel() == T and lens.numel() == T, "hc_norm: the convolution needs a request per token")
        _need(taps == 1 or (cs is not None and cs.dtype == torch.float32 and cs.is_contiguous()
                            and tuple(cs.shape[1:]) == (taps - 1, W)), "hc_norm: the convolution's state")
    _call("me_hc_norm", streams.data_ptr(), T * W, S, _ptr(y), _dt(y) if y is not None else 0, _ptr(mix), _ptr(outw), _ptr(mix_in),
          _ptr(norm_weight), float(eps), _ptr(out), _dt(out) if out is not None else 0, _ptr(rows), n, W, _ptr(cw),
          _ptr(cs) if taps > 1 else 0, _ptr(slots), _ptr(lens), taps, _stream())


def short_conv(h: torch.Tensor, weight: torch.Tensor, state: Optional[torch.Tensor], token_req: torch.Tensor, meta,
               state_slots: torch.Tensor, out: torch.Tensor, add_input: bool = True) -> None:
    """``out_t = [h_t +] sum_j weight[:, j] h_(t - taps + 1 + j)`` per channel over each request's tokens, zeros before
    its first token; inputs from before this step come from ``state`` [slots, taps - 1, W], which then takes the
    step's last inputs.  ``h`` [T, W], ``weight`` [W, taps] and ``state`` are float32."""
    T, W = h.shape
    taps = weight.shape[1]
    _need(h.dtype == torch.float32 and h.is_contiguous() and weight.dtype == torch.float32 and weight.is_contiguous()
          and weight.shape[0] == W, "short_conv: h [T, W] and weight [W, taps] must be float32")
    _need(taps == 1 or (state is not None and state.dtype == torch.float32 and state.is_contiguous()
                        and tuple(state.shape[1:]) == (taps - 1, W)), "short_conv: state must be float32 [slots, taps - 1, W]")
    _need(out.is_contiguous() and tuple(out.shape) == (T, W), "short_conv: output shape")
    _call("me_short_conv", h.data_ptr(), weight.data_ptr(), _ptr(state) if taps > 1 else 0, token_req.data_ptr(),
          meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), state_slots.data_ptr(), out.data_ptr(), _dt(out), T,
          meta.num_reqs, W, taps, 1 if add_input else 0, 1, _stream())


def polynorm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """``out = a N(z) + b N(z^2) + c N(z^3) + e`` row by row, N(v) = v / sqrt(mean(v^2) + eps); ``coef`` = (a, b, c, e)."""
    _need(z.dim() == 2 and z.stride(1) == 1 and out.stride(1) == 1 and out.shape == z.shape, "polynorm: shapes")
    _need(coef.dtype == torch.float32 and coef.numel() == 4, "polynorm: four float32 coefficients")
    _call("me_polynorm", z.data_ptr(), _dt(z), z.stride(0), coef.data_ptr(), float(eps), out.data_ptr(), _dt(out),
          out.stride(0), z.shape[0], z.shape[1], _stream())


# ---- the matrix-memory recurrence ------------------------------------------------------------------
mlstm_chunks = True       # portions of prompts by chunks of tokens (False: token by token, always); a switch for comparisons


def mlstm_scan(proj: torch.Tensor, offsets: dict, bias_i: torch.Tensor, bias_f: torch.Tensor, gate_cap: float,
               S: torch.Tensor, n: torch.Tensor, m: torch.Tensor, meta, state_slots: torch.Tensor, o: torch.Tensor,
               num_heads: int, dim: int, vdim: int, q_scale: float) -> None:
    """Walks every request's tokens of this step through the recurrence from the state in its slot (see csrc/mlstm.cu).
    ``proj`` [T, N] float32 holds q, k, v, i, f at the column ``offsets``; ``o`` [T, heads * vdim] float32.  A step in
    which some request brings several tokens runs the kernel that takes a chunk of 64 tokens at a time (``mlstm_chunks``)."""
    T = proj.shape[0]
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1, "mlstm_scan: projections must be float32 rows")
    _need(all(t.dtype == torch.float32 and t.is_contiguous() for t in (S, n, m, o, bias_i, bias_f)), "mlstm_scan: float32 state")
    _need(tuple(S.shape[1:]) == (num_heads, dim, vdim) and tuple(n.shape[1:]) == (num_heads, dim) and m.shape[1] == num_heads,
          "mlstm_scan: state shapes")
    _need(tuple(o.shape) == (T, num_heads * vdim), "mlstm_scan: output shape")
    _call("me_mlstm_scan", proj.data_ptr(), proj.stride(0), offsets["q"], offsets["k"], offsets["v"], offsets["i"], offsets["f"],
          bias_i.data_ptr(), bias_f.data_ptr(), float(gate_cap), S.data_ptr(), n.data_ptr(), m.data_ptr(),
          meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), state_slots.data_ptr(), o.data_ptr(), meta.num_reqs,
          num_heads, dim, vdim, float(q_scale), 1 if (mlstm_chunks and T > meta.num_reqs) else 0, _stream())


def mlstm_out(o: torch.Tensor, proj: torch.Tensor, off_g: int, weight: torch.Tensor, eps: float, out: torch.Tensor,
              num_heads: int, vdim: int, shared_weight: bool = False, gate: Optional[str] = "sigmoid") -> None:
    """Each head's ``o`` divided by its root mean square, times ``weight`` and the sigmoid of the gate columns of ``proj``.
    ``shared_weight``: the weight has ``vdim`` values that every head uses; ``gate`` "silu": g sigmoid(g) instead of sigmoid(g), None: no gate.
    ``out`` may be columns of a wider tensor."""
    T = o.shape[0]
    _need(gate in (None, "sigmoid", "silu"), "mlstm_out: the gate is 'sigmoid', 'silu' or None")
    _need(weight.dtype == torch.float32 and weight.numel() == (vdim if shared_weight else num_heads * vdim),
          "mlstm_out: weight must be float32 [heads * vdim] ([vdim] when the heads share it)")
    _need(out.stride(1) == 1 and tuple(out.shape) == (T, num_heads * vdim), "mlstm_out: output shape")
    _call("me_mlstm_out", o.data_ptr(), proj.data_ptr(), proj.stride(0), off_g, weight.data_ptr(), float(eps), out.data_ptr(),
          _dt(out), out.stride(0), T, num_heads, vdim, 1 if shared_weight else 0, {"sigmoid": 0, "silu": 1, None: 2}[gate], _stream())


# ---- gated linear attention --------------------------------------------------------------------------
def gla_decay(proj: torch.Tensor, off_a1: int, rank: int, w2: torch.Tensor, bias: torch.Tensor, tau: float, la: torch.Tensor) -> None:
    """``la`` [T, C] float32 = logsigmoid(w2 a1 + bias) / tau, with a1 the ``rank`` columns of ``proj`` from ``off_a1`` on: the
    logarithm of a decay sigmoid(z)^(1/tau) per key channel (see csrc/gla.cu)."""
    T, C = la.shape
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1 and proj.shape[0] == T and off_a1 + rank <= proj.shape[1],
          "gla_decay: projections must be float32 rows that hold the low-rank vector")
    _need(w2.is_contiguous() and tuple(w2.shape) == (C, rank) and bias.dtype == torch.float32 and bias.numel() == C
          and la.dtype == torch.float32 and la.is_contiguous(), "gla_decay: w2 [C, rank], float32 bias [C], float32 la [T, C]")
    _call("me_gla_decay", proj.data_ptr(), proj.stride(0), off_a1, rank, w2.data_ptr(), _dt(w2), bias.data_ptr(), float(tau),
          la.data_ptr(), T, C, _stream())


gla_chunks = True     # portions of prompts run the recurrence a chunk of tokens at a time; a switch for comparisons


GLA_CHUNK = 64        # tokens that the chunk kernels of csrc/gla.cu take at a time (a tile list of this size must exist)


def gla_scan(proj: torch.Tensor, offsets: dict, la: torch.Tensor, S: torch.Tensor, meta, state_slots: torch.Tensor, o: torch.Tensor,
             num_heads: int, dim: int, vdim: int, q_scale: float, scores: Optional[torch.Tensor] = None,
             chunk_states: Optional[torch.Tensor] = None, gate: Optional[tuple] = None) -> None:
    """Walks every request's tokens of this step through S_t = diag(exp(la_t)) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t from the
    state in its slot (see csrc/gla.cu).  ``proj`` [T, N] float32 holds q, k, v at the column ``offsets``; ``la`` [T, heads * dim]
    and ``o`` [T, heads * vdim] float32.  With the float32 workspaces ``scores`` ([T, heads, GLA_CHUNK]) and ``chunk_states``
    (heads * dim * vdim values for every run of GLA_CHUNK tokens: ``gla_chunk_count``) the requests that bring several tokens
    take GLA_CHUNK tokens at a time, all runs of the step side by side (``gla_chunks``); ``la`` is overwritten on the way.

    ``gate`` = (bias, lower), float32 [heads * dim] each: the recurrence with one gate a channel for keeping and writing (HGRN2).  The columns
    ``offsets["k"]`` then hold the gate's pre-activations z, and a = lower + (1 - lower) sigmoid(z + bias), k = 1 - a, q <- silu(q);
    ``la`` is a work buffer, and the q and k columns of ``proj`` are written on the way."""
    T = proj.shape[0]
    _need(gate is None or all(g.dtype == torch.float32 and g.is_contiguous() and g.numel() == num_heads * dim for g in gate),
          "gla_scan: a gate's bias and lower bound are float32 [heads * dim]")
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1, "gla_scan: projections must be float32 rows")
    _need(all(t.dtype == torch.float32 and t.is_contiguous() for t in (S, la, o)), "gla_scan: float32 state, decays and output")
    _need(tuple(S.shape[1:]) == (num_heads, dim, vdim) and tuple(la.shape) == (T, num_heads * dim)
          and tuple(o.shape) == (T, num_heads * vdim), "gla_scan: shapes")
    tiles, n_tiles = meta.tile_lists[GLA_CHUNK]
    chunked = gla_chunks and scores is not None and chunk_states is not None and n_tiles > 0
    if chunked:
        _need(scores.dtype == torch.float32 and scores.is_contiguous() and scores.numel() >= T * num_heads * GLA_CHUNK,
              "gla_scan: the workspace of scores is float32 [T, heads, GLA_CHUNK]")
        _need(chunk_states.dtype == torch.float32 and chunk_states.is_contiguous()
              and chunk_states.numel() >= n_tiles * num_heads * dim * vdim,
              "gla_scan: the workspace of states is float32 [runs of GLA_CHUNK tokens, heads, dim, vdim]")
    _call("me_gla_scan", proj.data_ptr(), proj.stride(0), offsets["q"], offsets["k"], offsets["v"], la.data_ptr(), S.data_ptr(),
          meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), state_slots.data_ptr(), o.data_ptr(), meta.num_reqs,
          num_heads, dim, vdim, float(q_scale), tiles.data_ptr() if chunked else 0, n_tiles if chunked else 0, meta.num_decodes,
          scores.data_ptr() if chunked else 0, chunk_states.data_ptr() if chunked else 0, _ptr(gate[0]) if gate else 0,
          _ptr(gate[1]) if gate else 0, _stream())


def gla_chunk_count(meta) -> int:
    """An upper bound of the runs of GLA_CHUNK tokens that the step's requests with several tokens are cut into (a bound that
    depends on the step's shape only, so that a recorded step keeps its workspace)."""
    multi = meta.num_reqs - meta.num_decodes
    return 0 if multi <= 0 else (meta.num_tokens - meta.num_decodes) // GLA_CHUNK + multi


# ---- attention through a latent --------------------------------------------------------------------
LATENT_TILE_Q = 16        # query tokens per block of csrc/latent_attention.cu
use_latent_mma = True     # bfloat16 latent attention on the tensor cores (csrc/latent_attention_mma.cu); a switch for comparisons


def latent_decode_plan(num_requests: int, num_heads: int, kv_rank: int, max_context: int) -> tuple[int, int]:
    """Into how many ranges of keys a single-token request is cut, and how long they are (a multiple of 64): enough blocks
    to give every multiprocessor two, no range shorter than 64 keys.  A block serves 64 heads and 128 latent columns."""
    blocks_per_range = num_requests * ((num_heads + 63) // 64) * ((kv_rank + 127) // 128)
    tiles = max(1, (max_context + 63) // 64)
    want = max(1, min(tiles, (2 * sm_count() + blocks_per_range - 1) // blocks_per_range))
    keys = (tiles + want - 1) // want * 64
    return (tiles * 64 + keys - 1) // keys, keys


def latent_prep(proj: torch.Tensor, offsets: dict, c_weight: torch.Tensor, eps: float, inv_freq: torch.Tensor, rot_dims: int,
                positions: torch.Tensor, slot_mapping: Optional[torch.Tensor], pool: torch.Tensor, q_plain: torch.Tensor,
                q_rot: torch.Tensor, gate: Optional[torch.Tensor], num_heads: int, dim: int, rot_dim: int, kv_rank: int) -> None:
    """From the packed float32 projections: the normed latent and the rotated shared key part into the cache rows named by
    ``slot_mapping``, the heads' plain and rotated query parts, the sigmoid of the gates (see csrc/latent_attention.cu)."""
    T = proj.shape[0]
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1, "latent_prep: projections must be float32 rows")
    _need(inv_freq.dtype == torch.float64 and inv_freq.numel() * 2 == rot_dims, "latent_prep: inv_freq must be float64 [rot_dims / 2]")
    _need(pool.is_contiguous() and pool.shape[-1] == kv_rank + rot_dim and pool.dtype == q_plain.dtype == q_rot.dtype,
          "latent_prep: cache rows must hold kv_rank + rot_dim values of the activations' dtype")
    _need(c_weight.dtype == torch.float32 and c_weight.numel() == kv_rank, "latent_prep: latent weight must be float32 [kv_rank]")
    _call("me_latent_prep", proj.data_ptr(), proj.stride(0), offsets["q"], offsets["c"], offsets.get("g", 0), c_weight.data_ptr(),
          float(eps), inv_freq.data_ptr(), rot_dims, positions.data_ptr(), _ptr(slot_mapping), pool.data_ptr(), q_plain.data_ptr(),
          q_rot.data_ptr(), _ptr(gate), _dt(pool), T, num_heads, dim, rot_dim, kv_rank, _stream())


def latent_attention(q_abs: torch.Tensor, q_rot: torch.Tensor, pool: torch.Tensor, page_size: int, block_tables: torch.Tensor,
                     meta, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], out: torch.Tensor, scale: float,
                     window: Optional[int] = None) -> None:
    """Causal multi-query attention over cache rows [c | rotated key part]: ``q_abs`` [H, T, C] against c, ``q_rot``
    [T, H, R] against the rest; ``out`` [H, T, C] = softmax-weighted sum of c (with ``sink`` [H] in the denominator),
    times ``gate`` [T, H].  ``window``: a query at position p sees the keys p - window < j <= p only."""
    H, T, C = q_abs.shape
    window = int(window or 0)
    R = q_rot.shape[2]
    _need(q_abs.is_contiguous() and q_rot.is_contiguous() and out.is_contiguous() and out.shape == q_abs.shape, "latent_attention: shapes")
    _need(pool.shape[-1] == C + R and pool.dtype == q_abs.dtype, "latent_attention: cache rows")
    lib = _lib or require_extension()
    if q_abs.dtype == torch.bfloat16 and use_latent_mma and lib.me_latent_attention_mma_takes(C, R):
        # the tensor-core kernels of csrc/latent_attention_mma.cu
        gp = lib.me_latent_attention_mma_heads_per_block(H)
        tiles, n_tiles = meta.tile_lists[64 // gp]
        common = (q_abs.data_ptr(), q_rot.data_ptr(), pool.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
                  meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr())
        if n_tiles:
            _call("me_latent_attention_mma", *common, tiles.data_ptr(), n_tiles, _ptr(sink), _ptr(gate), out.data_ptr(), T, H, C, R,
                  page_size, float(scale), window, _stream())
        D = meta.num_decodes
        if D:
            # (with a window a request's ranges start at the tile its window reaches first)
            splits, keys = latent_decode_plan(D, H, C, min(meta.max_context_len, window + 63) if window else meta.max_context_len)
            partial = meta.workspace("latent_partials", (D, splits, H, C + 2), torch.float32)
            _call("me_latent_attention_decode", *common, D, _ptr(sink), _ptr(gate), out.data_ptr(), partial.data_ptr(), splits, keys,
                  T, H, C, R, page_size, float(scale), window, _stream())
        return
    tiles, n_tiles = meta.tile_lists[LATENT_TILE_Q]
    _call("me_latent_attention", q_abs.data_ptr(), q_rot.data_ptr(), _dt(q_abs), pool.data_ptr(), block_tables.data_ptr(),
          block_tables.stride(0), meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), tiles.data_ptr(), n_tiles,
          meta.num_decodes, _ptr(sink), _ptr(gate), out.data_ptr(), T, H, C, R, page_size, float(scale), window, _stream())


def heads_to_rows(x: torch.Tensor, out: torch.Tensor) -> None:
    """[H, T, V] -> [T, H * V]."""
    H, T, V = x.shape
    _need(x.is_contiguous() and out.is_contiguous() and tuple(out.shape) == (T, H * V) and out.dtype == x.dtype, "heads_to_rows: shapes")
    _call("me_heads_to_rows", x.data_ptr(), out.data_ptr(), _dt(x), T, H, V, _stream())


def batched_heads_mm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """``out[h] = x[h] @ w[h]`` for every head: [H, T, K] x [H, K, N] -> [H, T, N], through the library's batched product
    (either operand may be a strided view).  float32 operands are multiplied in true 32-bit."""
    global library_calls
    _need(x.dim() == 3 and w.dim() == 3 and x.shape[0] == w.shape[0] and x.shape[2] == w.shape[1], "batched_heads_mm: shapes")
    _need(x.dtype == w.dtype == out.dtype, "batched_heads_mm: one dtype")
    if x.dtype == torch.float32 and torch.backends.cuda.matmul.allow_tf32:
        raise KernelError("batched_heads_mm: TF32 is switched on for float32 products; the float32 engine needs it off")
    with _Timed("library_bmm"):
        torch.bmm(x, w, out=out)
    library_calls += 1


# ---- a norm behind the sub-layer, in groups; pooled blocks of keys and values -------------------------------------------------
def group_norm(residual: torch.Tensor, y: Optional[torch.Tensor], weight: torch.Tensor, groups: int, eps: float,
               out: Optional[torch.Tensor], rows: Optional[torch.Tensor] = None) -> None:
    """RMS norm in ``groups`` equal consecutive parts of a row, each divided by its own sqrt(mean(part^2) + eps), times ``weight``.
    With ``y``: ``residual += norm(y)``; without: ``residual <- norm(residual)``; ``out`` (optional) receives the new rows of the
    float32 stream in its own dtype.  With ``rows``: ``out[i] = norm(residual[rows[i]])`` and the stream is left alone."""
    T, W = residual.shape
    n = T if rows is None else rows.shape[0]
    _need(residual.dtype == torch.float32 and residual.is_contiguous() and weight.dtype == torch.float32 and weight.numel() == W,
          "group_norm: a float32 stream [T, W] and a float32 weight [W]")
    _need(groups >= 1 and W % groups == 0, f"group_norm: {W} values do not split into {groups} groups")
    _need(y is None or (rows is None and y.shape[0] == T and y.shape[1] >= W and y.stride(1) == 1), "group_norm: the output's rows")
    _need(out is None or (out.is_contiguous() and tuple(out.shape) == (n, W)), "group_norm: the copy's shape")
    _need(rows is None or (rows.dtype == torch.int32 and out is not None), "group_norm: int32 rows and a place for them")
    _call("me_group_norm", residual.data_ptr(), _ptr(y), _dt(y) if y is not None else 0, y.stride(0) if y is not None else 0,
          weight.data_ptr(), int(groups), float(eps), _ptr(out), _dt(out) if out is not None else 0, _ptr(rows), n, W, _stream())


POOL_BY_BLOCK_MAX_REQUESTS = 64    # steps with prompts of up to this many requests: a block of threads per completed block of tokens


def pool_kv(pool: torch.Tensor, block_tables: torch.Tensor, pooled: torch.Tensor, pooled_tables: torch.Tensor, positions: torch.Tensor,
            token_req: torch.Tensor, block: int, dim: int, vdim: int, page_size: int, meta=None) -> None:
    """Behind a step's cache write: for every token of the step whose position ends a block of ``block`` tokens, the mean of the
    block's keys and the mean of its values (as ``pool`` holds them) go to row position // block of ``pooled``, a cache of the
    same layout with block tables of its own (see csrc/pooled_kv.cu).  ``meta`` (the step's shape): a step that brings portions
    of prompts for a few requests launches a block of threads for every block of tokens it can complete instead of one a token."""
    T = positions.numel()
    by_block = (meta is not None and meta.num_decodes < meta.num_reqs and meta.num_reqs <= POOL_BY_BLOCK_MAX_REQUESTS
                and meta.num_tokens == T)
    _need(pool.dim() == 5 and pool.shape[1] == 2 and pool.is_contiguous() and pooled.is_contiguous() and pooled.dtype == pool.dtype
          and pooled.shape[1:] == pool.shape[1:], "pool_kv: both caches are [pages, 2, kv heads, page, row] of one dtype")
    _need(block_tables.dtype == pooled_tables.dtype == torch.int32 and block_tables.stride(1) == 1 and pooled_tables.stride(1) == 1,
          "pool_kv: block tables")
    _need(token_req.numel() == T and block >= 1, "pool_kv: a request for every token and a block size")
    _call("me_pool_kv", pool.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), pooled.data_ptr(), pooled_tables.data_ptr(),
          pooled_tables.stride(0), positions.data_ptr(), token_req.data_ptr(), meta.cu_seqlens.data_ptr() if by_block else 0,
          meta.context_lens.data_ptr() if by_block else 0, meta.num_reqs if by_block else 0, 1 if by_block else 0, _dt(pool), T, int(block),
          pool.shape[2], dim, vdim, pool.shape[-1], page_size, _stream())


# ---- norms on both sides of a sub-layer, convolved and gated attention with a sink, routed feed-forwards ----------------
def sandwich_norm(residual: torch.Tensor, y: Optional[torch.Tensor], post_weight: Optional[torch.Tensor], mult: float,
                  pre_weight: Optional[torch.Tensor], eps: float, out: Optional[torch.Tensor],
                  rows: Optional[torch.Tensor] = None, norm_out: bool = True) -> None:
    """``residual += mult * y / rms(y) * post_weight`` (float32, in place; skipped without ``y``), then
    ``out = residual / rms(residual) * pre_weight`` (``norm_out`` False: ``out`` is the new residual itself, in ``out``'s
    dtype).  With ``rows`` only those rows are computed and ``residual`` is not written."""
    T, W = residual.shape
    _need(residual.dtype == torch.float32 and residual.is_contiguous(), "sandwich_norm: the residual must be float32 [T, W]")
    _need(y is None or (tuple(y.shape) == (T, W) and y.is_contiguous() and post_weight is not None), "sandwich_norm: y must be [T, W]")
    for w in (post_weight, pre_weight):
        _need(w is None or (w.dtype == torch.float32 and w.numel() == W and w.is_contiguous()), "sandwich_norm: weights are float32 [W]")
    n = T if rows is None else rows.shape[0]
    _need(out is None or (out.is_contiguous() and tuple(out.shape) == (n, W)), "sandwich_norm: output shape")
    _need(rows is None or (rows.dtype == torch.int32 and rows.is_contiguous()), "sandwich_norm: rows must be int32")
    _call("me_sandwich_norm", residual.data_ptr(), _ptr(y), _dt(y) if y is not None else 0, _ptr(post_weight), float(mult),
          _ptr(pre_weight), float(eps), _ptr(out), _dt(out) if out is not None else 0, _ptr(rows), n, W, 1 if norm_out else 0,
          _stream())


def parallel_norm(residual: torch.Tensor, adds: Sequence[torch.Tensor], vectors: Sequence[torch.Tensor], eps: float,
                  norm1: tuple, out1: torch.Tensor, norm2: Optional[tuple] = None, out2: Optional[torch.Tensor] = None,
                  rows: Optional[torch.Tensor] = None, embedding: Optional[tuple] = None) -> None:
    """``residual += sum(adds) + sum(vectors)`` (float32, in place; up to two [T, W] tensors of one dtype and two float32 [W]
    vectors), then one or two layer norms of the new rows: ``out = (x - mean) / sqrt(var + eps) * weight + bias`` with
    ``norm`` = (weight, bias or None).  With ``rows`` only those rows are computed and ``residual`` is not written.
    ``embedding`` = (token ids, table, feedback or None, scale): the tokens' rows of the table times the scale join the sum (ids as
    ``embed`` takes them)."""
    T, W = residual.shape
    adds, vectors = [a for a in adds if a is not None], [v for v in vectors if v is not None]
    _need(residual.dtype == torch.float32 and residual.is_contiguous(), "parallel_norm: the residual must be float32 [T, W]")
    _need(len(adds) <= 2 and len(vectors) <= 2, "parallel_norm: at most two outputs and two vectors can be added")
    _need(all(tuple(a.shape) == (T, W) and a.is_contiguous() and a.dtype == adds[0].dtype for a in adds), "parallel_norm: outputs must be [T, W]")
    _need(all(v.dtype == torch.float32 and v.numel() == W and v.is_contiguous() for v in vectors), "parallel_norm: vectors are float32 [W]")
    n = T if rows is None else rows.shape[0]
    for nm, out in ((norm1, out1), (norm2, out2)):
        if out is None:
            continue
        _need(nm is not None and nm[0].dtype == torch.float32 and nm[0].numel() == W and nm[0].is_contiguous()
              and (nm[1] is None or (nm[1].dtype == torch.float32 and nm[1].numel() == W and nm[1].is_contiguous())),
              "parallel_norm: weights and biases are float32 [W]")
        _need(out.is_contiguous() and tuple(out.shape) == (n, W) and out.dtype == out1.dtype, "parallel_norm: output shape")
    _need(rows is None or (rows.dtype == torch.int32 and rows.is_contiguous()), "parallel_norm: rows must be int32")
    ids, table, feedback, scale = embedding if embedding is not None else (None, None, None, 1.0)
    if embedding is not None:
        _need(rows is None and ids.dtype == torch.int32 and ids.is_contiguous() and ids.numel() == T and table.is_contiguous()
              and table.dim() == 2 and table.shape[1] == W, "parallel_norm: the embedding needs an int32 id a row and a table [vocabulary, W]")
    adds += [None] * (2 - len(adds))
    vectors += [None] * (2 - len(vectors))
    _call("me_parallel_norm", residual.data_ptr(), _ptr(adds[0]), _ptr(adds[1]), _dt(adds[0]) if adds[0] is not None else 0,
          _ptr(vectors[0]), _ptr(vectors[1]), norm1[0].data_ptr(), _ptr(norm1[1]), out1.data_ptr(),
          _ptr(norm2[0]) if out2 is not None else 0, _ptr(norm2[1]) if out2 is not None else 0, _ptr(out2), _dt(out1), _ptr(rows), n, W,
          float(eps), _ptr(ids), _ptr(table), _dt(table) if table is not None else 0, table.shape[0] if table is not None else 0, _ptr(feedback),
          feedback.numel() if feedback is not None else 0, float(scale), _stream())


# ---- the stream with everything pending, and its RMS norm -----------------------------------------------
def stream_norm(residual: torch.Tensor, terms: Sequence[tuple], vectors: Sequence[torch.Tensor], weight: Optional[torch.Tensor], eps: float,
                out: torch.Tensor, rows: Optional[torch.Tensor] = None) -> None:
    """``residual += sum of terms + sum of vectors`` (float32, in place), then ``out = residual / rms(residual) * weight``, or without a weight
    a copy of the stream (``out`` may be columns of wider rows).  A term is (y [T, W], scale, eps_y): scale * y with a float32 [W]
    scale or None, or, with eps_y not None, scale * y / sqrt(mean(y^2) + eps_y).  Up to three terms of one dtype and two float32 [W]
    vectors.  With ``rows`` only those rows are computed and ``residual`` is not written."""
    T, W = residual.shape
    terms, vectors = list(terms), list(vectors)
    _need(residual.dtype == torch.float32 and residual.is_contiguous(), "stream_norm: the residual must be float32 [T, W]")
    _need(len(terms) <= 3 and len(vectors) <= 2, "stream_norm: at most three outputs and two vectors can be added")
    _need(all(tuple(y.shape) == (T, W) and y.is_contiguous() and y.dtype == terms[0][0].dtype for y, _, _ in terms), "stream_norm: outputs must be [T, W]")
    floats = [s for _, s, _ in terms if s is not None] + vectors + ([weight] if weight is not None else [])
    _need(all(v.dtype == torch.float32 and v.numel() == W and v.is_contiguous() for v in floats), "stream_norm: scales, vectors and the weight are float32 [W]")
    n = T if rows is None else rows.shape[0]
    _need(tuple(out.shape) == (n, W) and out.stride(1) == 1, "stream_norm: output shape")
    _need(rows is None or (rows.dtype == torch.int32 and rows.is_contiguous()), "stream_norm: rows must be int32")
    terms += [(None, None, None)] * (3 - len(terms))
    vectors += [None] * (2 - len(vectors))
    _call("me_stream_norm", residual.data_ptr(), *(_ptr(y) for y, _, _ in terms), _dt(terms[0][0]) if terms[0][0] is not None else 0,
          *(_ptr(s) for _, s, _ in terms), *(-1.0 if e is None else float(e) for _, _, e in terms), _ptr(vectors[0]), _ptr(vectors[1]), _ptr(weight),
          float(eps), out.data_ptr(), _dt(out), out.stride(0), _ptr(rows), n, W, _stream())


# ---- recurrences whose state decays by one number a head ----------------------------------------------------
CONV_TILE = 16            # tokens per block of the convolution (csrc/short_conv.cu)


def conv_silu(u: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], state: Optional[torch.Tensor], meta, state_slots: torch.Tensor,
              out: torch.Tensor) -> None:
    """``out_t = silu(bias + sum_j weight[:, j] u_(t - taps + 1 + j))`` per channel over each request's tokens, zeros before its first
    token; inputs from before this step come from ``state`` [slots, taps - 1, C], which then takes the step's last inputs.  ``u`` float32
    [T, C], possibly columns of wider rows; ``weight`` [C, taps], ``bias`` [C] and ``state`` float32; ``out`` [T, C] of any dtype."""
    T, C = u.shape
    taps = weight.shape[1]
    _need(u.dtype == torch.float32 and u.stride(1) == 1 and weight.dtype == torch.float32 and weight.is_contiguous() and weight.shape[0] == C,
          "conv_silu: u [T, C] and weight [C, taps] must be float32")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == C and bias.is_contiguous()), "conv_silu: bias must be float32 [C]")
    _need(taps == 1 or (state is not None and state.dtype == torch.float32 and state.is_contiguous() and tuple(state.shape[1:]) == (taps - 1, C)),
          "conv_silu: state must be float32 [slots, taps - 1, C]")
    _need(out.is_contiguous() and tuple(out.shape) == (T, C), "conv_silu: output shape")
    tiles, n_tiles = meta.tile_lists[CONV_TILE]
    _call("me_conv_silu", u.data_ptr(), u.stride(0), weight.data_ptr(), _ptr(bias), _ptr(state) if taps > 1 else 0, tiles.data_ptr(), n_tiles,
          meta.num_decodes, meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), state_slots.data_ptr(), out.data_ptr(), _dt(out),
          meta.num_reqs, C, taps, _stream())
    global launches
    launches += 1 if taps > 1 and meta.num_decodes < meta.num_reqs else 0


HEAD_DECAY_CHUNK = 64     # tokens per run of the recurrence's prompt kernels (csrc/head_decay.cu)
HEAD_DECAY_RUN = 3 * HEAD_DECAY_CHUNK   # float32 values that hold a run's decays and factors of one head (64 float64 and 64 float32)
use_head_decay_mma = True # bfloat16 prompts on the tensor cores where the sizes allow (csrc/head_decay_mma.cu); a switch for comparisons
head_decay_chunks = True  # portions of prompts by runs of tokens (False: token by token, always); a switch for comparisons


def head_decay_chunk_count(meta) -> int:
    """An upper bound of the runs of HEAD_DECAY_CHUNK tokens that the step's requests with several tokens are cut into (it depends
    on the step's shape only, so that a recorded step keeps its workspace)."""
    multi = meta.num_reqs - meta.num_decodes
    return 0 if multi <= 0 else (meta.num_tokens - meta.num_decodes) // HEAD_DECAY_CHUNK + multi


def head_decay_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, S: torch.Tensor, meta, state_slots: torch.Tensor, o: torch.Tensor,
                    num_heads: int, num_groups: int, dim: int, vdim: int, *, k_scale: float = 1.0, dt: Optional[tuple] = None,
                    decay: Optional[tuple] = None, skip: Optional[torch.Tensor] = None, chunk_states: Optional[torch.Tensor] = None,
                    run_numbers: Optional[torch.Tensor] = None) -> None:
    """Walks every request's tokens of this step through S_t = a_t S_(t-1) + g_t k_t v_t^T, o_t = S_t^T q_t + skip v_t from the state in
    its slot, per head, with one decay a and one factor g a head and token (see csrc/head_decay.cu).  ``q``, ``k`` [T, groups * dim]
    and ``v`` [T, heads * vdim]: columns of rows of one dtype; head h reads group h // (heads / groups) of q and k.

    ``dt`` = (pre-activations [T, heads] float32 (columns of wider rows), bias [heads], a_log [heads]): g = softplus(dt + bias), a =
    exp(-exp(a_log) g).  Or ``decay`` = (decays float32 [heads], their log2 float64 [heads]): constants, and g = ``k_scale``.  With the float32 workspaces ``chunk_states``
    (heads * dim * vdim values a run of HEAD_DECAY_CHUNK tokens: ``head_decay_chunk_count``) and ``run_numbers`` (heads * HEAD_DECAY_RUN values a run) the
    requests that bring several tokens take a run at a time, all runs of the step side by side."""
    T = o.shape[0]
    _need(num_heads % num_groups == 0, "head_decay_scan: heads must be a multiple of the groups")
    _need(q.dtype == k.dtype == v.dtype and all(t.stride(1) == 1 for t in (q, k, v)), "head_decay_scan: q, k and v are rows of one dtype")
    _need(tuple(q.shape) == tuple(k.shape) == (T, num_groups * dim) and tuple(v.shape) == (T, num_heads * vdim), "head_decay_scan: shapes of q, k, v")
    _need(S.dtype == torch.float32 and S.is_contiguous() and tuple(S.shape[1:]) == (num_heads, dim, vdim), "head_decay_scan: state shape")
    _need(o.dtype == torch.float32 and o.is_contiguous() and tuple(o.shape) == (T, num_heads * vdim), "head_decay_scan: output shape")
    _need((dt is None) != (decay is None), "head_decay_scan: decays from dt or constants")
    per_head = [t for t in ((*dt[1:],) if dt is not None else (decay[0],)) + ((skip,) if skip is not None else ())]
    _need(all(t.dtype == torch.float32 and t.is_contiguous() and t.numel() == num_heads for t in per_head), "head_decay_scan: float32 numbers a head")
    _need(decay is None or (decay[1].dtype == torch.float64 and decay[1].is_contiguous() and decay[1].numel() == num_heads),
          "head_decay_scan: log2 of the decays is float64 [heads]")
    _need(dt is None or (dt[0].dtype == torch.float32 and dt[0].stride(1) == 1 and tuple(dt[0].shape) == (T, num_heads)), "head_decay_scan: dt is float32 [T, heads]")
    tiles, n_tiles = meta.tile_lists[HEAD_DECAY_CHUNK]
    chunked = head_decay_chunks and chunk_states is not None and run_numbers is not None and n_tiles > 0 and dim <= 256
    if chunked:
        _need(all(t.dtype == torch.float32 and t.is_contiguous() for t in (chunk_states, run_numbers))
              and chunk_states.numel() >= n_tiles * num_heads * dim * vdim and run_numbers.numel() >= n_tiles * num_heads * HEAD_DECAY_RUN, "head_decay_scan: workspaces")
    _call("me_head_decay_scan", q.data_ptr(), k.data_ptr(), v.data_ptr(), _dt(q), q.stride(0), k.stride(0), v.stride(0), num_heads, num_groups,
          dim, vdim, float(k_scale), _ptr(dt[0]) if dt else 0, dt[0].stride(0) if dt else 0, _ptr(dt[1]) if dt else 0, _ptr(dt[2]) if dt else 0,
          _ptr(decay[0]) if decay else 0, _ptr(decay[1]) if decay else 0, _ptr(skip), S.data_ptr(), meta.cu_seqlens.data_ptr(), meta.context_lens.data_ptr(), state_slots.data_ptr(),
          o.data_ptr(), meta.num_reqs, meta.num_decodes, tiles.data_ptr() if chunked else 0, n_tiles if chunked else 0,
          chunk_states.data_ptr() if chunked else 0, run_numbers.data_ptr() if chunked else 0, 1 if use_head_decay_mma else 0, _stream())
    global launches
    launches += (2 + (1 if meta.num_decodes else 0)) if chunked else 0


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: Optional[torch.Tensor], groups: int, eps: float, out: torch.Tensor,
                     gate_first: bool) -> None:
    """Rows of ``y`` (float32 [T, W]) normed in ``groups`` equal parts, each by its own root mean square, with the gate silu(``z``) in front of
    the norm (``gate_first``) or behind it, and a float32 [W] weight or None.  All rows may be columns of wider ones."""
    T, W = y.shape
    _need(y.dtype == torch.float32 and y.stride(1) == 1 and tuple(z.shape) == tuple(out.shape) == (T, W) and z.stride(1) == out.stride(1) == 1,
          "gated_group_norm: shapes")
    _need(weight is None or (weight.dtype == torch.float32 and weight.is_contiguous() and weight.numel() == W), "gated_group_norm: weight must be float32 [W]")
    _need(groups >= 1 and W % groups == 0, "gated_group_norm: groups must divide the row")
    _call("me_gated_group_norm", y.data_ptr(), y.stride(0), z.data_ptr(), _dt(z), z.stride(0), _ptr(weight), 1 if gate_first else 0, float(eps),
          out.data_ptr(), _dt(out), out.stride(0), T, W, groups, _stream())


ACTIVATIONS = {"relu_squared": 0, "gelu_tanh": 1, "silu": 2, "gelu": 3}     # "gelu": the exact form, z Phi(z)


def activation(x: torch.Tensor, out: torch.Tensor, kind: str) -> None:
    """``out = act(x)`` over rows; ``kind`` is a key of ``ACTIVATIONS``."""
    _need(kind in ACTIVATIONS, f"activation: {kind!r} is not one of {sorted(ACTIVATIONS)}")
    T, F = x.shape
    _need(tuple(out.shape) == (T, F) and x.stride(1) == 1 and out.stride(1) == 1, "activation: shapes")
    _call("me_activation", x.data_ptr(), _dt(x), x.stride(0), out.data_ptr(), _dt(out), out.stride(0), T, F, ACTIVATIONS[kind], _stream())


def soft_cap(x: torch.Tensor, cap: Optional[float], scale: float = 1.0) -> None:
    """``x <- cap * tanh(scale * x / cap)`` in place (float32); without a cap ``x <- scale * x``."""
    _need(x.dtype == torch.float32 and x.is_contiguous() and (cap is None or cap > 0), "soft_cap: float32 values and a positive cap")
    _call("me_soft_cap", x.data_ptr(), x.numel(), float(cap or 0.0), float(scale), _stream())


def add_row_vector(x: torch.Tensor, v: torch.Tensor) -> None:
    """``x[t] += v`` for every row (in place)."""
    _need(x.dim() == 2 and x.is_contiguous() and v.dtype == torch.float32 and v.is_contiguous() and v.numel() == x.shape[1],
          "add_row_vector: x [T, W] and a float32 vector [W]")
    _call("me_add_row_vector", x.data_ptr(), _dt(x), x.shape[0], x.shape[1], v.data_ptr(), _stream())


def attn_prep(proj: torch.Tensor, bias: Optional[torch.Tensor], q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor],
              norm: Optional[str], eps: float, freq: Optional[torch.Tensor], positions: torch.Tensor,
              slot_mapping: Optional[torch.Tensor], q_out: torch.Tensor, pool: Optional[torch.Tensor], page_size: int,
              num_heads: int, num_kv_heads: int, dim: int, vdim: int, q_scale: Optional[torch.Tensor] = None,
              own_kv: bool = True, maps: int = 1,
              temperature: Optional[tuple[float, float]] = None, v_scale: float = 1.0, magnitude: float = 1.0) -> None:
    """From the packed float32 projections q|k|v (the leading columns of ``proj``; q alone with ``own_kv`` False): bias, a weighted RMS norm of every q and k
    head in front of the rotation (``norm`` "before"), one over the whole q and the whole k of a token ("row", with a weight for every value)
    or a plain one behind it ("after"), the rotation of element i with
    element i + len(freq) by position x ``freq`` (float64 frequencies), queries to ``q_out`` and keys and values into the
    cache rows that ``slot_mapping`` names (see csrc/attn_prep.cu).  ``q_scale`` (float32 [heads]): every query head is
    multiplied by its number at the end.  ``temperature`` = (coef, every): q is multiplied by 1 + coef ln(floor((p + 1) / every) + 1).
    ``v_scale`` multiplies the values, ``magnitude`` the rotation's cosines and sines.  ``maps`` 2: every q and k head has two maps of ``dim`` elements; ``q_out`` then has a row for
    every map of every head.  ``q_out`` [T, rows * width]: rows wider than what they hold are filled with zeros (cache rows too)."""
    T = proj.shape[0]
    C = num_heads * maps * dim + (num_kv_heads * (maps * dim + vdim) if own_kv else 0)
    _need(own_kv or slot_mapping is None, "attn_prep: a mixer without keys and values of its own writes no cache rows")
    _need(q_scale is None or (q_scale.dtype == torch.float32 and q_scale.numel() == num_heads and q_scale.is_contiguous()),
          "attn_prep: q_scale must be float32 [heads]")
    _need(norm in (None, "before", "after", "row"), "attn_prep: norm is None, 'before', 'row' or 'after'")
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1 and proj.shape[1] >= C, "attn_prep: projections must be float32 rows")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == C), "attn_prep: bias must be float32 [channels]")
    if norm in ("before", "row"):
        sizes = (dim, dim) if norm == "before" else (num_heads * maps * dim, num_kv_heads * maps * dim)
        _need(all(w is not None and w.dtype == torch.float32 and w.is_contiguous() and w.numel() == n
                  for w, n in list(zip((q_norm, k_norm), sizes))[:2 if own_kv else 1]),
              "attn_prep: a weighted norm needs float32 weights, [dim] in front of the rotation or one for every value of the row")
    _need(freq is None or (freq.dtype == torch.float64 and freq.is_contiguous() and 2 * freq.numel() <= dim), "attn_prep: freq must be float64 [<= dim / 2]")
    rows = num_heads * maps
    _need(q_out.is_contiguous() and q_out.shape[0] == T and q_out.shape[1] % rows == 0 and q_out.shape[1] // rows >= maps * dim,
          "attn_prep: query output shape")
    _need(slot_mapping is None or (pool is not None and pool.is_contiguous() and pool.dim() == 5 and pool.shape[1] == 2
                                   and pool.shape[-1] >= max(maps * dim, vdim) and pool.dtype == q_out.dtype),
          "attn_prep: the cache must be [pages, 2, kv heads, page, >= max(maps * dim, vdim)] of the activations' dtype")
    _need(temperature is None or temperature[1] > 0, "attn_prep: the temperature's step must be positive")
    rot = 2 * freq.numel() if freq is not None else 0
    coef, every = temperature if temperature is not None else (0.0, 0.0)
    _call("me_attn_prep", proj.data_ptr(), proj.stride(0), _ptr(bias), _ptr(q_norm), _ptr(k_norm), {None: 0, "before": 1, "after": 2, "row": 3}[norm],
          float(eps), _ptr(freq) if rot else 0, rot, positions.data_ptr(), _ptr(slot_mapping), q_out.data_ptr(),
          q_out.shape[1] // rows, _ptr(pool), _dt(q_out), pool.shape[-1] if pool is not None else 0, page_size, num_heads, num_kv_heads, dim, vdim,
          maps, T, _ptr(q_scale), 1 if own_kv else 0, float(coef), float(every), float(v_scale), float(magnitude), _stream())


def padded_head(width: int) -> int:
    """The row width at which heads of ``width`` elements run the tensor-core attention kernels: 64 or 128 (the rest of a row is
    zeros); wider heads keep their width."""
    return 64 if width <= 64 else (128 if width <= 128 else width)


def diff_combine(maps: torch.Tensor, out: torch.Tensor, num_heads: int, vdim: int, lam: float, gain: float, eps: float, first: int = 0) -> None:
    """``maps`` [T, 2 * heads * vdim] holds two results a head; ``out`` [T, heads * vdim] = d / sqrt(mean(d^2) + eps) * gain per head with
    d = first - lam * second, for the rows from ``first`` on."""
    T = maps.shape[0]
    _need(maps.stride(1) == 1 and out.stride(1) == 1 and maps.shape[1] == 2 * num_heads * vdim and tuple(out.shape) == (T, num_heads * vdim),
          "diff_combine: shapes")
    _call("me_diff_combine", maps.data_ptr(), _dt(maps), maps.stride(0), out.data_ptr(), _dt(out), out.stride(0), first, T - first, num_heads, vdim,
          float(lam), float(gain), float(eps), _stream())


def clamped_glu(x: torch.Tensor, out: torch.Tensor, limit: float, alpha: float, shift: float = 1.0) -> None:
    """Rows [gate | up] -> ``g sigmoid(alpha g) (u + shift)`` with g = min(gate, limit), u = clamp(up, -limit, limit)."""
    T, F2 = x.shape
    _need(F2 % 2 == 0 and tuple(out.shape) == (T, F2 // 2) and x.stride(1) == 1 and out.stride(1) == 1, "clamped_glu: shapes")
    _call("me_clamped_glu", x.data_ptr(), _dt(x), x.stride(0), out.data_ptr(), _dt(out), out.stride(0), T, F2 // 2, float(limit),
          float(alpha), float(shift), _stream())


def conv_rope_kv(proj: torch.Tensor, bias: Optional[torch.Tensor], conv_weight: Optional[torch.Tensor],
                 state: Optional[torch.Tensor], inv_freq: torch.Tensor, rot_dims: int, ctx, slot_mapping: Optional[torch.Tensor],
                 q_out: torch.Tensor, pool: Optional[torch.Tensor], page_size: int, num_heads: int, num_kv_heads: int, dim: int,
                 vdim: int, own_kv: bool, angles: Optional[torch.Tensor] = None) -> None:
    """From the packed float32 projections q|k|v (the leading columns of ``proj``): bias, the short causal convolution with
    its state, the rotation of neighbouring pairs, queries to ``q_out`` and keys and values into the cache rows that
    ``slot_mapping`` names (see csrc/conv_rope_kv.cu).  Without ``own_kv`` only the queries exist."""
    T = proj.shape[0]
    C = num_heads * dim + (num_kv_heads * (dim + vdim) if own_kv else 0)
    taps = conv_weight.shape[1] if conv_weight is not None else 1
    _need(proj.dtype == torch.float32 and proj.stride(1) == 1 and proj.shape[1] >= C, "conv_rope_kv: projections must be float32 rows")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == C), "conv_rope_kv: bias must be float32 [channels]")
    _need(conv_weight is None or (conv_weight.dtype == torch.float32 and conv_weight.is_contiguous() and conv_weight.shape[0] == C),
          "conv_rope_kv: convolution weight must be float32 [channels, taps]")
    _need(taps == 1 or (state is not None and state.dtype == torch.float32 and state.is_contiguous()
                        and tuple(state.shape[1:]) == (taps - 1, C)), "conv_rope_kv: state must be float32 [slots, taps - 1, channels]")
    _need(inv_freq.dtype == torch.float64 and inv_freq.numel() * 2 == rot_dims, "conv_rope_kv: inv_freq must be float64 [rot_dims / 2]")
    _need(q_out.is_contiguous() and tuple(q_out.shape) == (T, num_heads * dim), "conv_rope_kv: query output shape")
    if own_kv:
        _need(pool is not None and pool.is_contiguous() and pool.dim() == 5 and pool.shape[1] == 2 and pool.shape[-1] >= max(dim, vdim)
              and pool.dtype == q_out.dtype and slot_mapping is not None,
              "conv_rope_kv: the cache must be [pages, 2, kv heads, page, >= max(dim, vdim)] of the activations' dtype")
    meta = ctx.attn_meta
    _call("me_conv_rope_kv", proj.data_ptr(), proj.stride(0), _ptr(bias), _ptr(conv_weight), _ptr(state) if taps > 1 else 0, taps,
          inv_freq.data_ptr(), rot_dims, ctx.positions.data_ptr(), ctx.token_req.data_ptr(), meta.cu_seqlens.data_ptr(),
          meta.context_lens.data_ptr(), ctx.state_slots.data_ptr(), _ptr(slot_mapping) if own_kv else 0, q_out.data_ptr(),
          _ptr(pool) if own_kv else 0, _dt(q_out), T, meta.num_reqs, num_heads, num_kv_heads, dim, vdim,
          pool.shape[-1] if own_kv else 0, 1 if own_kv else 0, page_size, 1 if meta.num_decodes == meta.num_reqs else 0,
          _ptr(angles), _stream())


ROPE_TABLE_MIN_TOKENS = 64     # steps from this many tokens on form the rotation's cosines and sines once for all layers


def rope_table(positions: torch.Tensor, inv_freq: torch.Tensor, out: torch.Tensor) -> None:
    """``out`` [T, rot_dims / 2, 2] float32: (cosine, sine) of position x frequency for every token of the step, the angle
    formed in double precision as ``conv_rope_kv`` forms it."""
    T, half = positions.shape[0], inv_freq.numel()
    _need(inv_freq.dtype == torch.float64 and out.dtype == torch.float32 and out.is_contiguous() and out.numel() == T * half * 2,
          "rope_table: inv_freq float64 [half], out float32 [T, half, 2]")
    _call("me_rope_table", positions.data_ptr(), inv_freq.data_ptr(), half, T, out.data_ptr(), _stream())


use_sink_attention_mma = True     # bfloat16 attention with a sink on the tensor cores where the sizes allow; a switch for comparisons


def sink_attention(q: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor, pool: torch.Tensor, page_size: int,
                   block_tables: torch.Tensor, meta, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                   window: Optional[int], sink: bool, sinks: Optional[torch.Tensor] = None, softcap: Optional[float] = None,
                   keep_first: int = 0, chunk: Optional[int] = None, pooled: Optional[tuple] = None, bias: Optional[tuple] = None,
                   pairs: Optional[tuple[float, float, float]] = None, padded: bool = False, gate_heads: bool = False) -> None:
    """Attention over the paged cache with keys of ``dim`` and values of ``vdim`` elements: ``q`` [T, heads * dim] -> ``out``
    [T, heads * vdim]; a query at position p sees keys p - window < j <= p; with ``sink`` the softmax's denominator has one
    more term, exp(0); ``gate`` (float32 rows of pre-activations, heads * vdim wide; with ``gate_heads`` one a head) multiplies the
    output by its sigmoid.
    ``sinks`` (float32 [heads]): the term is exp(sinks[head]) instead; ``softcap`` c: scores become c tanh(s / c) after the
    scale; ``keep_first``: the window also shows keys j < keep_first; ``chunk`` (instead of a window): a query sees the keys
    j <= p with floor(j / chunk) = floor(p / chunk).  ``pooled`` = (cache, block tables, P): a second cache of the same layout
    with one row per block of P tokens (``pool_kv``); beside its window a query sees the rows of the blocks that lie wholly in
    front of the window, (b + 1) P <= p - window + 1, in the same softmax.

    ``bias`` = (r1, r2), float32 [heads] each: r1 ln(1 + r2 (p - j)) is taken off the scaled score of a key at distance p - j.
    ``pairs`` = (lambda, gain, eps): heads 2h and 2h + 1 are two maps over the same values, and ``out`` [T, heads / 2 * vdim] is what
    ``diff_combine`` makes of them.  ``padded``: the rows of q and of the cached keys are filled with zeros up to the cache's row
    size (``dim`` is that size), so that heads of any size up to it run the tensor-core kernels.

    bfloat16 with keys and values of 64 or 128 elements (the cache row's size) runs the engine's tensor-core kernels, the
    tcgen05 one for portions of prompts and the split-K one for single tokens; everything else the CUDA-core kernel of
    csrc/sink_attention.cu."""
    T = q.shape[0]
    HD = pool.shape[-1]
    _need(q.stride(1) == 1 and out.stride(1) == 1 and q.shape[1] == num_heads * dim
          and tuple(out.shape) == (T, num_heads // (2 if pairs else 1) * vdim) and (not pairs or num_heads % 2 == 0), "sink_attention: shapes")
    _need(not padded or (dim == HD and (gate is None or gate_heads)),
          "sink_attention: padded rows of q are as wide as the cache's, and go without a gate an element")
    _need(bias is None or (all(b.dtype == torch.float32 and b.numel() == num_heads and b.is_contiguous() for b in bias)
                           and not (softcap or sink or sinks is not None or pooled or keep_first or chunk)),
          "sink_attention: a distance bias is two float32 numbers a head and goes with a plain window at most")
    _need(pairs is None or not (gate is not None or sink or sinks is not None or pooled), "sink_attention: pairs go without gates, sinks and pooled blocks")
    _need(pool.dtype == q.dtype == out.dtype and pool.is_contiguous() and pool.dim() == 5 and pool.shape[1] == 2 and HD >= max(dim, vdim),
          "sink_attention: the cache must be [pages, 2, kv heads, page, >= max(dim, vdim)] of the activations' dtype")
    _need(gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1 and gate.shape[1] == num_heads * (1 if gate_heads else vdim)),
          "sink_attention: the gate must be float32 rows")
    _need(block_tables.dtype == torch.int32 and block_tables.stride(1) == 1, "sink_attention: block tables")
    _need(sinks is None or (sinks.dtype == torch.float32 and sinks.numel() == num_heads and sinks.is_contiguous()),
          "sink_attention: learned sinks are float32 [heads]")
    _need(not (chunk and window), "sink_attention: a window or chunks, not both")
    masked = bool(softcap or keep_first or chunk or bias)      # what only the kernels fed by tensor-map loads know
    pool_p = 0
    if pooled is not None:
        _need(window and not chunk and not keep_first, "sink_attention: pooled blocks go with a plain window")
        _need(pooled[0].dtype == pool.dtype and pooled[0].shape[1:] == pool.shape[1:] and pooled[0].is_contiguous()
              and pooled[1].dtype == torch.int32 and pooled[1].stride(1) == 1 and int(pooled[2]) >= 1,
              "sink_attention: the pooled cache has the layout and dtype of the cache, int32 tables and a block size")
        pool_p = int(pooled[2])
    decodes, tiles_left = meta.num_decodes, True
    fast = (use_sink_attention_mma and q.dtype == torch.bfloat16 and (dim == vdim == HD or padded) and HD in (64, 128)
            and meta.error_flag is not None and q.is_contiguous() and q.data_ptr() % 16 == 0)
    extras = dict(keep_first=keep_first, chunk=chunk or 0, softcap=softcap or 0.0, sinks=sinks, bias=bias, out_dim=vdim, gate_heads=gate_heads)
    joined_from = 0                                     # with pairs: the rows from here on that diff_combine joins
    if fast and decodes and (not (masked or pooled) or (page_size >= 8 and DECODE_PARTITION % page_size == 0)):
        attention_decode(q, out, num_heads, num_kv_heads, HD, pool, page_size, block_tables, meta, scale, window, sink=sink, gate=gate,
                         pooled=pooled, pairs=pairs, **extras)
        joined_from, decodes = decodes, 0
    if (fast and meta.num_tiles > 0 and use_tcgen05_attention and prefill_tcgen05_heads_per_block(num_heads, num_kv_heads, HD, page_size) > 0
            and vdim % 8 == 0 and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0):
        attention_prefill_tcgen05(q, out, num_heads, num_kv_heads, HD, pool, page_size, block_tables, meta, scale, window,
                                  sink=sink, gate=gate, pooled=pooled, pairs=pairs, **extras)
        tiles_left = False
    tiles, n_tiles = meta.tile_lists[SINK_ATTN_TILE_Q]
    if not tiles_left:
        n_tiles = 0
    if decodes or n_tiles:
        joined = out
        if pairs:
            out = meta.workspace("attn_maps", (T, num_heads * vdim), q.dtype)
        _call("me_sink_attn", q.data_ptr(), _dt(q), q.stride(0), _ptr(gate), gate.stride(0) if gate is not None else 0, out.data_ptr(),
              out.stride(0), pool.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), meta.cu_seqlens.data_ptr(),
              meta.context_lens.data_ptr(), tiles.data_ptr(), n_tiles, decodes, num_heads, num_kv_heads, dim, vdim, HD, page_size,
              float(scale), int(window or 0), 1 if sink else 0, _ptr(sinks), float(softcap or 0.0), int(keep_first or 0),
              int(chunk or 0), pooled[0].data_ptr() if pool_p else 0, pooled[1].data_ptr() if pool_p else 0,
              pooled[1].stride(0) if pool_p else 0, pool_p, _ptr(bias[0]) if bias else 0, _ptr(bias[1]) if bias else 0, 1 if gate_heads else 0, _stream())
        if pairs:
            diff_combine(out, joined, num_heads // 2, vdim, *pairs, first=joined_from)


def moe_route(logits: torch.Tensor, bias: Optional[torch.Tensor], top: int, idx: torch.Tensor, weights: torch.Tensor) -> None:
    """The ``top`` largest of every row of ``logits`` [T, E] + ``bias`` (float32) and the softmax over those only."""
    T, E = logits.shape
    _need(logits.dtype == torch.float32 and logits.is_contiguous(), "moe_route: logits must be float32")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == E), "moe_route: bias must be float32 [E]")
    _need(idx.dtype == torch.int32 and weights.dtype == torch.float32 and tuple(idx.shape) == tuple(weights.shape) == (T, top)
          and idx.is_contiguous() and weights.is_contiguous(), "moe_route: outputs are [T, top]")
    _call("me_moe_route", logits.data_ptr(), _ptr(bias), T, E, top, idx.data_ptr(), weights.data_ptr(), _stream())


def moe_route_grouped(logits: torch.Tensor, correction: Optional[torch.Tensor], top: int, groups: int, keep: int, idx: torch.Tensor,
                      weights: torch.Tensor, softmax: bool = False, scale: float = 1.0) -> None:
    """Routing by sigmoid scores with a correction that only steers the choice, over groups of neighbouring experts: s =
    sigmoid(``logits``) [T, E]; choice scores s + ``correction``; a group's score is the sum of its two largest choice scores;
    the ``top`` best experts of the ``keep`` best groups are chosen (ties: the lower index); ``weights`` are their s times ``scale``.
    ``softmax``: s is the softmax over all experts, and a group's score is its largest choice score.  ``logits`` may be columns of
    wider rows."""
    T, E = logits.shape
    _need(logits.dtype == torch.float32 and logits.stride(1) == 1, "moe_route_grouped: logits must be float32")
    _need(correction is None or (correction.dtype == torch.float32 and correction.numel() == E), "moe_route_grouped: correction must be float32 [E]")
    _need(idx.dtype == torch.int32 and weights.dtype == torch.float32 and tuple(idx.shape) == tuple(weights.shape) == (T, top)
          and idx.is_contiguous() and weights.is_contiguous(), "moe_route_grouped: outputs are [T, top]")
    _call("me_moe_route_grouped", logits.data_ptr(), logits.stride(0), _ptr(correction), T, E, top, int(groups), int(keep),
          1 if softmax else 0, float(scale), idx.data_ptr(), weights.data_ptr(), _stream())


def moe_route_grouped_sort(logits: torch.Tensor, correction: Optional[torch.Tensor], top: int, groups: int, keep: int, idx: torch.Tensor,
                           weights: torch.Tensor, counts: torch.Tensor, offsets: torch.Tensor, order: torch.Tensor, place: torch.Tensor,
                           softmax: bool = False, scale: float = 1.0) -> None:
    """``moe_route_grouped`` and ``moe_sort`` together; a step of few tokens does both in one kernel."""
    T, E = logits.shape
    _need(logits.dtype == torch.float32 and logits.stride(1) == 1 and (correction is None or (correction.dtype == torch.float32 and correction.numel() == E)),
          "moe_route_grouped_sort: logits and correction must be float32")
    _need(idx.dtype == torch.int32 and weights.dtype == torch.float32 and tuple(idx.shape) == tuple(weights.shape) == (T, top)
          and idx.is_contiguous() and weights.is_contiguous(), "moe_route_grouped_sort: outputs are [T, top]")
    _need(all(t.dtype == torch.int32 and t.is_contiguous() for t in (counts, offsets, order, place)) and counts.numel() >= E
          and offsets.numel() >= E + 1 and order.numel() >= T * top and place.numel() >= T * top, "moe_route_grouped_sort: output sizes")
    _call("me_moe_route_grouped_sort", logits.data_ptr(), logits.stride(0), _ptr(correction), T, E, top, int(groups), int(keep),
          1 if softmax else 0, float(scale), idx.data_ptr(), weights.data_ptr(), counts.data_ptr(), offsets.data_ptr(), order.data_ptr(), place.data_ptr(), _stream())


def moe_sort(idx: torch.Tensor, num_experts: int, counts: torch.Tensor, offsets: torch.Tensor, order: torch.Tensor,
             place: torch.Tensor) -> None:
    """Group the (token, choice) pairs of ``idx`` [T, top] by expert: ``offsets`` [E + 1], ``order`` (pair ids in expert order,
    token order inside an expert), ``place`` (where every pair went)."""
    T, top = idx.shape
    _need(all(t.dtype == torch.int32 and t.is_contiguous() for t in (idx, counts, offsets, order, place)), "moe_sort: int32 tensors")
    _need(counts.numel() >= num_experts and offsets.numel() >= num_experts + 1 and order.numel() >= T * top and place.numel() >= T * top,
          "moe_sort: output sizes")
    _call("me_moe_sort", idx.data_ptr(), T, top, num_experts, counts.data_ptr(), offsets.data_ptr(), order.data_ptr(),
          place.data_ptr(), _stream())


def moe_route_sort(logits: torch.Tensor, bias: Optional[torch.Tensor], top: int, idx: torch.Tensor, weights: torch.Tensor,
                   counts: torch.Tensor, offsets: torch.Tensor, order: torch.Tensor, place: torch.Tensor) -> None:
    """``moe_route`` and ``moe_sort`` together; a step of few tokens does both in one kernel."""
    T, E = logits.shape
    _need(logits.dtype == torch.float32 and logits.is_contiguous() and (bias is None or (bias.dtype == torch.float32 and bias.numel() == E)),
          "moe_route_sort: logits and bias must be float32")
    _need(idx.dtype == torch.int32 and weights.dtype == torch.float32 and tuple(idx.shape) == tuple(weights.shape) == (T, top)
          and idx.is_contiguous() and weights.is_contiguous(), "moe_route_sort: outputs are [T, top]")
    _need(all(t.dtype == torch.int32 and t.is_contiguous() for t in (counts, offsets, order, place)) and counts.numel() >= E
          and offsets.numel() >= E + 1 and order.numel() >= T * top and place.numel() >= T * top, "moe_route_sort: output sizes")
    _call("me_moe_route_sort", logits.data_ptr(), _ptr(bias), T, E, top, idx.data_ptr(), weights.data_ptr(), counts.data_ptr(),
          offsets.data_ptr(), order.data_ptr(), place.data_ptr(), _stream())


use_moe_mma = True        # bfloat16 expert products on the tensor cores where the sizes allow; a switch for comparisons
moe_tcgen05_tile_n = 0    # 0: by rule; 128 or 256: the accumulator's width of the experts' tcgen05 product (for comparisons)
MOE_TCGEN05_MIN_ROWS = 512   # (token, choice) pairs from which the experts' products run the tcgen05 kernel (tiles of 128 rows)


def moe_gemm(a: torch.Tensor, order: Optional[torch.Tensor], top: int, weight: torch.Tensor, offsets: torch.Tensor,
             out: torch.Tensor, glu: Optional[tuple] = None, workspace=None, err: Optional[torch.Tensor] = None,
             activation: Optional[str] = None) -> None:
    """One product per expert: ``weight`` [E, N or 2N, K]; the rows of ``a`` are gathered through ``order`` (pair id // top) or,
    without it, lie in expert order already; ``out`` [pairs, N] in expert order.  ``glu`` = (limit, alpha[, shift]): the weight holds gate
    rows then up rows and the result is the gated activation g sigmoid(alpha g) (u + shift), clamped by a positive limit (shift 1
    when it is not given).  ``activation`` (a key of ``ACTIVATIONS``, instead of ``glu``): that function of the plain product, in the
    product's epilogue in all three kernels.

    bfloat16 operands with K a multiple of 8 run on the tensor cores: from ``MOE_TCGEN05_MIN_ROWS`` pairs on (and with
    ``workspace`` and ``err`` given) the tcgen05 kernel of csrc/gemm_tcgen05.cu over rows brought into expert order first,
    below that the mma.sync kernel of csrc/moe_mma.cu, which gathers its rows itself; everything else the CUDA cores."""
    E, NN, K = weight.shape
    N = NN // 2 if glu else NN
    rows = out.shape[0]
    _need(weight.is_contiguous() and a.stride(1) == 1 and a.shape[1] == K and out.stride(1) == 1 and out.shape[1] == N, "moe_gemm: shapes")
    _need(order is not None or a.shape[0] == rows, "moe_gemm: rows in expert order")
    limit, alpha, shift = (tuple(glu) + (1.0,))[:3] if glu else (0.0, 0.0, 0.0)
    _need(activation is None or (not glu and activation in ACTIVATIONS), "moe_gemm: an activation instead of the gate, by a known name")
    epi = 1 if glu else (2 + ACTIVATIONS[activation] if activation else 0)
    if (use_moe_mma and use_tcgen05_gemm and workspace is not None and err is not None and rows >= MOE_TCGEN05_MIN_ROWS
            and a.dtype == weight.dtype == torch.bfloat16 and K % 8 == 0 and weight.data_ptr() % 16 == 0
            and (out.dtype == torch.bfloat16 or (not glu and out.dtype == torch.float32))):
        if order is not None:
            gathered = workspace("moe_gathered", (rows, K), torch.bfloat16)
            _call("me_moe_gather", a.data_ptr(), _dt(a), a.stride(0), order.data_ptr(), top, gathered.data_ptr(), rows, K, _stream())
            a = gathered
        if a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0:
            bn = moe_tcgen05_tile_n if moe_tcgen05_tile_n else (256 if N >= 256 else 128)
            _call("me_gemm_tcgen05_grouped", matrix_tensor_map(a, 128).ptr, matrix_tensor_map(weight.view(E * NN, K), bn // 2 if glu else bn).ptr,
                  out.data_ptr(), _dt(out), out.stride(0), offsets.data_ptr(), E, rows, N, NN, K, epi, float(limit),
                  float(alpha), float(shift), bn, err.data_ptr(), _stream())
            return
        order = None
    _call("me_moe_gemm", a.data_ptr(), _dt(a), a.stride(0), _ptr(order), top, weight.data_ptr(), _dt(weight), weight.stride(0),
          offsets.data_ptr(), E, out.data_ptr(), _dt(out), out.stride(0), rows, N, K, epi, float(limit), float(alpha),
          float(shift), 1 if use_moe_mma else 0, _stream())


def moe_combine(rows: torch.Tensor, place: torch.Tensor, weights: torch.Tensor, shared: Optional[torch.Tensor], out: torch.Tensor,
                shared_gate: Optional[torch.Tensor] = None) -> None:
    """``out[t] = sum_k weights[t, k] * rows[place[t, k]]`` (+ ``shared[t]``); ``rows`` float32 in expert order.  ``shared_gate`` (float32,
    one number a token, possibly a column of wider rows): its sigmoid multiplies ``shared[t]``."""
    T, top = weights.shape
    W = rows.shape[1]
    _need(rows.dtype == torch.float32 and rows.stride(1) == 1 and tuple(out.shape) == (T, W) and out.stride(1) == 1, "moe_combine: shapes")
    _need(shared is None or (tuple(shared.shape) == (T, W) and shared.stride(1) == 1), "moe_combine: the shared expert's output")
    _need(shared_gate is None or (shared_gate.dtype == torch.float32 and shared_gate.shape[0] == T), "moe_combine: the shared expert's gate is float32 [T]")
    _call("me_moe_combine", rows.data_ptr(), rows.stride(0), place.data_ptr(), weights.data_ptr(), top, _ptr(shared),
          _dt(shared) if shared is not None else 0, shared.stride(0) if shared is not None else 0, _ptr(shared_gate),
          shared_gate.stride(0) if shared_gate is not None else 0, out.data_ptr(), _dt(out), out.stride(0), T, W, _stream())


def token_side_gate(z: torch.Tensor, token_ids: torch.Tensor, feedback: Optional[torch.Tensor], table: torch.Tensor, first: int,
                    out: torch.Tensor) -> None:
    """``out[t, j] = gelu_tanh(z[t, j]) * table[token_t, first + j]``."""
    T, dim = z.shape
    _need(z.stride(1) == 1 and out.is_contiguous() and tuple(out.shape) == (T, dim) and table.is_contiguous(), "token_side_gate: shapes")
    _need(token_ids.dtype == torch.int32 and token_ids.numel() == T, "token_side_gate: token ids must be int32 [T]")
    _call("me_token_side_gate", z.data_ptr(), _dt(z), z.stride(0), token_ids.data_ptr(), _ptr(feedback), table.data_ptr(), _dt(table),
          table.stride(0), table.shape[0], first, dim, out.data_ptr(), _dt(out), T, _stream())
