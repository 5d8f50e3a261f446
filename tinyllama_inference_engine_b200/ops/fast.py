"""The bfloat16 serving kernels: tensor-core matrix products and attention.

Kept apart from the core set because they are specialised (by head size, by shape)
and compiled only for what a model needs.
"""
from __future__ import annotations

import functools
import os
import weakref
from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from ..errors import KernelError
from .build import build_library, load_library

library_gemm_calls = 0  # vendor-library matrix products issued (not this engine's kernels)


@functools.lru_cache(maxsize=None)
def sm_count() -> int:
    """Streaming multiprocessors of the current CUDA device (148 on a B200, which is also the answer without a device)."""
    if torch.cuda.is_available():
        return int(torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count)
    return 148

DEFAULT_HEAD_DIMS = (64, 128)
DEFAULT_MIXED_PREFILL_SETS = ((64, 64, 4), (128, 128, 8))   # (key width, value width, key heads per folded query) built ahead; others on first use
DEFAULT_SIGMOID_SETS = ((64, 64, 4), (128, 128, 4))   # (key width, value width, key/value heads) of attention with sigmoid weights built ahead; others on first use
DEFAULT_HEADS_DECODE_SETS = ((64, 64), (128, 128), (192, 128))   # (key width, value width) of softmax attention of single rows built ahead; others on first use
DEFAULT_DIFF_SETS = ((64, 128), (128, 128))   # (key width per map, value width) of differential attention built ahead; others on first use
_scratch: dict[torch.device, list[torch.Tensor]] = {}


def build_all() -> list:
    built = [build_library(f"tlie_attn_decode_d{d}", ["attention_decode.cu"], {"HEAD_DIM": d}) for d in DEFAULT_HEAD_DIMS]
    built.append(build_library("tlie_attn_decode_d64_w4", ["attention_decode.cu"], {"HEAD_DIM": 64, "DECODE_WARPS": 4, "DECODE_STAGES": 3}))
    built += [build_library(f"tlie_attn_prefill_d{d}", ["attention_prefill.cu"], {"HEAD_DIM": d}) for d in DEFAULT_HEAD_DIMS]
    built.append(build_library("tlie_gemv_fused", ["gemv_fused.cu"]))
    built.append(build_library("tlie_gemm_skinny", ["gemm_skinny.cu"]))
    built.append(build_library("tlie_gemm_tcgen05", TCGEN05_SOURCES))
    built.append(build_library("tlie_attn_prefill_tc", ["attention_prefill_tc.cu"]))
    built.append(build_library("tlie_attn_prefill_tc_sigmoid", ["attention_prefill_tc.cu"], {"SIGMOID_WEIGHTS": 1}))
    built.append(build_library("tlie_attn_prefill_tc_capped", ["attention_prefill_tc.cu"], {"SCORE_CAP": 1}))
    built.append(build_library("tlie_attn_prefill_tc_planes_k192_v128_capped", ["attention_prefill_tc.cu"], {"PLANES": 1, "KEY_DIM": 192, "VALUE_DIM": 128, "SCORE_CAP": 1}))
    built += [build_library(f"tlie_attn_heads_decode_k{k}_v{v}", ["attention_heads_decode.cu"], {"KEY_DIM": k, "VALUE_DIM": v}) for k, v in DEFAULT_HEADS_DECODE_SETS]
    built.append(build_library("tlie_probes", ["probes.cu"]))
    for key_dim, value_dim, parts in DEFAULT_MIXED_PREFILL_SETS:
        built.append(build_library(f"tlie_attn_mixed_k{key_dim}_v{value_dim}_p{parts}", ["attention_mixed_prefill.cu"], {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "PARTS": parts}))
        built.append(build_library(f"tlie_attn_mixed_decode_k{key_dim}_v{value_dim}_g{parts}", ["attention_mixed_decode.cu"],
                                   {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "KV_HEADS": parts}))
    built.append(build_library("tlie_attn_latent_rows_k192_r64_v128", ["attention_prefill_tc.cu"], {"LATENT_ROWS": 1, "KEY_DIM": 192, "ROT_DIM": 64, "VALUE_DIM": 128}))
    built.append(build_library("tlie_attn_latent_k576_v512", ["attention_latent_prefill.cu"], {"KEY_DIM": 576, "VALUE_DIM": 512}))   # other widths on first use
    for key_dim, value_dim, kv_heads in DEFAULT_SIGMOID_SETS:
        built.append(build_library(f"tlie_attn_sigmoid_k{key_dim}_v{value_dim}_p1", ["attention_mixed_prefill.cu"], {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "PARTS": 1, "SIGMOID_WEIGHTS": 1}))
        built.append(build_library(f"tlie_attn_mixed_decode_k{key_dim}_v{value_dim}_g{kv_heads}", ["attention_mixed_decode.cu"],
                                   {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "KV_HEADS": kv_heads}))
    for key_dim, value_dim in DEFAULT_DIFF_SETS:
        built.append(build_library(f"tlie_attn_diff_k{key_dim}_v{value_dim}", ["attention_diff_prefill.cu"], {"KEY_DIM": key_dim, "VALUE_DIM": value_dim}))
    return built


_ops_module = None


def _ops():
    global _ops_module
    if _ops_module is None:
        from .. import ops

        _ops_module = ops
    return _ops_module


GEMV_KERNEL_MAX_ROWS = 16   # what gemv_fused.cu can take
# Up to this many rows a step uses the fused decode kernels (norm + product, product + residual add, gate).  Measured on the
# 1.1B shapes, a decode step of 9 / 12 / 16 requests: 1.10 / 1.15 / 1.20 ms on them, 1.14 / 1.20 / 1.23 to 1.30 ms on the
# library's product with separate norm and activation kernels.  (With four weight blocks in flight per thread instead of
# eight in the 16-row kernels that read x directly, the fused step took 1.34 to 1.49 ms and lost.)
FUSED_MAX_ROWS = 16
_EPILOGUES = {"store": None, "accumulate": 2, "gated": 3}


def gemv_library():
    return load_library("tlie_gemv_fused", ["gemv_fused.cu"])


def gemv_fits(rows: int, K: int, norm: bool, gated: bool = False, N: int | None = None) -> bool:
    """Whether the fused kernel's shared memory (x as bfloat16 and the warps' partial tiles) fits.

    ``N`` (plain bfloat16 x only): with no more 16-row tiles than the kernel has CTA slots, every CTA computes one tile, uses each
    element of x once and reads it straight from global memory: nothing of x is staged, and any K fits (the down projection of
    wide models: K = 14,336 would need 229 KB for eight staged rows)."""
    if rows > GEMV_KERNEL_MAX_ROWS or K % 8 != 0:
        return False
    if not norm and not gated and N is not None and -(-N // 16) <= 2 * sm_count():
        return True
    padded_rows = 8 if rows <= 8 else 16
    stride = K + ((32 - K % 64) + 64) % 64
    stride += 64 if stride == K else 0
    need = padded_rows * stride * 2 + 8 * 16 * (padded_rows + 1) * 4
    return need <= 200 * 1024


def prepared_norm_buffers(rows: int, width: int, device) -> tuple:
    """Where a product that completes the residual leaves the next norm's input: bfloat16(residual * norm weight) [rows, width]
    and the rows' sums of squares per 16 columns, 32-bit [rows, ceil(width / 16)]."""
    return (torch.empty((rows, width), dtype=torch.bfloat16, device=device), torch.empty((rows, -(-width // 16)), dtype=torch.float32, device=device))


GEMV_ACTIVATIONS = {None: 0, "relu_squared": 1, "gelu_tanh": 2, "silu": 3, "xielu": 4}


GEMV_GATES = {"silu": 0, "gelu_tanh": 2}   # the gated epilogue's activation (1 is the clamped gate, chosen by ``clamp``)


def gemv_fused(x, weight, out, *, norm=None, epilogue: str = "store", prepared=None, prepare=None, activation: str | None = None, constants=(0.0, 0.0),
               clamp=None, gate: str = "silu", bias=None, prepare_curve=None) -> None:
    """out (+)= f(x) . weight^T for up to 16 rows, one kernel.

    norm      None: ``x`` is bfloat16 [M, K].  (norm_weight, eps, rows): ``x`` is the 32-bit residual stream and
              the operand is rmsnorm(x[rows]) * norm_weight (rows None: the first M rows).
    prepared  (squares, eps): ``x`` is bfloat16(residual * norm weight) [M, K] and ``squares`` [M, tiles] the rows' sums of
              squares, as an earlier "accumulate" with ``prepare`` left them; the operand is the same rmsnorm.
    epilogue  "store": out [M, N] bfloat16 or 32-bit;  "accumulate": out is the 32-bit residual, out += result;
              "gated": weight is [gate rows | up rows], out [M, N / 2] = silu(gate) * up; with ``clamp`` = (limit, alpha, shift) instead
              g * sigmoid(alpha * g) * (u + shift) for g = min(gate, limit), u = clamp(up, -limit, limit); with ``gate`` = "gelu_tanh" the gate's
              activation is gelu in its tanh form.
    activation ("store" into bfloat16 only) "relu_squared", "gelu_tanh", "silu" or "xielu" (which takes two ``constants``, see ``ops.activation``): applied to
              the rounded product before it is stored.
    bias      ("store" into bfloat16 only) 32-bit [N], added to the sums before they are rounded.
    prepare   ("accumulate" only) (norm_weight [N], x_out bfloat16 [M, N], squares_out [M, ceil(N / 16)]): also store
              bfloat16(out * norm_weight) and the rows' sums of squares per 16 columns, for a later call with ``prepared``.
    prepare_curve ("accumulate" only, in the place of ``prepare``) (alpha, weight [N], bias [N], x_out bfloat16 [M, N]): also store
              bfloat16(tanh(alpha * out) * weight + bias), the finished operand of the product after this one.
    """
    ops = _ops()
    N, K = weight.shape
    M = out.shape[0]
    if weight.dtype != torch.bfloat16 or M > GEMV_KERNEL_MAX_ROWS or K % 8 != 0:
        raise KernelError(f"gemv_fused takes bfloat16 weights with K % 8 == 0 and at most {GEMV_KERNEL_MAX_ROWS} rows", code="invalid_shape")
    code = _EPILOGUES[epilogue]
    if epilogue == "store":
        code = 1 if out.dtype == torch.float32 else 0
    elif epilogue == "accumulate" and out.dtype != torch.float32:
        raise KernelError("gemv_fused accumulates into the 32-bit residual only", code="invalid_dtype")
    if activation is not None and (epilogue != "store" or out.dtype != torch.bfloat16 or activation not in GEMV_ACTIVATIONS):
        raise KernelError("gemv_fused applies an activation only when it stores bfloat16", code="invalid_argument")
    if bias is not None and (epilogue != "store" or out.dtype != torch.bfloat16 or bias.dtype != torch.float32 or bias.numel() != N):
        raise KernelError("gemv_fused adds a 32-bit bias [N] only when it stores bfloat16", code="invalid_argument")
    if out.shape[1] != (N // 2 if epilogue == "gated" else N):
        raise KernelError("gemv_fused: the output's width does not fit the weight", code="invalid_shape")
    consume = (c_void_p(0), c_int(0))
    if prepared is not None:
        squares, eps = prepared
        if x.dtype != torch.bfloat16 or x.shape != (M, K) or not x.is_contiguous() or squares.dtype != torch.float32 or squares.shape[0] != M or not squares.is_contiguous():
            raise KernelError("gemv_fused: a prepared norm is bfloat16 [M, K] with 32-bit sums of squares [M, tiles]", code="invalid_shape")
        args = (c_int(3), ops._ptr(x), c_int(K), c_void_p(0), c_void_p(0), c_float(eps))
        consume = (ops._ptr(squares), c_int(squares.shape[1]))
    elif norm is None:
        if x.dtype != torch.bfloat16 or x.shape != (M, K) or x.stride(1) != 1 or x.stride(0) % 8 != 0:
            raise KernelError("gemv_fused: x must be bfloat16 [M, K] with rows 16-byte aligned", code="invalid_shape")
        args = (c_int(0), c_void_p(x.data_ptr()), c_int(x.stride(0)), c_void_p(0), c_void_p(0), c_float(0.0))
    else:
        norm_weight, eps, rows = norm
        if x.dtype != torch.float32 or x.shape[1] != K or norm_weight.dtype != torch.float32 or norm_weight.numel() != K:
            raise KernelError("gemv_fused: the residual and the norm weight must be 32-bit and K wide", code="invalid_shape")
        args = (c_int(1), ops._ptr(x), c_int(K), ops._i32(rows, "rows"), ops._ptr(norm_weight), c_float(eps))
    if not out.is_cuda:
        raise KernelError("this engine has no CPU path: a kernel was given a tensor that is not on a CUDA device")
    emit = (c_void_p(0), c_void_p(0), c_void_p(0))
    if prepare is not None:
        norm_weight, x_out, squares_out = prepare
        if (epilogue != "accumulate" or norm_weight.dtype != torch.float32 or norm_weight.numel() != N or x_out.dtype != torch.bfloat16 or x_out.shape != (M, N)
                or squares_out.dtype != torch.float32 or squares_out.shape != (M, -(-N // 16)) or not x_out.is_contiguous() or not squares_out.is_contiguous()):
            raise KernelError("gemv_fused: prepare takes a 32-bit norm weight [N], bfloat16 [M, N] and 32-bit [M, ceil(N / 16)], with accumulate", code="invalid_shape")
        emit = (ops._ptr(norm_weight), ops._ptr(x_out), ops._ptr(squares_out))
    curve = (c_int(0), c_float(0.0), c_void_p(0))
    if prepare_curve is not None:
        alpha, curve_weight, curve_bias, x_out = prepare_curve
        if (epilogue != "accumulate" or prepare is not None or curve_weight.dtype != torch.float32 or curve_weight.numel() != N or curve_bias.dtype != torch.float32
                or curve_bias.numel() != N or x_out.dtype != torch.bfloat16 or x_out.shape != (M, N) or not x_out.is_contiguous()):
            raise KernelError("gemv_fused: prepare_curve takes a number, 32-bit weight and bias [N] and bfloat16 [M, N], with accumulate", code="invalid_shape")
        emit = (ops._ptr(curve_weight), ops._ptr(x_out), c_void_p(0))
        curve = (c_int(1), c_float(alpha), ops._ptr(curve_bias))
    ops._check(gemv_library().tlie_gemv_fused(*args, ops._ptr(weight), ops._ptr(out), c_int(M), c_int(N), c_int(K), c_int(code), *consume, *emit, c_int(GEMV_ACTIVATIONS[activation]),
                                             c_int(GEMV_GATES[gate] if clamp is None else 1), *(c_float(float(v)) for v in (clamp or (0.0, 0.0, 0.0))), *(c_float(float(v)) for v in constants), ops._ptr(bias),
                                             *curve, ops._stream()), "gemv_fused")


# --- tensor-core product for 17 to 127 rows (tcgen05 with the operands swapped, K cut over a cluster) -----------------
SKINNY_MAX_ROWS = 127      # steps of more rows than the register-fed kernels take and fewer than a 128-row tile
# Off unless asked for (``enable_skinny`` or TLIE_SKINNY=1).  Measured on the 1.1B shapes, a decode step of 24 / 32 / 64 requests:
# 1.28 / 1.28 / 1.64 ms with this kernel and its fusions against 1.14 / 1.15 / 1.29 ms on the library's products with separate
# norm and activation kernels.  Its tiles are few (10 for 2,560 weight rows), so K is cut over a cluster, and what the CTAs then
# exchange (64 rows x 256 columns of 32-bit partial sums each) is half as many bytes as the weights they read.
use_skinny = False


def enable_skinny(on: bool = True) -> None:
    """Route products of 17 to 127 rows (and what surrounds them: norm in front, gate or residual add behind) to ``gemm_skinny``."""
    global use_skinny, FUSED_MAX_ROWS
    use_skinny = bool(on)
    FUSED_MAX_ROWS = SKINNY_MAX_ROWS if on else GEMV_KERNEL_MAX_ROWS


_SKINNY_EPILOGUES = {"store": None, "gated": 2, "accumulate": 3}


def skinny_library():
    return load_library("tlie_gemm_skinny", ["gemm_skinny.cu"])


def skinny_fits(rows: int, weight, x=None) -> bool:
    """Whether ``gemm_skinny`` takes a product of this many rows with this weight (and this x, if given)."""
    if not 1 <= rows <= SKINNY_MAX_ROWS or weight.dtype != torch.bfloat16 or weight.shape[1] % 8 != 0 or not weight.is_contiguous():
        return False
    return x is None or (x.dtype == torch.bfloat16 and x.is_contiguous() and x.data_ptr() % 16 == 0)


_skinny_packed: dict[tuple, tuple] = {}


def skinny_packed(weight: torch.Tensor, gated: bool = False) -> torch.Tensor:
    """The copy of ``weight`` that ``gemm_skinny`` streams: its 128 x 64 operand tiles, each as the contiguous 16 KB image the tensor
    cores read from shared memory (``gated``: a group is 64 gate rows and the 64 up rows of the same outputs).  Made on first use and
    kept for as long as the weight tensor lives: weights do not change, and a captured graph keeps pointing at the copy.  The entry
    is tied to the tensor object itself (an address alone could be handed to another tensor once this one is freed)."""
    key = (weight.data_ptr(), tuple(weight.shape), bool(gated), weight.device)
    found = _skinny_packed.get(key)
    if found is not None and found[0]() is weight:
        return found[1]
    ops = _ops()
    N, K = weight.shape
    library = skinny_library()
    if not getattr(library, "_tlie_typed", False):
        library.tlie_gemm_skinny_packed_elements.restype = c_longlong
        library._tlie_typed = True
    elements = library.tlie_gemm_skinny_packed_elements(c_int(N), c_int(K), c_int(1 if gated else 0))
    packed = torch.empty(elements, dtype=torch.bfloat16, device=weight.device)
    ops._check(library.tlie_gemm_skinny_pack(ops._ptr(weight), ops._ptr(packed), c_int(N), c_int(K), c_int(1 if gated else 0), ops._stream()), "gemm_skinny_pack")
    _skinny_packed[key] = (weakref.ref(weight, lambda _, key=key: _skinny_packed.pop(key, None)), packed)
    return packed


def skinny_square_runs(rows: int, N: int, K: int) -> int:
    """Partial sums of squares per row that ``gemm_skinny(..., prepare=)`` leaves for a [N, K] weight and this many rows."""
    return int(skinny_library().tlie_gemm_skinny_square_runs(c_int(rows), c_int(N), c_int(K)))


def gemm_skinny(x, weight, out, *, epilogue: str = "store", prepared=None, prepare=None) -> None:
    """out (+)= x . weight^T for up to 128 rows on the tensor cores, the weights streamed once; one kernel.

    x         bfloat16 [M, K], contiguous.
    prepared  (squares, eps): x is bfloat16(residual * norm weight) and ``squares`` [M, runs] (rows may be strided) partial sums of
              squares of the residual's rows; every result is scaled by its row's 1 / sqrt(mean + eps) (not with "accumulate").
    epilogue  "store": out [M, N] bfloat16 or 32-bit; "gated": weight is [gate rows | up rows], out [M, N / 2] = silu(gate) * up;
              "accumulate": out is the 32-bit residual [M, N], out += result.
    prepare   ("accumulate" only) (norm_weight [N], x_out bfloat16 [M, N], squares_out [M, skinny_square_runs(M, N, K)], rows may be
              strided): also leave the next norm's input, for a later call with ``prepared``.
    """
    ops = _ops()
    N, K = weight.shape
    M = x.shape[0]
    if not skinny_fits(M, weight, x) or x.shape[1] != K:
        raise KernelError(f"gemm_skinny takes contiguous bfloat16 operands with K % 8 == 0 and at most {SKINNY_MAX_ROWS + 1} rows", code="invalid_shape")
    code = _SKINNY_EPILOGUES[epilogue]
    if epilogue == "store":
        if out.dtype not in (torch.bfloat16, torch.float32):
            raise KernelError("gemm_skinny stores bfloat16 or 32-bit", code="invalid_dtype")
        code = 1 if out.dtype == torch.float32 else 0
    elif epilogue == "accumulate" and out.dtype != torch.float32:
        raise KernelError("gemm_skinny accumulates into the 32-bit residual only", code="invalid_dtype")
    elif epilogue == "gated" and (out.dtype != torch.bfloat16 or N % 2):
        raise KernelError("gemm_skinny: a gated product stores bfloat16 and its weight has an even number of rows", code="invalid_shape")
    if out.shape != (M, N // 2 if epilogue == "gated" else N) or not out.is_contiguous():
        raise KernelError("gemm_skinny: the output's shape does not fit the weight", code="invalid_shape")
    consume = (c_void_p(0), c_int(0), c_int(0), c_float(0.0))
    if prepared is not None:
        squares, eps = prepared
        if epilogue == "accumulate" or squares.dtype != torch.float32 or squares.dim() != 2 or squares.shape[0] != M or squares.stride(1) != 1 or not squares.is_cuda:
            raise KernelError("gemm_skinny: a prepared norm brings 32-bit sums of squares [M, runs], and not with accumulate", code="invalid_shape")
        consume = (c_void_p(squares.data_ptr()), c_int(squares.shape[1]), c_int(squares.stride(0)), c_float(eps))
    emit = (c_void_p(0), c_void_p(0), c_void_p(0), c_int(0))
    if prepare is not None:
        norm_weight, x_out, squares_out = prepare
        if (epilogue != "accumulate" or norm_weight.dtype != torch.float32 or norm_weight.numel() != N or x_out.dtype != torch.bfloat16 or x_out.shape != (M, N)
                or squares_out.dtype != torch.float32 or squares_out.dim() != 2 or squares_out.shape != (M, skinny_square_runs(M, N, K)) or squares_out.stride(1) != 1
                or not x_out.is_contiguous() or not squares_out.is_cuda):
            raise KernelError("gemm_skinny: prepare takes a 32-bit norm weight [N], bfloat16 [M, N] and 32-bit [M, skinny_square_runs(M, N, K)], with accumulate", code="invalid_shape")
        emit = (ops._ptr(norm_weight), ops._ptr(x_out), c_void_p(squares_out.data_ptr()), c_int(squares_out.stride(0)))
    ops._check(skinny_library().tlie_gemm_skinny(ops._ptr(x), ops._ptr(skinny_packed(weight, epilogue == "gated")), ops._ptr(out), c_int(M), c_int(N), c_int(K), c_int(code),
                                                 *consume, *emit, ops._ptr(tcgen05_error_flag(x.device)), ops._stream()), "gemm_skinny")


# --- tensor-core product for many rows (tcgen05, TMA, tensor memory) -------------------------------------
# Where the engine's own tcgen05 kernels run instead of the library's product (and, for the fused forms, the small kernel after
# it).  Measured with CUDA events in a replayed graph, weights from HBM, at 1.1B, 7B and 8B widths, 128 to 8,192 rows
# (`kernel-bench --products`): the engine's kernels are level with or ahead of the library wherever their tiles are wide and keep the
# SMs busy over whole waves and the product is large enough for its start and end not to count, and behind elsewhere, since a CTA
# runs all of K for its tile where the library also splits K:
#   * 1.1B widths, 2,048 rows: qkv 19.9 us (one wave of 288-wide tiles) against 19.0, o (adding) 17.5 against 22.0 for product + add
#     kernel; 1,024 rows: qkv 14.7 against 10.9 (half the work, the same start and end), o 16.5 against 14.1 (32 tiles for 74 pairs);
#   * 7B widths, 1,024 rows: o 28.1 against 33.8, down 67.3 against 71.2, qkv level; 8B widths, 1,024 rows: qkv 44.8 against 37.4 (96
#     tiles for 74 pairs: two waves, the second a third full);
#   * the gated product on pairs of SMs is ahead of product + activation kernel from 1,024 rows on (7B widths: 130 against
#     160 us; 1.1B widths: 46.7 against 45.5); below that it is ahead where the product is a large one (7B widths, 768 rows: 104
#     against 112 us; 8B widths, 512 rows: 100 against 112) and behind where it is not (1.1B widths, 768 rows: 36.4 against 34.5).
TCGEN05_MIN_ROWS = 1024            # below this the library was ahead at every width
TCGEN05_GATED_MIN_ROWS = 1024
TCGEN05_GATED_LARGE = (512, 80e9)  # the gated product also from this many rows on where it is this many flop or more
OWN_PRODUCT_MIN_EFFICIENCY = 0.75  # what the product's tiling costs against 256-wide tiles on every SM with no wave left partly empty (0.76: ahead, 0.73: behind)
OWN_PRODUCT_MIN_FLOP = 20e9        # a smaller product is mostly its start and end, where the library is ahead
OWN_ADDING_MIN_FLOP = 10e9         # the adding product also saves the add kernel
use_tcgen05 = True


TCGEN05_SOURCES = ["gemm_tcgen05.cu", "gemm_tcgen05_pair.cu"]


def tcgen05_takes(M: int, N: int, K: int, adding: bool = False) -> bool:
    """Whether a plain product (``adding``: one that adds into the residual) runs on this engine's tcgen05 kernels (else on the
    library's): from TCGEN05_MIN_ROWS rows on, where the tiling it would get is an efficient one (waves that are full, tiles that
    are not narrow: the cost model of ``_cheapest_tiles`` against its own ideal) and the product is not a small one.

    (Sharing a tile's k blocks among CTAs, which would fill the SMs for small products too, was tried in the one-SM kernel: the
    owner of a tile collects the others' partial accumulators at the very end of its share, eight trips to the L2 per partial
    tile with nothing left to hide them behind, and that cost more than even shares saved.)"""
    if M < TCGEN05_MIN_ROWS:
        return False
    pair = (use_sm_pairs and M >= PAIR_MIN_ROWS) if adding else pair_tiles_pay(M, N)
    _, cost, _ = _cheapest_tiles(M, N, pair, adding)
    ideal = -(-M // (256 if pair else 128)) * N / (sm_count() // 2 if pair else sm_count()) * (256 + 300) / 256
    return ideal / cost >= OWN_PRODUCT_MIN_EFFICIENCY and 2.0 * M * N * K >= (OWN_ADDING_MIN_FLOP if adding else OWN_PRODUCT_MIN_FLOP)


def gated_takes(M: int, N: int, K: int) -> bool:
    """Whether the gated product ([gate rows | up rows]: N rows of w in all) of a step of M rows runs on this engine's tcgen05 kernel."""
    return M >= TCGEN05_GATED_MIN_ROWS or (M >= TCGEN05_GATED_LARGE[0] and 2.0 * M * N * K >= TCGEN05_GATED_LARGE[1])


def tcgen05_library():
    return load_library("tlie_gemm_tcgen05", TCGEN05_SOURCES)


def tcgen05_error_flag(device: torch.device) -> torch.Tensor:
    """The device's error word: the tensor-core kernels set bit 0 of it if one of their bounded waits gave up."""
    return _ops().error_flag(device)


GEMM_TILE_WIDTHS = (256, 192, 160, 128)
GEMM_WIDE_TILES = (288, 320)   # two MMAs wide, one accumulator: for products that fit one wave of CTAs so (one-SM tiles only)


# Tiles of 256 rows on pairs of SMs (tcgen05 cta_group::2, gemm_tcgen05_pair.cu) bring a third less from L2 per flop.  That pays
# where a product is several waves of tiles, so that what the SMs can pull from L2 sets the pace: measured at 2,048 rows and
# K = 4,096, N = 12,288: 139 us on pairs, 153 on single SMs (the library: 142); N = 4,096, K = 11,008: 129, 163 (144); 8,192 rows,
# N = 6,144: 278, 317 (278).  The pairs have wide tiles of their own (two MMAs wide, one accumulator) for products that fit one
# wave of the pairs so: 2,048 x 4,096 is 128 tiles of 256 columns for 74 pairs, or 72 tiles of 480 (K = 11,008, adding into the
# residual: 132 -> 123.5 us; 2,048 x 3,072 x 3,072 with 384-wide tiles: 42.7 -> 36.6 us).  The gated product runs on pairs from
# 1,024 rows.
PAIR_MIN_ROWS = 1024
PAIR_TILE_WIDTHS = (256,)          # narrower tiles on pairs were behind the 256-wide ones wherever they were measured
PAIR_WIDE_TILES = (288, 384, 480)
PAIR_ADDING_WIDE_TILES = (384, 480)
PAIR_TILE_GAIN = 0.9               # a tile on a pair of SMs against two tiles of the same width on single SMs, where L2 sets the pace
use_sm_pairs = True


def _cheapest_tiles(M: int, N: int, pair: bool, adding: bool) -> tuple[int, int, int]:
    """(tile width, cost, waves) of the cheapest way to tile an M x N product on single SMs or on pairs: cost = waves x (width + 300).

    A tile costs its width plus a fixed part about as large as 300 columns (measured: a 128 x 160 tile takes 0.8 of the time
    of a 128 x 256 one), so the widest tile wins unless a narrower one saves a whole wave; the wider tile on a tie.  A wide
    tile has no second accumulator to work on while its epilogue runs, so it is a candidate only where no CTA gets two."""
    workers = sm_count() // 2 if pair else sm_count()
    row_blocks = -(-M // (256 if pair else 128))
    if pair:
        widths, wide = PAIR_TILE_WIDTHS, (PAIR_ADDING_WIDE_TILES if adding else PAIR_WIDE_TILES)
    else:
        widths, wide = ((256,), ()) if adding else (GEMM_TILE_WIDTHS, GEMM_WIDE_TILES)
    candidates = tuple(width for width in wide if row_blocks * -(-N // width) <= workers) + widths
    waves = lambda width: -(-(row_blocks * -(-N // width)) // workers)  # noqa: E731
    best = min(candidates, key=lambda width: (waves(width) * (width + 300), -width))
    return best, waves(best) * (best + 300), waves(best)


@functools.lru_cache(maxsize=4096)
def gemm_tile_width(M: int, N: int, pair: bool = False, adding: bool = False) -> int:
    """The tile width whose waves of persistent CTAs (or pairs of them) cost least; ``adding``: for the product that adds into the residual."""
    return _cheapest_tiles(M, N, pair, adding)[0]


@functools.lru_cache(maxsize=4096)
def pair_tiles_pay(M: int, N: int) -> bool:
    """Whether a plain product of this shape runs on pairs of SMs: where their cheapest tiling (with what a pair gains on two single
    SMs, if it is waves of tiles) costs less than the cheapest one-SM tiling; a product that one wave of one-SM tiles holds stays there."""
    if not use_sm_pairs or M < PAIR_MIN_ROWS:
        return False
    _, pair_cost, pair_waves = _cheapest_tiles(M, N, True, False)
    return (PAIR_TILE_GAIN if pair_waves > 1 else 1.0) * pair_cost < _cheapest_tiles(M, N, False, False)[1]


def gemm_tcgen05(x, weight, out, tile_n: int | None = None, pair: bool | None = None) -> None:
    """out[M, N] = x[M, K] . weight[N, K]^T on the 5th-generation tensor cores; bfloat16 in, bfloat16 or 32-bit out.

    ``pair``: 256-row tiles on pairs of SMs (each CTA loads half of the weight rows of a tile)."""
    ops = _ops()
    M, K = x.shape
    N = weight.shape[0]
    if x.dtype != torch.bfloat16 or weight.dtype != torch.bfloat16 or K % 8 != 0 or not x.is_contiguous():
        raise KernelError("gemm_tcgen05 takes contiguous bfloat16 operands with K % 8 == 0", code="invalid_shape")
    if pair is None:
        pair = tile_n is None and pair_tiles_pay(M, N)
    if tile_n is None:
        tile_n = gemm_tile_width(M, N, pair)
    library = tcgen05_library()
    entry = library.tlie_gemm_tcgen05_pair if pair else library.tlie_gemm_tcgen05
    ops._check(
        entry(ops._ptr(x), ops._ptr(weight), ops._ptr(out), c_int(M), c_int(N), c_int(K), c_int(1 if out.dtype == torch.float32 else 0),
              c_int(tile_n), ops._ptr(tcgen05_error_flag(x.device)), ops._stream()),
        "gemm_tcgen05",
    )


use_accumulate_epilogue = True   # o-proj and down-proj of prompt portions add into the residual from the product's epilogue


def can_accumulate(rows: int, weight) -> bool:
    """Whether ``gemm_tcgen05_accumulate`` takes residual += x . weight^T for this many rows."""
    N, K = weight.shape
    return (use_tcgen05 and use_accumulate_epilogue and weight.dtype == torch.bfloat16 and N % 4 == 0 and K % 8 == 0 and tcgen05_takes(rows, N, K, adding=True))


def gemm_tcgen05_accumulate(x, weight, residual, pair: bool | None = None, tile_n: int | None = None) -> None:
    """residual[M, N] (32-bit) += x[M, K] . weight[N, K]^T: the product's tiles are added by bulk tensor reductions, each element once.

    ``pair``: on pairs of SMs (default: from PAIR_MIN_ROWS rows on; these tiles are 256 wide either way, and the pairs were ahead
    at every shape measured: down-proj of 2,048 rows at 1.1B widths 38.4 -> 35.3 us, at 7B widths 146 -> 133, at 8B widths and
    8,192 rows 749 -> 668)."""
    ops = _ops()
    M, K = x.shape
    N = weight.shape[0]
    if (x.dtype != torch.bfloat16 or weight.dtype != torch.bfloat16 or residual.dtype != torch.float32 or residual.shape != (M, N) or K % 8 != 0 or N % 4 != 0
            or not x.is_contiguous() or not residual.is_contiguous()):
        raise KernelError("gemm_tcgen05_accumulate takes contiguous bfloat16 operands (K % 8 == 0) and a contiguous 32-bit residual [M, N] with N % 4 == 0", code="invalid_shape")
    if pair is None:
        pair = use_sm_pairs and M >= PAIR_MIN_ROWS
    if tile_n is None:
        tile_n = gemm_tile_width(M, N, pair, adding=True)
    library = tcgen05_library()
    entry = library.tlie_gemm_tcgen05_pair if pair else library.tlie_gemm_tcgen05
    ops._check(
        entry(ops._ptr(x), ops._ptr(weight), ops._ptr(residual), c_int(M), c_int(N), c_int(K), c_int(3), c_int(tile_n),
              ops._ptr(tcgen05_error_flag(x.device)), ops._stream()),
        "gemm_tcgen05_accumulate",
    )


def gemm_tcgen05_gated(x, weight, out, pair: bool | None = None) -> None:
    """out[M, I] = silu(x . gate^T) * (x . up^T) for weight = [gate rows | up rows] ([2 I, K]), one kernel."""
    ops = _ops()
    M, K = x.shape
    inter = weight.shape[0] // 2
    if x.dtype != torch.bfloat16 or weight.dtype != torch.bfloat16 or out.dtype != torch.bfloat16 or K % 8 != 0 or not x.is_contiguous() or out.shape != (M, inter):
        raise KernelError("gemm_tcgen05_gated takes contiguous bfloat16 operands with K % 8 == 0 and out [M, rows / 2]", code="invalid_shape")
    if pair is None:   # below the pairs' usual row count: where the rows are whole 256-row tiles (640 rows at 7B widths: 102 us on pairs, 96 on single SMs)
        pair = use_sm_pairs and (M >= PAIR_MIN_ROWS or (M >= 512 and M % 256 == 0))
    library = tcgen05_library()
    entry = library.tlie_gemm_tcgen05_pair if pair else library.tlie_gemm_tcgen05
    ops._check(
        entry(ops._ptr(x), ops._ptr(weight), ops._ptr(out), c_int(M), c_int(inter), c_int(K), c_int(2), c_int(256),
              ops._ptr(tcgen05_error_flag(x.device)), ops._stream()),
        "gemm_tcgen05_gated",
    )


def linear_bf16(x, weight, out) -> None:
    global library_gemm_calls
    if weight.dtype != torch.bfloat16 or out.dtype not in (torch.bfloat16, torch.float32):
        raise KernelError("linear: the bfloat16 path takes bfloat16 weights", code="invalid_dtype")
    if x.stride(0) % 8 == 0 and gemv_fits(x.shape[0], weight.shape[1], norm=False, N=weight.shape[0]):
        gemv_fused(x, weight, out)
        return
    if use_tcgen05 and tcgen05_takes(x.shape[0], weight.shape[0], weight.shape[1]) and weight.shape[1] % 8 == 0 and x.is_contiguous():
        gemm_tcgen05(x, weight, out)
        return
    if use_skinny and skinny_fits(x.shape[0], weight, x) and out.is_contiguous():
        gemm_skinny(x, weight, out)
        return
    library_gemm_calls += 1
    if out.dtype == torch.float32:
        torch.mm(x, weight.t(), out_dtype=torch.float32, out=out)
    else:
        torch.mm(x, weight.t(), out=out)


# --- decode attention -------------------------------------------------------------------------
def decode_attention_library(head_dim: int, narrow: bool = False):
    """The decode attention library of a head size.

    Default build: eight warps and two stages per CTA for head sizes up to 64 (one CTA per SM pulls enough bandwidth when
    there are few (request, kv head) pairs).  ``narrow``: four warps and three stages, two CTAs per SM, for steps with
    more pairs than SMs, where the wide CTAs would run in two uneven waves.
    """
    if narrow and head_dim <= 64:
        lib = load_library(f"tlie_attn_decode_d{head_dim}_w4", ["attention_decode.cu"], {"HEAD_DIM": head_dim, "DECODE_WARPS": 4, "DECODE_STAGES": 3})
    else:
        lib = load_library(f"tlie_attn_decode_d{head_dim}", ["attention_decode.cu"], {"HEAD_DIM": head_dim})
    if not getattr(lib, "_tlie_typed", False):
        lib.tlie_decode_attention_scratch_floats.restype = c_longlong
        lib._tlie_typed = True
    return lib


def decode_splits(requests: int, kv_heads: int, max_context: int) -> int:
    """Parts the key range is cut into: at most one CTA (eight warps) per SM, at least 256 keys per part, at most 32 parts."""
    by_occupancy = max(1, sm_count() // max(1, requests * kv_heads))   # rounded down: one CTA too many is a second wave
    by_length = max(1, -(-max_context // 256))
    return max(1, min(by_occupancy, by_length, 32))


def scratch(device: torch.device, floats: int) -> torch.Tensor:
    """Scratch memory of stable address (captured graphs keep pointing at it): grown, never freed."""
    held = _scratch.setdefault(device, [])
    if not held or held[-1].numel() < floats:
        held.append(torch.zeros(max(floats, 1 << 20), dtype=torch.float32, device=device))  # zero: it starts with the merge counters
    return held[-1]


def decode_attention(qkv, pages, positions, block_table, out, q_heads: int, kv_heads: int, head_dim: int, page_size: int,
                     window: int, scale: float, splits: int, fuse_rope: bool = False, inv_freq=None, write_cache: bool = True) -> None:
    """One query token per request (row i of qkv belongs to request i) over its cached keys; bfloat16.

    ``fuse_rope``: the rows of qkv are the unrotated [q | k | v] of the new tokens; the kernel rotates q and k with
    ``inv_freq`` (None: no rotation) and, with ``write_cache``, stores the new key and value in the request's page.
    """
    ops = _ops()
    requests = qkv.shape[0]
    lib = decode_attention_library(head_dim, narrow=requests * kv_heads > sm_count())
    floats = lib.tlie_decode_attention_scratch_floats(c_int(requests), c_int(q_heads), c_int(splits))
    buffer = scratch(qkv.device, floats)
    ops._check(
        lib.tlie_decode_attention(
            ops._ptr(qkv), c_int(qkv.shape[1]), ops._ptr(pages), ops._i32(positions, "positions"), ops._i32(block_table, "block_table"),
            c_int(block_table.shape[1]), ops._ptr(out), ops._ptr(buffer), c_int(requests), c_int(q_heads), c_int(kv_heads), c_int(page_size),
            c_int(window), c_float(scale), c_int(splits), c_int(1 if fuse_rope else 0), ops._ptr(inv_freq), c_int(1 if write_cache else 0), ops._stream(),
        ),
        "decode_attention",
    )


def can_fuse_rope_into_decode(batch, qkv, head_dim: int, q_heads: int, kv_heads: int, inv_freq, rotary_dim: int) -> bool:
    """Whether a decode step's rotation and cache write can happen inside the attention kernel."""
    if batch is None or qkv.dtype != torch.bfloat16 or not batch.decode_only or qkv.shape[0] != batch.num_seqs:
        return False
    if head_dim % 16 != 0 or head_dim > 128 or q_heads // kv_heads > 16 or batch.num_seqs * kv_heads > 16384:
        return False
    return inv_freq is None or (rotary_dim == head_dim and head_dim % 32 == 0)


# --- prompt (and mixed) attention -----------------------------------------------------------------
ATTENTION_TILE_ROWS = 64       # rows of one work item of the mma.sync prompt kernel (csrc/attention_prefill.cu: PREFILL_ROWS)
ATTENTION_TC_TILE_ROWS = 128   # rows of one work item of the tensor-memory kernel (csrc/attention_prefill_tc.cu)


def leading_single_rows(q_lens: list[int]) -> int:
    """How many entries at the head of a step bring one token each (the scheduler puts the decoding requests first).  In a step
    that also carries prompt portions these rows go to the decode kernel (split keys, a CTA per part) and the work lists of the
    prompt kernels leave them out: as 1-row tiles of a prompt kernel each of them cost a whole tile's pass over its keys, and
    enough of them took the step off the tensor-memory kernel altogether."""
    lead = 0
    while lead < len(q_lens) and q_lens[lead] == 1:
        lead += 1
    return lead if lead < len(q_lens) else 0


def attention_tiles(q_lens: list[int], first_positions: list[int], seq_starts: list[int], first_entry: int = 0, end_entry: int | None = None) -> list[int]:
    """Work items of the mma.sync prompt kernel: (entry, first row) of every run of up to ATTENTION_TILE_ROWS rows of one entry."""
    tiles: list[int] = []
    for index in range(first_entry, len(q_lens) if end_entry is None else end_entry):
        for offset in range(0, q_lens[index], ATTENTION_TILE_ROWS):
            tiles += [index, seq_starts[index] + offset]
    return tiles


def _row_tiles_by_work(q_lens: list[int], first_positions: list[int], seq_starts: list[int], first_entry: int) -> list[tuple[int, int, int]]:
    """(key tiles it sees, entry, first row) of every run of ATTENTION_TC_TILE_ROWS rows, the heaviest first."""
    singles = []
    for index in range(first_entry, len(q_lens)):
        count = q_lens[index]
        for offset in range(0, count, ATTENTION_TC_TILE_ROWS):
            rows = min(ATTENTION_TC_TILE_ROWS, count - offset)
            work = -(-(first_positions[index] + offset + rows) // 64)
            singles.append((work, index, seq_starts[index] + offset))
    singles.sort(key=lambda item: -item[0])
    return singles


def paired_attention_tiles(q_lens: list[int], first_positions: list[int], seq_starts: list[int], first_entry: int = 0) -> list[int]:
    """Work items of two row tiles for the tensor-memory attention kernel: (entry, first row, entry or -1, first row) per item.

    A run of ATTENTION_TC_TILE_ROWS rows late in a long request sees many keys, an early one few.  Pairing the heaviest
    tile with the lightest, the second heaviest with the second lightest, and so on, gives every CTA about the same
    number of key tiles.  The kernel takes such items, but steps do not send them: a CTA is a chain of dependent waits,
    so twice the CTAs with half the work each are faster at every length (one request of 512 tokens at 32 heads of 64:
    15.6 us in pairs, 11.9 us as single tiles; 1,024: 25.7 / 21.1; 2,048: 42.5 / 41.2; 4,096: 139 / 129; head size 128, 2,048:
    60.9 / 54.1).  Kept for the kernel's tests and its cycle counters."""
    singles = _row_tiles_by_work(q_lens, first_positions, seq_starts, first_entry)
    flat: list[int] = []
    low, high = 0, len(singles) - 1
    while low <= high:
        _, index, row = singles[low]
        if low < high:
            _, index2, row2 = singles[high]
            flat += [index, row, index2, row2]
        else:
            flat += [index, row, -1, 0]
        low += 1
        high -= 1
    return flat


def single_attention_tiles(q_lens: list[int], first_positions: list[int], seq_starts: list[int], first_entry: int = 0) -> list[int]:
    """Work items of the tensor-memory attention kernel, a row tile each, heaviest first: (entry, first row, -1, 0) per item.  The CTAs
    are handed out in this order, so every slot that comes free takes the heaviest tile left."""
    flat: list[int] = []
    for _, index, row in _row_tiles_by_work(q_lens, first_positions, seq_starts, first_entry):
        flat += [index, row, -1, 0]
    return flat


def _register_step_plans() -> None:
    """The prompt-attention kernels' work lists travel with every step that is not pure decoding (engine.batch.register_step_plan).

    They leave out the decoding requests at the head of the step (``leading_single_rows``); ``attention_tiles_lead`` holds those as
    1-row tiles, for shapes the decode kernel does not take."""
    from ..engine.batch import StepPlan, register_step_plan

    not_decode = lambda q_lens: max(q_lens) > 1  # noqa: E731
    register_step_plan(StepPlan("attention_tiles", 2, lambda q, f, s: attention_tiles(q, f, s, leading_single_rows(q)), not_decode), replace=True)
    register_step_plan(StepPlan("attention_tiles_tc", 4, lambda q, f, s: single_attention_tiles(q, f, s, leading_single_rows(q)), not_decode), replace=True)
    register_step_plan(StepPlan("attention_tiles_lead", 2, lambda q, f, s: attention_tiles(q, f, s, 0, leading_single_rows(q)),
                                lambda q_lens: max(q_lens) > 1 and leading_single_rows(q_lens) > 0), replace=True)


_register_step_plans()


def prefill_attention(qkv, pages, tiles, seq_starts, first_positions, block_table, out, q_heads: int, kv_heads: int, head_dim: int,
                      page_size: int, window: int, scale: float) -> None:
    """Flash attention of every tile in ``tiles`` (int32 [n, 2]: request, first row; up to 128 rows each) over the paged cache; bfloat16."""
    ops = _ops()
    lib = load_library(f"tlie_attn_prefill_d{head_dim}", ["attention_prefill.cu"], {"HEAD_DIM": head_dim})
    ops._check(
        lib.tlie_prefill_attention(
            ops._ptr(qkv), c_int(qkv.shape[1]), ops._ptr(pages), ops._i32(tiles, "tiles"), c_int(tiles.shape[0]), ops._i32(seq_starts, "seq_starts"),
            ops._i32(first_positions, "first_positions"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]), ops._ptr(out),
            c_int(q_heads), c_int(kv_heads), c_int(page_size), c_int(window), c_float(scale), ops._stream(),
        ),
        "prefill_attention",
    )


use_tc_attention = True    # the tcgen05 / tensor-memory prompt attention (head size 64 or 128, pages of a multiple of 64 keys)
TC_ATTENTION_HEAD_DIMS = (64, 128)
TC_ATTENTION_MIN_ROWS_PER_TILE = 32


def tc_attention_library(sigmoid: bool = False, capped: bool = False):
    if capped and not sigmoid:
        return load_library("tlie_attn_prefill_tc_capped", ["attention_prefill_tc.cu"], {"SCORE_CAP": 1})
    if sigmoid:
        return load_library("tlie_attn_prefill_tc_sigmoid", ["attention_prefill_tc.cu"], {"SIGMOID_WEIGHTS": 1})
    return load_library("tlie_attn_prefill_tc", ["attention_prefill_tc.cu"])


def tc_attention_tiles(batch, head_dim: int | None, page_size: int, lead: int):
    """The step's row tiles for the tensor-memory kernel, or None if the step or the sizes are not for it (``lead``: the single rows at the
    step's head, which the tiles leave out; ``head_dim`` None: the widths have been looked at)."""
    tiles = batch.plan("attention_tiles_tc")
    if not use_tc_attention or tiles is None or (head_dim is not None and head_dim not in TC_ATTENTION_HEAD_DIMS) or page_size % 64 != 0:
        return None
    return tiles if batch.num_tokens - lead >= TC_ATTENTION_MIN_ROWS_PER_TILE * tiles.shape[0] else None


def prefill_attention_tc(qkv, pages, tiles, seq_starts, first_positions, block_table, out, q_heads: int, kv_heads: int, head_dim: int, page_size: int,
                         window: int, scale: float, softcap: float = 0.0, sigmoid: bool = False, shifts=None, gate_offset: int = -1,
                         sinks=None) -> None:
    """Flash attention of the work items in ``tiles`` (int32 [n, 4], see ``paired_attention_tiles``) on the 5th-generation tensor cores; head size 64 or 128, bfloat16.
    ``sigmoid``, ``softcap``, ``shifts``: weights without a softmax (see ``ops.mixed_heads_attention``), a build of its own.  ``gate_offset`` >= 0: the column
    of ``qkv`` where one gate per head starts, whose sigmoid multiplies the head's output.  ``softcap`` without ``sigmoid``: a softmax over bounded scores, a build of
    its own; ``sinks`` (32-bit [heads]): exp(sink) joins the softmax's denominator."""
    ops = _ops()
    if head_dim not in TC_ATTENTION_HEAD_DIMS or page_size % 64 != 0:
        raise KernelError("the tensor-memory attention takes head sizes 64 and 128 and pages of a multiple of 64 keys", code="invalid_shape")
    lib = tc_attention_library(sigmoid, softcap > 0.0)
    gate = c_void_p(0) if gate_offset < 0 else c_void_p(qkv.data_ptr() + gate_offset * qkv.element_size())
    ops._check(
        lib.tlie_prefill_attention_tc(
            ops._ptr(qkv), c_int(qkv.shape[1]), c_int(qkv.shape[0]), ops._ptr(pages), c_int(pages.shape[0]), ops._i32(tiles, "tiles"), c_int(tiles.shape[0]),
            ops._i32(seq_starts, "seq_starts"), ops._i32(first_positions, "first_positions"), ops._i32(block_table, "block_table"),
            c_int(block_table.shape[1]), ops._ptr(out), c_int(q_heads), c_int(kv_heads), c_int(head_dim), c_int(page_size), c_int(window), c_float(scale),
            c_float(softcap), ops._ptr(shifts), gate, c_int(qkv.shape[1]), ops._ptr(sinks), ops._ptr(tcgen05_error_flag(qkv.device)), ops._stream(),
        ),
        "prefill_attention_tc",
    )


def tc_planes_fit(key_dim: int, value_dim: int) -> bool:
    """Whether the tensor-memory kernel has a build for keys and values of these widths in planes of their own."""
    return key_dim % 8 == 0 and value_dim % 8 == 0 and 0 < key_dim <= 192 and 0 < value_dim <= 128


def tc_planes_library(key_dim: int, value_dim: int, capped: bool):
    """One build per (widths rounded up to whole 64-wide boxes, bounded scores or not): compiled when a model of these sizes first runs a prompt."""
    k, v = -(-key_dim // 64) * 64, -(-value_dim // 64) * 64
    defines = {"PLANES": 1, "KEY_DIM": k, "VALUE_DIM": v}
    return load_library(f"tlie_attn_prefill_tc_planes_k{k}_v{v}" + ("_capped" if capped else ""), ["attention_prefill_tc.cu"], {**defines, "SCORE_CAP": 1} if capped else defines)


def prefill_attention_tc_planes(rows, pool, planes, tiles, seq_starts, first_positions, block_table, out, heads: int, kv_heads: int, key_dim: int, value_dim: int, page_size: int,
                                scale: float, softcap: float = 0.0, gate_offset: int = -1, sinks=None) -> None:
    """``prefill_attention_tc`` for keys and values in planes of any two widths (``tc_planes_fit``): ``planes`` = (key plane, its page stride in elements, value plane, its
    page stride), ``pool`` the tensor whose first axis counts the pages.  A softmax; ``softcap``, ``sinks`` and one gate per head as there."""
    ops = _ops()
    if not tc_planes_fit(key_dim, value_dim) or page_size % 64 != 0:
        raise KernelError("the tensor-memory attention takes widths that are multiples of 8 up to 192 and 128 and pages of a multiple of 64 keys", code="invalid_shape")
    k_ptr, k_stride, v_ptr, v_stride = planes
    if k_stride % key_dim or v_stride % value_dim:
        raise KernelError("a plane's page stride is whole rows", code="invalid_shape")
    gate = c_void_p(0) if gate_offset < 0 else c_void_p(rows.data_ptr() + gate_offset * rows.element_size())
    ops._check(
        tc_planes_library(key_dim, value_dim, softcap > 0.0).tlie_prefill_attention_tc_planes(
            ops._ptr(rows), c_int(rows.shape[1]), c_int(rows.shape[0]), k_ptr, c_int(k_stride // key_dim), v_ptr, c_int(v_stride // value_dim), c_int(pool.shape[0]), ops._i32(tiles, "tiles"),
            c_int(tiles.shape[0]), ops._i32(seq_starts, "seq_starts"), ops._i32(first_positions, "first_positions"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]),
            ops._ptr(out), c_int(heads), c_int(kv_heads), c_int(key_dim), c_int(value_dim), c_int(page_size), c_int(0), c_float(scale), c_float(softcap), gate, c_int(rows.shape[1]),
            ops._ptr(sinks), ops._ptr(tcgen05_error_flag(rows.device)), ops._stream()),
        "prefill_attention_tc_planes")


def paged_attention_bf16(qkv, pages, positions, token_seq, block_table, out, q_heads, kv_heads, head_dim, page_size, window, scale, batch) -> bool:
    """Run a specialised kernel if one covers this shape; False sends the caller to the general one."""
    if batch is None or pages.dtype != torch.bfloat16:
        return False
    if batch.decode_only and qkv.shape[0] == batch.num_seqs and head_dim <= 128 and q_heads // kv_heads <= 16:
        splits = decode_splits(batch.num_seqs, kv_heads, batch.max_seq_len)
        decode_attention(qkv, pages, positions, block_table, out, q_heads, kv_heads, head_dim, page_size, window, scale, splits)
        return True
    if head_dim > 128:
        return False
    lead = leading_single_rows(batch.host_q_lens)
    if lead:   # decoding requests at the head of a step that also carries prompt portions: rows 0 .. lead - 1, one per entry
        if q_heads // kv_heads <= 16:
            decode_attention(qkv[:lead], pages, positions[:lead], block_table[:lead], out[:lead], q_heads, kv_heads, head_dim, page_size, window, scale,
                             decode_splits(lead, kv_heads, batch.max_seq_len))
        else:
            prefill_attention(qkv, pages, batch.plan("attention_tiles_lead"), batch.seq_starts, batch.first_positions, block_table, out, q_heads, kv_heads,
                              head_dim, page_size, window, scale)
    tc_tiles = tc_attention_tiles(batch, head_dim, page_size, lead)
    if tc_tiles is not None and pages.is_contiguous():
        prefill_attention_tc(qkv, pages, tc_tiles, batch.seq_starts, batch.first_positions, block_table, out, q_heads, kv_heads, head_dim, page_size, window, scale)
        return True
    tiles = batch.plan("attention_tiles")
    if tiles is not None:
        prefill_attention(qkv, pages, tiles, batch.seq_starts, batch.first_positions, block_table, out, q_heads, kv_heads,
                          head_dim, page_size, window, scale)
        return True
    return False


# --- attention with mixed heads, prompt portions on the tensor cores -----------------------------------------------------------------
use_mixed_prefill = True
MIXED_PREFILL_MIN_ROWS = 8    # a step whose longest entry has fewer rows stays on the general kernel (a tile is at least 16 rows)


def mixed_prefill_library(key_dim: int, value_dim: int, parts: int, sigmoid: bool = False, capped: bool = False):
    """The kernel set of one (key width, value width, key heads per folded query, kind of weights): compiled when a model of these sizes first runs a prompt."""
    defines = {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "PARTS": parts}
    if sigmoid:
        return load_library(f"tlie_attn_sigmoid_k{key_dim}_v{value_dim}_p{parts}", ["attention_mixed_prefill.cu"], {**defines, "SIGMOID_WEIGHTS": 1})
    if capped:
        return load_library(f"tlie_attn_capped_k{key_dim}_v{value_dim}_p{parts}", ["attention_mixed_prefill.cu"], {**defines, "SCORE_CAP": 1})
    return load_library(f"tlie_attn_mixed_k{key_dim}_v{value_dim}_p{parts}", ["attention_mixed_prefill.cu"], defines)


def mixed_prefill_takes(batch, rows, page_size: int, parts: int, key_dim: int, value_dim: int, gate_offset: int, gate_per_head: bool = False,
                        sigmoid: bool = False, capped: bool = False) -> bool:
    """Whether a step's attention with mixed heads runs on the tensor-core kernel: bfloat16, a prompt portion among the entries,
    widths that are multiples of 16, and tiles that fit shared memory (the kernel set says how many rows its tile has: 0 = none)."""
    if not use_mixed_prefill or batch is None or batch.max_q_len < MIXED_PREFILL_MIN_ROWS or rows.dtype != torch.bfloat16:
        return False
    if key_dim % 16 or value_dim % 16 or page_size % 16 or rows.shape[1] % 8 or (gate_offset >= 0 and not gate_per_head and gate_offset % 2) or batch.num_seqs > 65535:
        return False
    if ((parts * key_dim + 8) * 16 + 3 * 64 * (key_dim + 8) + (3 if parts == 1 else 2) * 64 * (value_dim + 8)) * 2 > 227 * 1024:
        return False   # not even 16 rows of folded queries fit beside the rings of keys and values
    return mixed_prefill_library(key_dim, value_dim, parts, sigmoid, capped).tlie_mixed_prefill_tile_rows() > 0


def folded_slopes(slopes, mix):
    """slope'_h = sum_g mix[h, g] slope_g: the distance bias of head h once the heads' scores are mixed.  A part works this out once
    when it is built and hands it to every call."""
    if slopes is None or mix is None:
        return slopes
    return (mix.view(slopes.numel(), -1).double() @ slopes.double()).float().contiguous()


_mixed_scratch: dict[tuple, list] = {}


def mixed_scratch(device: torch.device, elements: int, dtype: torch.dtype) -> torch.Tensor:
    """Scratch of the attention kernels with mixed heads (folded queries, the parts of rows cut over several CTAs): buffers of
    stable address, grown by adding a larger one and never freed, since a captured graph may still point at an earlier one.  Apart
    from ``scratch``, whose first words the split-key decode kernel keeps as counters."""
    held = _mixed_scratch.setdefault((device, dtype), [])
    if not held or held[-1].numel() < elements:
        held.append(torch.empty(max(elements, 1 << 20), dtype=dtype, device=device))
    return held[-1]


def mixed_prefill(rows, gate_offset: int, batch, block_table, planes, folded, mix, out, heads: int, kv_heads: int, key_dim: int, value_dim: int,
                  page_size: int, window: int, scale: float, keep_first: int = 0, gate_per_head: bool = False, softcap: float = 0.0, sigmoid: bool = False,
                  shifts=None, sinks=None) -> None:
    """Attention with mixed heads for a step that carries prompt portions (csrc/attention_mixed_prefill.cu): the mix is folded into
    the queries by a first kernel, the second is flash attention over the concatenated key heads.  ``planes``: (key plane pointer,
    its page stride in elements, value plane pointer, its page stride); ``folded``: the folded slopes (``folded_slopes``) or None.
    ``keep_first``: with a window, the keys below this position stay visible; ``gate_per_head``: the gate is one column per head.
    With nothing to fold (no mix, ``scale`` 1) the first kernel is left out and the queries are read where they are.  ``sigmoid``, ``softcap``,
    ``shifts``, ``sinks``: see ``ops.mixed_heads_attention``."""
    ops = _ops()
    parts = kv_heads if mix is not None else 1
    tokens = rows.shape[0]
    need = tokens * heads * parts * key_dim
    held = None if mix is None and scale == 1.0 else mixed_scratch(rows.device, need, torch.bfloat16)
    k_ptr, k_stride, v_ptr, v_stride = planes
    ops._check(
        mixed_prefill_library(key_dim, value_dim, parts, sigmoid, softcap > 0.0).tlie_mixed_prefill(
            ops._ptr(rows), c_int(rows.shape[1]), c_int(gate_offset), ops._ptr(mix), c_float(scale), ops._ptr(held), k_ptr, c_longlong(k_stride), v_ptr,
            c_longlong(v_stride), ops._i32(batch.seq_starts, "seq_starts"), ops._i32(batch.first_positions, "first_positions"), ops._i32(block_table, "block_table"),
            c_int(block_table.shape[1]), ops._ptr(folded), ops._ptr(out), c_int(tokens), c_int(batch.num_seqs), c_int(batch.max_q_len),
            c_int(heads), c_int(kv_heads), c_int(page_size), c_int(window), c_int(keep_first), c_int(1 if gate_per_head else 0), c_float(softcap),
            ops._ptr(shifts), ops._ptr(sinks), ops._stream()),
        "mixed_prefill")
    ops.launch_count += 0 if held is None else 1   # two kernels: the fold and the attention


# --- latent attention, prompt portions on the tensor cores -----------------------------------------------------------------------------
use_latent_prefill = True
LATENT_PREFILL_MIN_ROWS = 1    # the longest entry's tokens from which a step runs on the tensor-core kernel (steps of single tokens split their keys)


def latent_prefill_library(key_dim: int, value_dim: int):
    """The kernel set of one (cached row width, value width): compiled when a model of these sizes first runs a prompt portion."""
    return load_library(f"tlie_attn_latent_k{key_dim}_v{value_dim}", ["attention_latent_prefill.cu"], {"KEY_DIM": key_dim, "VALUE_DIM": value_dim})


def latent_prefill_takes(batch, queries, key_dim: int, value_dim: int) -> bool:
    """Whether attention over one cached row per token (values inside the keys) runs on the tensor-core kernel: bfloat16, a prompt
    portion among the entries, a row width that is a multiple of 16 and a value width that is a multiple of 32 and at most 512 (a warp keeps
    16 x value width / 2 accumulators in registers), tiles that fit."""
    if not use_latent_prefill or batch is None or batch.max_q_len < LATENT_PREFILL_MIN_ROWS or queries.dtype != torch.bfloat16:
        return False
    if key_dim % 16 or value_dim % 32 or value_dim > key_dim or value_dim > 512 or batch.num_seqs > 65535 or (64 + 2 * 32) * (key_dim + 8) * 2 > 227 * 1024:
        return False
    return latent_prefill_library(key_dim, value_dim).tlie_latent_prefill_fits() == 1


def latent_prefill(queries, batch, block_table, pages_ptr, page_stride: int, sinks, out, heads: int, key_dim: int, value_dim: int, page_size: int, scale: float) -> None:
    """Causal attention of ``heads`` query heads per token over one cached row per token whose first ``value_dim`` columns are the
    values (csrc/attention_latent_prefill.cu).  ``queries`` [T, heads * key_dim], ``out`` [T, heads * value_dim].  A step whose CTAs
    would leave most SMs empty (few rows per request) deals every row tile's keys to several CTAs, down to four
    tiles of 32 keys each, and merges the parts with the general kernel's merge.  Steps of single tokens run on a kernel whose rows are
    a token's heads, the keys dealt to as many CTAs as there are SMs, down to a tile of 64 keys each."""
    ops = _ops()
    tokens = queries.shape[0]
    if batch.max_q_len == 1 and latent_prefill_library(key_dim, value_dim).tlie_latent_decode_fits() == 1:
        splits = max(1, min(sm_count() // (tokens * -(-heads // 16)), -(-batch.max_seq_len // 64), 64))
        partial = mixed_scratch(queries.device, tokens * splits * (heads * value_dim + 2 * heads), torch.float32) if splits > 1 else None
        ops._check(
            latent_prefill_library(key_dim, value_dim).tlie_latent_decode(
                ops._ptr(queries), pages_ptr, c_longlong(page_stride), ops._i32(batch.first_positions, "first_positions"), ops._i32(block_table, "block_table"),
                c_int(block_table.shape[1]), ops._ptr(sinks), ops._ptr(out), c_int(tokens), c_int(heads), c_int(page_size), c_float(scale), c_int(splits), ops._ptr(partial),
                ops._stream()),
            "latent_decode")
        if splits > 1:
            ops._check(ops.mixed_attention().tlie_merge_parts(ops._ptr(partial), ops._ptr(out), c_int(tokens), c_int(heads), c_int(value_dim), c_int(splits), ops._ptr(sinks),
                                                              ops._stream()), "merge_parts")
        return
    row_tiles = -(-batch.max_q_len * heads // 64) * batch.num_seqs
    splits, partial = 1, None
    if 2 * row_tiles <= sm_count():
        splits = max(1, min(sm_count() // row_tiles, -(-batch.max_seq_len // 128), 64))
    if splits > 1:
        partial = mixed_scratch(queries.device, tokens * splits * (heads * value_dim + 2 * heads), torch.float32)
    ops._check(
        latent_prefill_library(key_dim, value_dim).tlie_latent_prefill(
            ops._ptr(queries), pages_ptr, c_longlong(page_stride), ops._i32(batch.seq_starts, "seq_starts"), ops._i32(batch.first_positions, "first_positions"),
            ops._i32(block_table, "block_table"), c_int(block_table.shape[1]), ops._ptr(sinks), ops._ptr(out), c_int(queries.shape[0]), c_int(batch.num_seqs),
            c_int(batch.max_q_len), c_int(heads), c_int(page_size), c_float(scale), c_int(splits), ops._ptr(partial), ops._stream()),
        "latent_prefill")
    if splits > 1:
        ops._check(ops.mixed_attention().tlie_merge_parts(ops._ptr(partial), ops._ptr(out), c_int(tokens), c_int(heads), c_int(value_dim), c_int(splits), ops._ptr(sinks),
                                                          ops._stream()), "merge_parts")


# --- latent attention with its keys and values expanded, for steps that begin their requests -------------------------------------------
use_latent_rows = True


def latent_rows_library(key_dim: int, rot: int, value_dim: int):
    """The kernel set of one (key width, shared rotated width, value width): compiled when a model of these sizes first runs a whole prompt."""
    return load_library(f"tlie_attn_latent_rows_k{key_dim}_r{rot}_v{value_dim}", ["attention_prefill_tc.cu"],
                        {"LATENT_ROWS": 1, "KEY_DIM": key_dim, "ROT_DIM": rot, "VALUE_DIM": value_dim})


def latent_rows_fit(plain: int, rot: int, value_dim: int, dtype: torch.dtype) -> bool:
    """Whether the sizes are ones the tensor-memory kernel takes: boxes of 64 columns, keys of up to 192, values of up to 128."""
    return use_latent_rows and dtype == torch.bfloat16 and plain % 64 == 0 and rot % 64 == 0 and 0 < rot and plain + rot <= 192 and value_dim in (64, 128)


def latent_rows_tiles(batch):
    """The row tiles of a step whose every entry begins its request (no row sees a cached key, so that the step's own rows are all the
    keys there are), or None for other steps."""
    if not getattr(batch, "starts_requests", False) or leading_single_rows(batch.host_q_lens):
        return None
    tiles = batch.plan("attention_tiles_tc")
    return tiles if tiles is not None and batch.num_tokens >= TC_ATTENTION_MIN_ROWS_PER_TILE * tiles.shape[0] else None


def latent_rows(queries, expanded, shared, tiles, batch, out, heads: int, plain: int, rot: int, value_dim: int, scale: float) -> None:
    """Causal attention of every request's rows among themselves (csrc/attention_prefill_tc.cu, LATENT_ROWS): ``queries`` [T, heads (plain + rot)], ``expanded``
    [T, heads plain keys | heads value_dim values], ``shared`` [T, rot] (the key columns all heads share), ``out`` [T, heads value_dim]; bfloat16."""
    ops = _ops()
    tokens = queries.shape[0]
    if (queries.shape[1] != heads * (plain + rot) or expanded.shape != (tokens, heads * (plain + value_dim)) or shared.shape != (tokens, rot) or out.shape != (tokens, heads * value_dim)
            or not latent_rows_fit(plain, rot, value_dim, queries.dtype)):
        raise KernelError("latent_rows: queries [T, heads (plain + rot)], expanded [T, heads (plain + value_dim)], shared [T, rot], out [T, heads value_dim], bfloat16", code="invalid_shape")
    ops._check(latent_rows_library(plain + rot, rot, value_dim).tlie_prefill_attention_rows(
        ops._ptr(queries), ops._ptr(expanded), ops._ptr(shared), c_int(tokens), ops._i32(tiles, "tiles"), c_int(tiles.shape[0]), ops._i32(batch.seq_starts, "seq_starts"),
        ops._i32(batch.first_positions, "first_positions"), ops._ptr(out), c_int(heads), c_float(scale), ops._ptr(tcgen05_error_flag(queries.device)), ops._stream()), "latent_rows")


# --- attention with mixed heads, steps of few rows on the tensor cores ------------------------------------------------------------------
use_mixed_decode = True


def mixed_decode_library(key_dim: int, value_dim: int, kv_heads: int):
    """The kernel set of one (key width, value width, key/value heads of a CTA): compiled when a model of these sizes first decodes."""
    lib = load_library(f"tlie_attn_mixed_decode_k{key_dim}_v{value_dim}_g{kv_heads}", ["attention_mixed_decode.cu"],
                       {"KEY_DIM": key_dim, "VALUE_DIM": value_dim, "KV_HEADS": kv_heads})
    if not getattr(lib, "_tlie_typed", False):
        lib.tlie_mixed_decode_smem_bytes.restype = c_longlong
        lib._tlie_typed = True
    return lib


def mixed_decode_share(kv_heads: int, mixed: bool) -> int:
    """How many key/value heads one CTA of the decode kernel takes: all of them if the heads are mixed, else the largest divisor up to four (a warp each)."""
    return kv_heads if mixed else max(n for n in (1, 2, 3, 4) if kv_heads % n == 0)


def mixed_decode_takes(rows, heads: int, kv_heads: int, key_dim: int, value_dim: int, gate_offset: int, mixed: bool, gate_per_head: bool = False) -> bool:
    """Whether a step of few rows runs its attention with mixed heads on the tensor-core decode kernel: bfloat16, widths that are
    multiples of 16, at most 16 heads per key/value head, and a tile that fits shared memory."""
    if not use_mixed_decode or rows.dtype != torch.bfloat16 or key_dim % 16 or value_dim % 16 or heads // kv_heads > 16 or rows.shape[1] % 8:
        return False
    if gate_offset >= 0 and not gate_per_head and gate_offset % 2:
        return False
    share = mixed_decode_share(kv_heads, mixed)
    heads = heads // (kv_heads // share)
    fixed = 512 + share * (16 * (key_dim + 8) + 32 * (key_dim + 8) + 32 * (value_dim + 8) + 16 * 40) * 2
    return fixed + heads * 32 * 4 + (heads * heads * 4 if mixed else 0) + 3 * heads * 4 + 16 <= 200 * 1024


def mixed_decode(rows, gate_offset: int, positions, token_seq, block_table, planes, slopes, mix, out, heads: int, kv_heads: int, key_dim: int, value_dim: int,
                 page_size: int, window: int, scale: float, splits: int, keep_first: int = 0, gate_per_head: bool = False, softcap: float = 0.0,
                 sigmoid: bool = False, shifts=None, sinks=None) -> None:
    """Attention with mixed heads for a step of few rows (csrc/attention_mixed_decode.cu).  ``planes`` as in ``mixed_prefill``;
    ``splits``: CTAs that share a row's key tiles (their parts are merged by a second kernel)."""
    ops = _ops()
    tokens = rows.shape[0]
    partial = mixed_scratch(rows.device, tokens * splits * (heads * value_dim + 2 * heads), torch.float32) if splits > 1 else None
    k_ptr, k_stride, v_ptr, v_stride = planes
    ops._check(
        mixed_decode_library(key_dim, value_dim, mixed_decode_share(kv_heads, mix is not None)).tlie_mixed_decode(
            ops._ptr(rows), c_int(rows.shape[1]), c_int(gate_offset), k_ptr, c_longlong(k_stride), v_ptr, c_longlong(v_stride), ops._i32(positions, "positions"),
            ops._i32(token_seq, "token_seq"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]), ops._ptr(slopes), ops._ptr(mix), ops._ptr(out),
            c_int(tokens), c_int(heads), c_int(kv_heads), c_int(page_size), c_int(window), c_float(scale), c_int(splits), ops._ptr(partial), c_int(keep_first),
            c_int(1 if gate_per_head else 0), c_float(softcap), c_int(1 if sigmoid else 0), ops._ptr(shifts), ops._ptr(sinks), ops._stream()),
        "mixed_decode")


# --- softmax attention of single rows, heads unmixed, planes of any two widths --------------------------------------------------------
use_heads_decode = True


def heads_decode_library(key_dim: int, value_dim: int):
    """The kernel set of one pair of widths: compiled when a model of these sizes first decodes."""
    lib = load_library(f"tlie_attn_heads_decode_k{key_dim}_v{value_dim}", ["attention_heads_decode.cu"], {"KEY_DIM": key_dim, "VALUE_DIM": value_dim})
    if not getattr(lib, "_tlie_typed", False):
        lib.tlie_heads_decode_scratch_floats.restype = c_longlong
        lib._tlie_typed = True
    return lib


def heads_decode_takes(rows, page_size: int, heads: int, kv_heads: int, key_dim: int, value_dim: int) -> bool:
    """Whether a step of few rows per request runs its (unmixed, unwindowed) softmax attention on csrc/attention_heads_decode.cu."""
    return (use_heads_decode and rows.dtype == torch.bfloat16 and key_dim % 16 == 0 and value_dim % 16 == 0 and key_dim <= 256 and value_dim <= 128 and heads // kv_heads <= 16
            and rows.stride(0) % 2 == 0 and page_size % 16 == 0 and rows.shape[0] * kv_heads <= 16384)


def heads_decode(rows, gate_offset: int, gate_per_head: bool, positions, token_seq, block_table, planes, out, heads: int, kv_heads: int, key_dim: int, value_dim: int, page_size: int,
                 scale: float, softcap: float, sinks, max_seq_len: int) -> None:
    """Every row of ``rows`` over its request's keys up to its own position; ``planes`` as in ``mixed_prefill``.  A row's keys are dealt to several CTAs where there are
    fewer (row, key/value head) pairs than SMs."""
    ops = _ops()
    tokens = rows.shape[0]
    lib = heads_decode_library(key_dim, value_dim)
    splits = decode_splits(tokens, kv_heads, max_seq_len)
    buffer = scratch(rows.device, lib.tlie_heads_decode_scratch_floats(c_int(tokens), c_int(heads), c_int(splits)))
    k_ptr, k_stride, v_ptr, v_stride = planes
    ops._check(
        lib.tlie_heads_decode(
            ops._ptr(rows), c_int(rows.stride(0)), c_int(gate_offset), c_int(1 if gate_per_head else 0), k_ptr, c_longlong(k_stride), v_ptr, c_longlong(v_stride),
            ops._i32(positions, "positions"), ops._i32(token_seq, "token_seq"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]), ops._ptr(out), ops._ptr(buffer),
            c_int(tokens), c_int(heads), c_int(kv_heads), c_int(page_size), c_float(scale), c_float(softcap), ops._ptr(sinks), c_int(splits), ops._stream()),
        "heads_decode")


if os.environ.get("TLIE_SKINNY", "0") == "1":
    enable_skinny(True)


# --- scratch by name ---------------------------------------------------------------------------
_named_scratch: dict = {}


def named_scratch(device: torch.device, name: str, elements: int, dtype: torch.dtype) -> torch.Tensor:
    """Scratch that several kernels of one step hold at the same time, one buffer per name: of stable address, grown by adding a larger
    one and never freed, since a captured graph may still point at an earlier one."""
    held = _named_scratch.setdefault((device, name, dtype), [])
    if not held or held[-1].numel() < elements:
        held.append(torch.empty(max(elements, 1 << 16), dtype=dtype, device=device))
    return held[-1][:elements]


# --- differential attention on the tensor cores ---------------------------------------------------
use_diff_prefill = True
DIFF_PREFILL_MIN_ROWS = 8    # a step whose longest entry has fewer rows stays on the general kernel, which cuts a row's keys into runs


def diff_prefill_library(dim: int, vdim: int):
    """The kernel set of one (key width, value width): compiled when a model of these sizes first runs a prompt portion."""
    return load_library(f"tlie_attn_diff_k{dim}_v{vdim}", ["attention_diff_prefill.cu"], {"KEY_DIM": dim, "VALUE_DIM": vdim})


def diff_prefill_takes(batch, rows, page_size: int, dim: int, vdim: int) -> bool:
    """Whether a step's differential attention runs on the tensor-core kernel: bfloat16, a prompt portion among the entries, widths
    that are multiples of 16, and a tile that fits shared memory (the kernel set says how many rows its tile has: 0 = none)."""
    if not use_diff_prefill or batch is None or batch.max_q_len < DIFF_PREFILL_MIN_ROWS or rows.dtype != torch.bfloat16:
        return False
    if dim % 16 or vdim % 16 or page_size % 16 or rows.shape[1] % 8 or batch.num_seqs > 65535:
        return False
    if ((2 * dim + 8) * 16 + 2 * (2 * 64 * (dim + 8) + 64 * (vdim + 8))) * 2 > 227 * 1024:
        return False   # not even 16 rows of queries fit beside two stages of keys and values
    return diff_prefill_library(dim, vdim).tlie_diff_prefill_tile_rows() > 0


def diff_prefill(rows, batch, block_table, planes, out, heads: int, kv_heads: int, dim: int, vdim: int, page_size: int, scale: float, lam: float, eps: float,
                 out_scale: float) -> None:
    """Differential attention for a step that carries prompt portions (csrc/attention_diff_prefill.cu).  ``planes``: (key plane, its page
    stride in elements, value plane, its page stride)."""
    ops = _ops()
    k_pages, k_stride, v_pages, v_stride = planes
    ops._check(
        diff_prefill_library(dim, vdim).tlie_diff_prefill(
            ops._ptr(rows), c_int(rows.shape[1]), ops._ptr(k_pages), c_longlong(k_stride), ops._ptr(v_pages), c_longlong(v_stride), ops._i32(batch.seq_starts, "seq_starts"),
            ops._i32(batch.first_positions, "first_positions"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]), ops._ptr(out), c_int(rows.shape[0]),
            c_int(batch.num_seqs), c_int(batch.max_q_len), c_int(heads), c_int(kv_heads), c_int(page_size), c_float(scale), c_float(lam), c_float(eps), c_float(out_scale),
            ops._stream()),
        "diff_prefill")


use_diff_decode = True


def diff_decode_takes(rows, page_size: int, dim: int, vdim: int) -> bool:
    """Whether a step of few rows per entry (decoded tokens, portions shorter than ``DIFF_PREFILL_MIN_ROWS``) runs its differential
    attention on the tensor-core kernel whose rows are a token's heads: bfloat16, widths that are multiples of 16, a warp's tile of
    keys and values within shared memory (the kernel set says how many warps a CTA has: 0 = none)."""
    if not use_diff_decode or rows.dtype != torch.bfloat16 or dim % 16 or vdim % 16 or vdim > 256 or page_size % 16 or rows.shape[1] % 8:
        return False
    if (16 * (2 * dim + 8) + 2 * 64 * (dim + 8) + 64 * (vdim + 8)) * 2 > 227 * 1024:
        return False
    return diff_prefill_library(dim, vdim).tlie_diff_decode_warps() > 0


def diff_decode(rows, positions, token_seq, block_table, planes, out, heads: int, kv_heads: int, dim: int, vdim: int, page_size: int, scale: float, lam: float,
                eps: float, out_scale: float, longest: int) -> None:
    """Differential attention for a step of few rows per entry: per token, the heads of a key/value head are the rows of the
    products and every warp takes tiles of 64 keys of its own; the parts are joined, subtracted and normalised by the general
    kernel set's merge.  ``longest``: the most keys any row sees, from which the CTAs along the keys are chosen."""
    ops = _ops()
    tokens = rows.shape[0]
    lib = diff_prefill_library(dim, vdim)
    chunks = -(-(heads // kv_heads) // 16)
    tiles = max(1, -(-longest // 64))
    # one wave: as many CTAs along the keys as are resident together (a CTA holds the queries and two stages of a tile of both maps' keys
    # and the values); a CTA with several tiles fetches the next one under the products of this one
    smem = (16 * (2 * dim + 8) + 2 * (2 * 64 * (dim + 8) + 64 * (vdim + 8))) * 2 + 1024
    resident = sm_count() * max(1, min(227 * 1024 // smem, 16))
    ctas = max(1, min(tiles, resident // max(1, tokens * kv_heads * chunks), 64))
    runs = ctas
    parts = mixed_scratch(rows.device, tokens * runs * 2 * heads * (vdim + 2), torch.float32)
    k_pages, k_stride, v_pages, v_stride = planes
    ops._check(
        lib.tlie_diff_decode(ops._ptr(rows), c_int(rows.shape[1]), ops._ptr(k_pages), c_longlong(k_stride), ops._ptr(v_pages), c_longlong(v_stride),
                             ops._i32(positions, "positions"), ops._i32(token_seq, "token_seq"), ops._i32(block_table, "block_table"), c_int(block_table.shape[1]),
                             ops._ptr(parts), c_int(tokens), c_int(heads), c_int(kv_heads), c_int(page_size), c_float(scale), c_int(ctas), ops._stream()),
        "diff_decode")
    ops._check(ops.diff_attention_library().tlie_diff_merge(ops._code(rows), ops._ptr(parts), ops._ptr(out), c_int(tokens), c_int(heads), c_int(vdim), c_int(runs),
                                                            c_float(lam), c_float(eps), c_float(out_scale), ops._stream()), "diff_merge")
    ops.launch_count += 1   # two kernels


# --- routed experts on the tensor cores -------------------------------------------------------------
use_moe_grouped = True
MOE_GROUPED_MIN_ROWS = 17     # steps of up to 16 rows read each chosen expert's rows directly, as the other small-step products do
MOE_GROUPED_MIN_SLOTS = 64    # (token, expert) pairs from which sorting them by expert pays
use_moe_tc = True
MOE_TC_MIN_ROWS_PER_EXPERT = 48   # mean rows per expert from which tiles of 128 rows per expert (half of them padding, at worst) beat tiles of 64 on mma.sync


def moe_grouped_takes(tokens: int, top: int, width: int, ff: int, experts: int) -> bool:
    """Whether a step's routed experts run as products per expert over the sorted (token, expert) pairs (csrc/moe_grouped.cu)."""
    return use_moe_grouped and tokens >= MOE_GROUPED_MIN_ROWS and tokens * top >= MOE_GROUPED_MIN_SLOTS and width % 8 == 0 and ff % 8 == 0 and experts <= 4096


def moe_grouped(x, gate_up, down, ids, weights, shared, out, kind: int, weight_input: bool = False, shared_gate=None, clamp=None) -> None:
    ops = _ops()
    clamp = tuple(c_float(float(v)) for v in clamp or (0.0, 0.0, 0.0))
    tokens, width = x.shape
    experts, _, ff = down.shape
    top = ids.shape[1]
    slots = tokens * top
    device = x.device
    if use_moe_tc and slots >= MOE_TC_MIN_ROWS_PER_EXPERT * experts and width >= 64 and ff >= 64:   # a TMA box is 64 numbers of a row
        # every expert's rows padded to tiles of 128: the TMA / tcgen05 kernel (csrc/moe_grouped_tc.cu)
        max_rows = (slots // 128 + experts) * 128
        row_of_slot = named_scratch(device, "moe_row_of_slot", slots, torch.int32)
        token_of_row = named_scratch(device, "moe_token_of_row", max_rows, torch.int32)
        meta = named_scratch(device, "moe_tile_expert", 1 + max_rows // 128, torch.int32)
        xs = named_scratch(device, "moe_rows", max_rows * width, torch.bfloat16)
        act = named_scratch(device, "moe_act", max_rows * ff, torch.bfloat16)
        y = named_scratch(device, "moe_by_row", max_rows * width, torch.float32)
        ops._check(ops.moe_library().tlie_moe_grouped_tc(ops._ptr(x), ops._ptr(gate_up), ops._ptr(down), ops._ptr(ids), ops._ptr(weights), ops._ptr(shared), ops._ptr(shared_gate),
                                                         ops._ptr(row_of_slot),
                                                         ops._ptr(token_of_row), ops._ptr(meta), ops._ptr(xs), ops._ptr(act), ops._ptr(y), ops._ptr(out), c_int(tokens), c_int(width),
                                                         c_int(ff), c_int(experts), c_int(top), c_int(kind), c_int(1 if weight_input else 0), *clamp, ops._ptr(tcgen05_error_flag(device)), ops._stream()), "moe_grouped_tc")
        ops.launch_count += 4   # five kernels: the layout, the gathered rows, two products over all experts, the sum
        return
    sorted_slots = named_scratch(device, "moe_sorted", slots, torch.int32)
    meta = named_scratch(device, "moe_tiles", 1 + 3 * (slots // 64 + experts), torch.int32)
    act = named_scratch(device, "moe_act", slots * ff, torch.bfloat16)
    y = named_scratch(device, "moe_by_slot", slots * width, torch.float32)
    ops._check(ops.moe_library().tlie_moe_grouped(ops._ptr(x), ops._ptr(gate_up), ops._ptr(down), ops._ptr(ids), ops._ptr(weights), ops._ptr(shared), ops._ptr(shared_gate), ops._ptr(sorted_slots),
                                                  ops._ptr(meta), ops._ptr(act), ops._ptr(y), ops._ptr(out), c_int(tokens), c_int(width), c_int(ff), c_int(experts), c_int(top),
                                                  c_int(kind), c_int(1 if weight_input else 0), *clamp, ops._stream()), "moe_grouped")
    ops.launch_count += 3   # four kernels: the sort, two products per expert, the sum
