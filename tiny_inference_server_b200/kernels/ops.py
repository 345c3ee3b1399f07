"""The device operations of the engine: thin wrappers over the ``extern "C"`` launchers
of the CUDA library.  There is one implementation of each operation and no fallback:
without a CUDA device, nvcc-built library and sm_100-class GPU the first call raises.

Conventions: tensors are contiguous CUDA tensors; ``T`` is the compute dtype (bfloat16
or float32); the residual stream, norm scales, rotary tables and logits are float32;
integer metadata is int32.  Launches go to torch's current CUDA stream.
"""
from __future__ import annotations

import collections
import ctypes
import math
import os
from typing import Optional

import torch

from . import build as _build

_lib = None
ABI_VERSION = 13
#: launches of this library's kernels so far (library matrix products are not counted)
launches = 0
#: calls by kind, for tests that must know which kernel a product or an attention went to
#: ("gemm_skinny", "gemm_tc", "gemm_library", "attn_tc", "attn_keys", "attn_rows", ...)
calls: "collections.Counter[str]" = collections.Counter()


class KernelError(RuntimeError):
    pass


def library():
    """Load (building at the first call) the CUDA library; raise if that is impossible."""
    global _lib
    if _lib is not None:
        return _lib
    if not torch.cuda.is_available():
        raise KernelError("no CUDA device: this engine runs on hand-written sm_100a kernels only and has no "
                          "CPU path")
    major, _minor = torch.cuda.get_device_capability()
    if major != 10:
        raise KernelError(f"the kernels are built for sm_100a (B200); this device is sm_{major}{_minor}")
    path = _build.build()
    lib = ctypes.CDLL(path)
    lib.tis_last_error.restype = ctypes.c_char_p
    lib.tis_abi_version.restype = ctypes.c_int
    if lib.tis_abi_version() != ABI_VERSION:
        raise KernelError(f"{path}: launcher interface {lib.tis_abi_version()}, expected {ABI_VERSION}")
    _lib = lib
    return lib


def is_loaded() -> bool:
    return _lib is not None


def _check(status: int, lib) -> None:
    global launches
    if status != 0:
        raise KernelError(lib.tis_last_error().decode())
    launches += 1


def _dt(t: torch.Tensor) -> int:
    if t.dtype == torch.float32:
        return 0
    if t.dtype == torch.bfloat16:
        return 1
    raise KernelError(f"unsupported dtype {t.dtype}")


def _p(t: Optional[torch.Tensor]):
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def _stream():
    """torch's current CUDA stream as a raw handle (the direct getter is 40 times cheaper than going
    through a Stream object, and this runs once per launch)."""
    if _raw_stream is not None:
        return ctypes.c_void_p(_raw_stream(torch.cuda.current_device()))
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def _f(x: float):
    return ctypes.c_float(x)


# ---------------------------------------------------------------------------------------
# matrix products (library GEMMs, as upstream uses for every projection:
# main_models_new.py:20,29,226)
# ---------------------------------------------------------------------------------------

#: rows up to which bfloat16 products go to the weight-streaming kernels of this library instead of the library
#: product (and up to which a step's norms are folded into them).  Measured inside the decode step of the 0.9B model
#: on a B200, ms a step with the limit at 8 / 16: batch 10 1.467 / 1.387, batch 12 1.491 / 1.397, batch 16
#: 1.544 / 1.437; at 16 / 32: batch 24 2.045 / 1.986, batch 32 2.132 / 2.068; at 64 rows the library wins by far
#: (batch 64: 3.02 against 4.22 ms).  (Before the reductions of these kernels were pushed and the norms folded in,
#: the library won from 9 rows, and before that from 5.)  TIS_SKINNY_MAX_ROWS in the environment overrides it
#: (0 sends everything to the library; the kernels themselves take up to 64 rows).
SKINNY_MAX_ROWS = int(os.environ.get("TIS_SKINNY_MAX_ROWS", "32"))
#: the gate/up product with the gating in its epilogue saves a launch and the round trip of the
#: ungated product: the kernel keeps it up to more rows (measured alone at 8 rows: 8.4 us against 9.1 us
#: for the library product plus the gating kernel; inside the decode step at batch 8: 5123 -> 5207 tok/s)
SKINNY_SWIGLU_MAX_ROWS = int(os.environ.get("TIS_SKINNY_SWIGLU_MAX_ROWS", "16"))
#: above that and up to this many rows the gate/up product with the gating goes to the tcgen05 kernel with swapped
#: operands (csrc/gemm_swap.cu).  Measured alone at the 0.9B shapes: 9.9 us at 32 rows and 11.7 us at 64, against 10.4 and
#: 10.6 us for the library product, which still needs the gating kernel (~2.5 us) after it; the plain products of these
#: row counts stay with the library (qkv at 64 rows: 4.6 us against 7.8).  Inside the decode step of the 0.9B model:
#: batch 24 2.022 -> 2.012 ms, batch 32 2.135 -> 2.119, batch 64 3.052 -> 3.078, so it is used up to 32 rows.
#: TIS_SWAP_SWIGLU_MAX_ROWS overrides (0: never).
SWAP_SWIGLU_MAX_ROWS = int(os.environ.get("TIS_SWAP_SWIGLU_MAX_ROWS", "32"))
EPI_STORE, EPI_SWIGLU, EPI_RESIDUAL = 0, 1, 2
#: a store through an activation, by the activation's name (the weight-streaming products)
EPI_ACT = {"relu2": 3, "gelu_tanh": 4, "silu": 5}
#: the last of several products in one launch (``gemm_side_by_side``) may also pass tanh
EPI_GROUP_ACT = dict(EPI_ACT, tanh=6)
#: the norm between two weight-streaming products is folded into them (``ResidualSink`` / ``ScaledRows``);
#: TIS_FUSED_NORM=0 keeps the norm kernel
FUSED_NORM = os.environ.get("TIS_FUSED_NORM", "1") != "0"


class GateForm(ctypes.Structure):
    """What a gated unit does with a gate g and an up value u: ``g' * sigmoid(g' * (c1 + c3 * g'^2)) * (u' + shift)`` with
    ``g' = min(g, limit)`` and ``u' = min(max(u, -limit), limit)`` (``csrc/common.cuh``)."""

    _fields_ = [("limit", ctypes.c_float), ("c1", ctypes.c_float), ("c3", ctypes.c_float), ("shift", ctypes.c_float)]


def gate_silu() -> GateForm:
    """``silu(g) * u``"""
    return GateForm(math.inf, 1.0, 0.0, 0.0)


def gate_gelu_tanh() -> GateForm:
    """``gelu(g) * u`` with gelu in its tanh form (``0.5 (1 + tanh(y)) = sigmoid(2 y)``)"""
    c = 2.0 * math.sqrt(2.0 / math.pi)
    return GateForm(math.inf, c, 0.044715 * c, 0.0)


def gate_clamped(limit: float, alpha: float = 1.702, shift: float = 1.0) -> GateForm:
    """``g' * sigmoid(alpha * g') * (u' + shift)``, the gate bounded above by ``limit``, the up value on both sides"""
    return GateForm(limit, alpha, 0.0, shift)


SILU = gate_silu()

#: the factor a norm multiplies a row with, as a function of the row's sum of squares s over a width d:
#: "l2_eps": sqrt(d) / (sqrt(s) + eps) (eps added to the L2 norm); "mean_eps": rsqrt(s / d + eps); "none": 1 (the row kernels
#: only: the stream as it is, in the type of the products)
NORM_KINDS = {"l2_eps": 0, "mean_eps": 1, "none": 2}


class ResidualSink:
    """Where a product adds its result itself: the float32 residual stream ``values`` (n, d); it then also
    leaves the stream times ``weight`` (the weight of the norm that reads the stream next) and partial sums of
    squares, so that the norm's factor per row (``kind``, one of ``NORM_KINDS``) can be applied after the next
    product instead of before it.  ``norm`` is whoever made the sink (the reader checks it is the same norm)."""

    def __init__(self, values: torch.Tensor, weight: torch.Tensor, eps: float, norm=None, kind: str = "l2_eps"):
        if kind not in NORM_KINDS or kind == "none":
            raise KernelError(f"norm factor {kind!r}: the products know {sorted(NORM_KINDS)}")
        self.values, self.weight, self.eps, self.norm, self.kind = values, weight, float(eps), norm, kind


class ScaledRows:
    """Rows of a norm's output that still lack the factor of their row: ``rows`` (n, d) bfloat16 = stream *
    norm weight, ``parts`` (n, T) float32 = partial sums of squares of the stream.  Row r of the norm's
    output is ``rows[r]`` times the factor of ``kind`` (``NORM_KINDS``) at ``parts[r].sum()``; a weight-streaming
    product applies the factor to its own result (``gemm`` and ``gemm_swiglu`` take these rows), ``dense()`` makes
    the rows whole."""

    def __init__(self, rows: torch.Tensor, parts: torch.Tensor, eps: float, norm=None, kind: str = "l2_eps"):
        self.rows, self.parts, self.eps, self.norm, self.kind = rows, parts, float(eps), norm, kind

    @property
    def shape(self):
        return self.rows.shape

    @property
    def dtype(self):
        return self.rows.dtype

    def dense(self) -> torch.Tensor:
        lib = library()
        n, d = self.rows.shape
        out = torch.empty_like(self.rows)
        calls["scale_rows"] += 1
        _check(lib.tis_scale_rows(_p(self.rows), self.rows.stride(0), _p(self.parts), self.parts.shape[1], _f(self.eps),
                                  NORM_KINDS[self.kind], _p(out), out.stride(0), n, d, _stream()), lib)
        return out


def sink_usable(values: torch.Tensor, dtype: torch.dtype) -> bool:
    """Whether a step of these rows can fold its norms into the products around them: bfloat16 products of
    few enough rows that they all go to the weight-streaming kernels."""
    n, d = values.shape
    return (FUSED_NORM and dtype == torch.bfloat16 and 0 < n <= SKINNY_MAX_ROWS and d % 8 == 0
            and values.stride(1) == 1 and values.stride(0) % 2 == 0)


def _skinny_ok(a: torch.Tensor, w: torch.Tensor, max_rows: Optional[int] = None) -> bool:
    return (a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16
            and 0 < a.shape[0] <= (SKINNY_MAX_ROWS if max_rows is None else max_rows)
            and w.stride(1) == 1 and a.stride(1) == 1 and a.shape[1] % 8 == 0 and w.shape[1] % 8 == 0
            and a.stride(0) % 8 == 0 and w.stride(0) % 8 == 0)


#: The ring kernel wins where a CTA's share of K is short: up to RING_MAX_TILES tiles of 64 rows.  With longer
#: shares (the products of larger models) the loop is what counts, and the TMA-fed tcgen05 kernel with swapped
#: operands streams better.  Measured alone on a B200 at 1..8 rows, us ring / library / swapped: 3B-sized model
#: (width 3072, ffn 8192) qkv (12 tiles a CTA) 11.2 / 7.3 / 9.8, o (6) 6.1 / 8.5 / 7.3, gate/up with gating (24)
#: 21.8 / 22.8 + gating / 19.0, down (16) 14.2 / 17.9 / 12.6; 8B-sized (4096, 14336) qkv (16) 14.4 / 10.0 / 12.3,
#: o (8) 8.9 / 13.5 / 9.6, gate/up (64) 57 / 40 + gating / 38, down (28) 24.4 / 22.9 / 20.9.  So: short shares to the
#: ring; long ones to the swapped kernel when the matrix is tall (K >= 2 N) or carries the gating, else to the library.
RING_MAX_TILES = int(os.environ.get("TIS_RING_MAX_TILES", "8"))


def _ring_tiles(n_cols: int, k: int) -> int:
    """Tiles of 64 rows of K that a CTA of the ring kernel walks."""
    return -(-(-(-k // _ksplit(n_cols, k))) // 64)


def _swap_ok(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, swiglu: bool = False) -> bool:
    return (a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0 and (not swiglu or w.shape[1] % 64 == 0)
            and (out is None or out.stride(1) == 1))


def _ksplit(n_cols: int, k: int) -> int:
    """CTAs that share a 64-column strip of the weights (a cluster adding up over K): as many as
    keep the grid near two CTAs per SM, each with at least 128 rows of K."""
    strips = (n_cols + 63) // 64
    ks = 8
    while ks > 1 and (strips * ks > 2 * 148 * 2 or k // ks < 128):
        ks //= 2
    return ks


#: The weight-streaming product comes in two kernels: weights copied by the threads into a ring of four
#: stages (csrc/gemm_skinny.cu), and weights ordered as TMA boxes, a CTA's whole share of K at once
#: (csrc/gemm_stream.cu).  Measured alone on a B200 at the 0.9B shapes (us at 1 / 8 / 16 rows; library beside):
#: qkv 4.1 / 4.4 / 4.6 ring, 5.2 / 5.8 / 6.3 boxes (4.8 / 4.8 / 4.5); gate/up with gating 7.6 / 8.3 / 9.1 ring,
#: 10.9 / 11.9 / 13.5 boxes; down (K 4096, 512 rows of K a CTA) 7.4 / 7.8 / 8.2 ring, 6.2 / 6.5 / 6.9 boxes
#: (7.4 / 7.4 / 7.4).  A box row is 128 bytes, one request of the TMA engine each: with many CTAs per SM the
#: engine is the bottleneck, while a long share of K gains from having all of it in flight from the start.  With
#: shares of more than one round of boxes (the 3B- and 8B-sized models: 1024 rows of K a CTA and more) the kernel
#: loses to both others (8B model at one row: 132 against 210 tok/s).  So the boxes take products whose share of
#: K per CTA is STREAM_MIN_KC..STREAM_MAX_KC rows (one full round), of at most STREAM_MAX_CTAS CTAs, up to
#: STREAM_MAX_ROWS rows of x.
STREAM_GEMM = os.environ.get("TIS_STREAM_GEMM", "1") != "0"
STREAM_MIN_KC = int(os.environ.get("TIS_STREAM_MIN_KC", "512"))
STREAM_MAX_KC = int(os.environ.get("TIS_STREAM_MAX_KC", "512"))
STREAM_MAX_CTAS = int(os.environ.get("TIS_STREAM_MAX_CTAS", "296"))
STREAM_MAX_ROWS = int(os.environ.get("TIS_STREAM_MAX_ROWS", "32"))


def _stream_pays(n: int, k: int, cols: int, ksplit: Optional[int] = None) -> bool:
    ks = ksplit or _ksplit(cols, k)
    kc = -(-k // ks)
    return (STREAM_GEMM and n <= STREAM_MAX_ROWS and STREAM_MIN_KC <= kc <= max(STREAM_MAX_KC, STREAM_MIN_KC)
            and -(-cols // 64) * ks <= STREAM_MAX_CTAS)


def _ksplit_swap(n_cols: int, k: int) -> int:
    """CTAs that share a strip of 128 columns in the tcgen05 product with swapped operands."""
    strips = (n_cols + 127) // 128
    ks = 8
    while ks > 1 and (strips * ks > 2 * 148 or k // ks < 128):
        ks //= 2
    return ks


def gemm_swap(a, w: torch.Tensor, out: Optional[torch.Tensor] = None, swiglu: bool = False,
              ksplit: Optional[int] = None, sink: Optional["ResidualSink"] = None, form: GateForm = SILU):
    """``a (n <= 64, K) @ w (K, N)`` in bfloat16 on the tcgen05 tensor cores with the operands swapped (128
    columns of ``w`` are the rows of the tile, the rows of ``a`` its narrow side); with ``swiglu`` the columns of
    ``w`` are [32 gate | 32 up] blocks and the result is (n, N/2), gated in ``form``.  ``a`` may be ``ScaledRows``; with
    ``sink`` the result is added to the residual stream and comes back as ``ScaledRows``."""
    lib = library()
    scaled = a if isinstance(a, ScaledRows) else None
    if scaled is not None:
        a = scaled.rows
    n, k = a.shape
    cols = w.shape[1]
    if not _sink_fits(sink, n, cols, out) or (sink is not None and swiglu):
        raise KernelError("gemm_swap: the sink does not fit the product")
    head, tail, result = _fused_args(scaled, sink, n, cols, a.device)
    if sink is not None:
        out = result.rows
    elif out is None:
        out = torch.empty((n, cols // 2 if swiglu else cols), dtype=a.dtype, device=a.device)
    calls["gemm_swap"] += 1
    epi = EPI_RESIDUAL if sink is not None else (EPI_SWIGLU if swiglu else EPI_STORE)
    _check(lib.tis_gemm_swap_fused(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), n, cols, k,
                                   ksplit or _ksplit_swap(cols, k), epi, form, *head, *tail, _p(tc_fault()), _stream()), lib)
    return result if sink is not None else out


def _stream_fits(n: int, k: int, ksplit: int) -> bool:
    """Whether a CTA's share of the rows (all of its share of K, in shared memory for the whole loop) and
    a round of weight boxes fit the TMA-fed kernel's shared memory."""
    kc = -(-(-(-k // ksplit)) // 64) * 64
    rows = 16 if n <= 16 else (32 if n <= 32 else 64)
    received = ksplit * -(-rows // ksplit) * 64 * 4          # partial sums pushed by the cluster
    return min(kc // 64, 8) * 8192 + rows * (kc + 8) * 2 + received + 1024 <= 224 * 1024


def _fused_args(scaled: Optional[ScaledRows], sink: Optional[ResidualSink], n: int, cols: int, device):
    """The arguments of the fused entry points after (ksplit, epi): the partial sums of the rows, and the
    sink with the tensors it fills."""
    result = None
    if scaled is not None:
        head = (_p(scaled.parts), scaled.parts.shape[1], _f(scaled.eps), scaled.rows.shape[1], NORM_KINDS[scaled.kind])
    else:
        head = (None, 0, _f(0.0), 0, 0)
    if sink is not None:
        parts = torch.empty((n, -(-cols // 64)), dtype=torch.float32, device=device)
        rows = torch.empty((n, cols), dtype=torch.bfloat16, device=device)
        result = ScaledRows(rows, parts, sink.eps, sink.norm, sink.kind)
        tail = (_p(sink.values), sink.values.stride(0), _p(sink.weight), _p(parts))
    else:
        tail = (None, 0, None, None)
    return head, tail, result


def _sink_fits(sink: Optional[ResidualSink], n: int, cols: int, out) -> bool:
    return sink is None or (out is None and tuple(sink.values.shape) == (n, cols) and sink.weight.shape[0] == cols
                            and sink.weight.dtype == torch.float32 and sink.values.dtype == torch.float32)


def gemm_stream(a, w: torch.Tensor, out: Optional[torch.Tensor] = None, swiglu: bool = False,
                ksplit: Optional[int] = None, sink: Optional[ResidualSink] = None, act: Optional[str] = None,
                form: GateForm = SILU):
    """``a (n <= 64, K) @ w (K, N)`` in bfloat16 by the TMA-fed weight-streaming kernel; with ``swiglu``
    the columns of ``w`` are [32 gate | 32 up] blocks and the result is (n, N/2), gated in ``form``.  ``a`` may be
    ``ScaledRows``; with ``sink`` the result is added to the residual stream and comes back as ``ScaledRows``; with ``act`` (a key of
    ``EPI_ACT``; not with ``swiglu`` or ``sink``) the 32-bit sums pass that activation on their way out."""
    lib = library()
    scaled = a if isinstance(a, ScaledRows) else None
    if scaled is not None:
        a = scaled.rows
    n, k = a.shape
    cols = w.shape[1]
    if not _sink_fits(sink, n, cols, out) or (sink is not None and swiglu):
        raise KernelError("gemm_stream: the sink does not fit the product")
    head, tail, result = _fused_args(scaled, sink, n, cols, a.device)
    if sink is not None:
        out = result.rows
    elif out is None:
        out = torch.empty((n, cols // 2 if swiglu else cols), dtype=a.dtype, device=a.device)
    calls["gemm_stream"] += 1
    epi = _epilogue(sink, swiglu, act)
    _check(lib.tis_gemm_stream_fused(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), n, cols, k,
                                     ksplit or _ksplit(cols, k), epi, form, *head, *tail, _p(tc_fault()), _stream()), lib)
    return result if sink is not None else out


def _epilogue(sink, swiglu: bool, act: Optional[str]) -> int:
    if act is not None:
        if sink is not None or swiglu or act not in EPI_ACT:
            raise KernelError(f"activation epilogue {act!r}: known are {sorted(EPI_ACT)}, and not with gating or a sink")
        return EPI_ACT[act]
    return EPI_RESIDUAL if sink is not None else (EPI_SWIGLU if swiglu else EPI_STORE)


def gemm_skinny(a, w: torch.Tensor, out: Optional[torch.Tensor] = None, swiglu: bool = False,
                ksplit: Optional[int] = None, sink: Optional[ResidualSink] = None, act: Optional[str] = None,
                form: GateForm = SILU):
    """``a (n <= 64, K) @ w (K, N)`` in bfloat16 by a weight-streaming kernel; with ``swiglu``
    the columns of ``w`` are [32 gate | 32 up] blocks and the result is (n, N/2), gated in ``form``.  ``a`` may be
    ``ScaledRows``; with ``sink`` the result is added to the residual stream and comes back as ``ScaledRows``; ``act`` as in
    ``gemm_stream``."""
    rows = a.rows if isinstance(a, ScaledRows) else a
    if (_stream_pays(rows.shape[0], rows.shape[1], w.shape[1], ksplit) and rows.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0
            and _stream_fits(rows.shape[0], rows.shape[1], ksplit or _ksplit(w.shape[1], rows.shape[1]))):
        return gemm_stream(a, w, out, swiglu, ksplit, sink, act, form)
    lib = library()
    scaled = a if isinstance(a, ScaledRows) else None
    a = rows
    n, k = a.shape
    cols = w.shape[1]
    if not _sink_fits(sink, n, cols, out) or (sink is not None and swiglu):
        raise KernelError("gemm_skinny: the sink does not fit the product")
    head, tail, result = _fused_args(scaled, sink, n, cols, a.device)
    if sink is not None:
        out = result.rows
    elif out is None:
        out = torch.empty((n, cols // 2 if swiglu else cols), dtype=a.dtype, device=a.device)
    calls["gemm_skinny"] += 1
    epi = _epilogue(sink, swiglu, act)
    _check(lib.tis_gemm_skinny_fused(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), n, cols, k,
                                     ksplit or _ksplit(cols, k), epi, form, *head, *tail, _p(tc_fault()), _stream()), lib)
    return result if sink is not None else out


#: The tcgen05 kernel of this library (csrc/gemm_tc.cu) against the library product, measured on a
#: B200 at the 0.9B model's shapes (replayed from CUDA graphs, weights rotated through more than L2):
#: gate/up with the SwiGLU gating in its epilogue it wins from about 3000 rows (4096 rows: 78 against
#: 94 us for the library product plus the gating kernel; 2048 rows: 52 against 49 us); plain products
#: it loses (2048 x 1536 x 4096: 28 against 19.5 us — one CTA per tile moves more bytes from L2 per
#: multiply-add than the library's two-CTA tiles).  So by default it takes gate/up products of at
#: least TC_MIN_ROWS rows and no plain ones; TIS_TC_MIN_ROWS / TIS_TC_PLAIN_MIN_ROWS in the
#: environment override the two limits (0 = never).
TC_MIN_ROWS = int(os.environ.get("TIS_TC_MIN_ROWS", "3072"))
TC_PLAIN_MIN_ROWS = int(os.environ.get("TIS_TC_PLAIN_MIN_ROWS", "0"))
_tc_fault = None


def tc_fault() -> torch.Tensor:
    """The fault word of the tcgen05 products (non-zero after a wait inside one ran out)."""
    global _tc_fault
    if _tc_fault is None:
        _tc_fault = torch.zeros(4, dtype=torch.int32, device="cuda")
    return _tc_fault


def _tc_ok(a: torch.Tensor, w: torch.Tensor, min_rows: int) -> bool:
    return (min_rows > 0 and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16
            and a.shape[0] >= min_rows and w.stride(1) == 1 and a.stride(1) == 1
            and a.shape[1] % 8 == 0 and w.shape[1] % 8 == 0 and a.stride(0) % 8 == 0 and w.stride(0) % 8 == 0
            and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def gemm_tc(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, swiglu: bool = False,
            form: GateForm = SILU) -> torch.Tensor:
    """``a (n, K) @ w (K, N)`` in bfloat16 on the tcgen05 tensor cores (TMA-fed, accumulator in
    tensor memory); with ``swiglu`` the columns of ``w`` are [32 gate | 32 up] blocks and the
    result is (n, N/2)."""
    lib = library()
    n, k = a.shape
    cols = w.shape[1]
    if out is None:
        out = torch.empty((n, cols // 2 if swiglu else cols), dtype=a.dtype, device=a.device)
    calls["gemm_tc"] += 1
    _check(lib.tis_gemm_tc(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), n, cols, k,
                           EPI_SWIGLU if swiglu else EPI_STORE, form, _p(tc_fault()), _stream()), lib)
    return out


#: bfloat16 library products go to cuBLAS directly (the same kernels as torch.mm, a third of the host
#: time per call); TIS_LIBRARY_GEMM=torch sends them through torch.mm instead
LIBRARY_GEMM_DIRECT = os.environ.get("TIS_LIBRARY_GEMM", "direct") != "torch"
_blas_state = None          # None: not tried yet; False: unavailable; else the workspace tensor


def _blas_workspace(lib, device) -> bool:
    """Give the library its workspace at the first call; False when cuBLAS cannot be called directly."""
    global _blas_state
    if not LIBRARY_GEMM_DIRECT or _blas_state is False:
        return False
    if _blas_state is None:
        ws = torch.empty(32 << 20, dtype=torch.uint8, device=device)
        _blas_state = ws if lib.tis_gemm_library_init(_p(ws), ctypes.c_size_t(ws.numel())) else False
    return _blas_state is not False


def _library_gemm(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor], f32_out: bool) -> Optional[torch.Tensor]:
    """``a @ w`` by a direct cuBLAS call, or None when that is not possible (then torch.mm does it)."""
    global _blas_state, launches
    if not LIBRARY_GEMM_DIRECT or _blas_state is False:
        return None
    if (a.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or a.stride(1) != 1 or w.stride(1) != 1
            or a.stride(0) < a.shape[1] or w.stride(0) < w.shape[1]):
        return None
    lib = library()
    if not _blas_workspace(lib, a.device):
        return None
    n, k = a.shape
    cols = w.shape[1]
    want = torch.float32 if f32_out else torch.bfloat16
    if out is None:
        out = torch.empty((n, cols), dtype=want, device=a.device)
    elif out.dtype != want or out.stride(1) != 1 or out.stride(0) < cols:
        return None
    calls["gemm_library"] += 1
    status = lib.tis_gemm_library(_p(a), a.stride(0), _p(w), w.stride(0), _p(out), out.stride(0), n, cols, k,
                                  int(f32_out), _stream())
    if status != 0:
        raise KernelError(lib.tis_last_error().decode())
    return out


def gemm(a, w: torch.Tensor, out: Optional[torch.Tensor] = None, sink: Optional[ResidualSink] = None,
         act: Optional[str] = None):
    """``a (n, K) @ w (K, N)`` in the dtype of ``a``; float32 means true float32.  Few bfloat16
    rows go to the weight-streaming kernel of this library, many to its tcgen05 kernel,
    everything else to the library product.

    ``a`` may be ``ScaledRows``.  With ``sink``, a product that goes to a weight-streaming kernel adds its
    result to the residual stream itself and returns ``ScaledRows`` for the norm that follows; any other
    product ignores the sink and returns its result, which the caller adds as before.  With ``act`` (not with a
    sink) the result passes that activation: in the epilogue of a weight-streaming kernel, else by the activation
    kernel behind the product."""
    if act is not None:
        if sink is not None:
            raise KernelError("gemm: an activation and a sink do not go together")
        rows = a.rows if isinstance(a, ScaledRows) else a
        streams = _stream_pays(rows.shape[0], rows.shape[1], w.shape[1]) and rows.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0
        if act in EPI_ACT and ((_skinny_ok(rows, w) and (streams or _ring_tiles(w.shape[1], rows.shape[1]) <= RING_MAX_TILES)) or
                               (_skinny_ok(rows, w, STREAM_MAX_ROWS) and streams)):
            return gemm_skinny(a, w, out, act=act)
        h = gemm(a, w, out)
        return activation(h, h, act)
    scaled = a if isinstance(a, ScaledRows) else None
    if scaled is not None:
        a = scaled.rows
    if a.dtype == torch.float32 and torch.backends.cuda.matmul.allow_tf32:
        raise KernelError("float32 products must not run in TF32: torch.backends.cuda.matmul.allow_tf32 is set")
    streams = _stream_pays(a.shape[0], a.shape[1], w.shape[1]) and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0
    if (_skinny_ok(a, w) and (streams or _ring_tiles(w.shape[1], a.shape[1]) <= RING_MAX_TILES)) or \
            (_skinny_ok(a, w, STREAM_MAX_ROWS) and streams):
        if sink is not None and not _sink_fits(sink, a.shape[0], w.shape[1], out):
            sink = None
        return gemm_skinny(scaled if scaled is not None else a, w, out, sink=sink)
    if _skinny_ok(a, w) and a.shape[1] >= 2 * w.shape[1] and _swap_ok(a, w, out):
        # a long share of K per CTA and a tall matrix: the tcgen05 kernel with swapped operands
        if sink is not None and not (_sink_fits(sink, a.shape[0], w.shape[1], out) and sink.values.stride(0) % 4 == 0
                                     and sink.values.data_ptr() % 16 == 0 and sink.weight.data_ptr() % 16 == 0):
            sink = None
        return gemm_swap(scaled if scaled is not None else a, w, out, sink=sink)
    if scaled is not None:
        a = scaled.dense()
    if _tc_ok(a, w, TC_PLAIN_MIN_ROWS) and (out is None or (out.stride(1) == 1 and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0)):
        return gemm_tc(a, w, out)
    direct = _library_gemm(a, w, out, False)
    if direct is not None:
        return direct
    if out is None:
        return torch.mm(a, w)
    return torch.mm(a, w, out=out)


def gemm_swiglu(a, w_gu: torch.Tensor, hidden: int, block: int, form: GateForm = SILU) -> torch.Tensor:
    """``gated(a @ w_gu)`` in the form ``form``: (n, hidden).  ``w_gu`` (K, 2*hidden) holds gate and up columns in
    alternating blocks of ``block``.  Few bfloat16 rows with block 32: one kernel with the
    gating in its epilogue; else the product and the gating kernel.  ``a`` may be ``ScaledRows``."""
    scaled = a if isinstance(a, ScaledRows) else None
    if scaled is not None:
        a = scaled.rows
    if block == 32 and _skinny_ok(a, w_gu, SKINNY_SWIGLU_MAX_ROWS) and (
            _ring_tiles(w_gu.shape[1], a.shape[1]) <= RING_MAX_TILES or not _swap_ok(a, w_gu, swiglu=True)):
        return gemm_skinny(scaled if scaled is not None else a, w_gu, swiglu=True, form=form)
    if (block == 32 and _skinny_ok(a, w_gu, SWAP_SWIGLU_MAX_ROWS) and w_gu.shape[1] % 64 == 0
            and a.data_ptr() % 16 == 0 and w_gu.data_ptr() % 16 == 0):
        return gemm_swap(scaled if scaled is not None else a, w_gu, swiglu=True, form=form)
    if scaled is not None:
        a = scaled.dense()
    if block == 32 and _tc_ok(a, w_gu, TC_MIN_ROWS) and w_gu.shape[1] % 64 == 0:
        return gemm_tc(a, w_gu, swiglu=True, form=form)
    gu = gemm(a, w_gu)
    out = torch.empty((a.shape[0], hidden), dtype=a.dtype, device=a.device)
    return swiglu(gu, out, block, form)


def gemm_f32_out(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``a (n, K) @ w (K, N)`` with a float32 result whatever the dtype of the operands."""
    if a.dtype == torch.float32:
        return gemm(a, w)
    direct = _library_gemm(a, w, None, True)
    if direct is not None:
        return direct
    return torch.mm(a, w, out_dtype=torch.float32)


# ---------------------------------------------------------------------------------------
# row-wise kernels
# ---------------------------------------------------------------------------------------

def embed_rows(table: torch.Tensor, tokens: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    """out[r] = float(table[tokens[r]]) * scale; out is the float32 residual stream (n, d)."""
    lib = library()
    n, d = out.shape
    _check(lib.tis_embed_rows(_dt(table), _p(table), _p(tokens), _p(out), n, d, _f(scale), _stream()), lib)
    return out


def add_rmsnorm(residual: torch.Tensor, delta: Optional[torch.Tensor], scale: Optional[torch.Tensor], eps: float,
                out: Optional[torch.Tensor], kind: str = "l2_eps", delta_norm=None) -> Optional[torch.Tensor]:
    """residual += delta (when given), then out = residual * factor * scale with the row's factor of ``kind``
    (``NORM_KINDS``): sqrt(d) / (||residual|| + eps), or 1 / sqrt(mean(residual^2) + eps).  ``out`` None: only the
    sum.  ``delta_norm = (weight (d,) float32, eps, kind)``: the update passes a norm of its own on its way into the
    stream, ``residual += delta * factor(delta) * weight``, all in 32-bit."""
    lib = library()
    n, d = residual.shape
    ref = out if out is not None else delta
    dw, deps, dkind = (None, 0.0, "l2_eps") if delta_norm is None or delta is None else delta_norm
    _check(lib.tis_add_rmsnorm(_dt(ref), _p(residual), _p(delta), _p(scale), _f(eps), NORM_KINDS[kind], _p(out), n, d,
                               _p(dw), _f(deps), NORM_KINDS[dkind], _stream()), lib)
    return out


def residual_add(residual: torch.Tensor, delta: torch.Tensor) -> torch.Tensor:
    lib = library()
    n, d = residual.shape
    _check(lib.tis_residual_add(_dt(delta), _p(residual), _p(delta), n, d, _stream()), lib)
    return residual


def rope_kv_write(qkv: torch.Tensor, positions: torch.Tensor, row_slot: torch.Tensor, cos: torch.Tensor,
                  sin: torch.Tensor, plane: Optional[torch.Tensor], block_table: Optional[torch.Tensor],
                  num_heads: int, kv_heads: int, head_dim: int, page_size: int, fault: torch.Tensor,
                  interleaved: bool = False, write_kv: bool = True) -> None:
    """Rotate the queries of ``qkv`` (n, (H+2*KVH)*hd) in place; rotate the keys and write
    keys and values of every row into its page of ``plane`` [pages, 2, KVH, page, hd]."""
    lib = library()
    n = qkv.shape[0]
    rot = 2 * cos.shape[1]
    write = bool(write_kv and plane is not None)
    _check(lib.tis_rope_kv_write(
        _dt(qkv), _p(qkv), qkv.stride(0), _p(positions), _p(row_slot), _p(cos), _p(sin),
        _p(plane if write else None), _p(block_table if write else None),
        block_table.stride(0) if write else 0, plane.shape[0] if write else 0,
        n, num_heads, kv_heads, head_dim, rot, int(interleaved), page_size, int(write), _p(fault), _stream()), lib)


_attn_libs = {}

def attention_library(head_dim: int):
    """The tensor-core attention kernels for one head size, compiled when first needed."""
    lib = _attn_libs.get(head_dim)
    if lib is None:
        library()
        lib = ctypes.CDLL(_build.build_attention(head_dim))
        lib.tis_last_error.restype = ctypes.c_char_p
        lib.tis_attn_scratch_floats.restype = ctypes.c_size_t
        lib.resident = {}
        lib.tc_attention = bool(lib.tis_attn_tc_supported())
        if lib.tis_attn_head_dim() != head_dim:
            raise KernelError(f"attention library built for head size {lib.tis_attn_head_dim()}, wanted {head_dim}")
        _attn_libs[head_dim] = lib
    return lib


#: long prompt portions (tiles of up to 128 rows) go to the tcgen05 attention kernel where the head
#: size (64, 128) and the page size (16..128) allow it; TIS_TC_ATTENTION=0 keeps them on the
#: mma.sync kernel
TC_ATTENTION = os.environ.get("TIS_TC_ATTENTION", "1") != "0"
TC_ATTENTION_MIN_TILES = 2
TC_ATTENTION_SHORT_CONTEXT = 1024

#: CTAs of the attention kernels that are resident at a time when the library cannot be asked
#: (148 SMs, two CTAs each at head size 128)
ATTN_RESIDENT_CTAS = 148 * 2
#: cost of starting and finishing a CTA, and of merging one more split, in units of one 64-key tile
ATTN_CTA_OVERHEAD_TILES = 8.0
ATTN_MERGE_PER_SPLIT_TILES = 0.1
#: most key splits of a decode tile (one cluster): 16, a cluster size that the device allows on request, while
#: the CTAs of the kernel with a producer warp are all resident (two to an SM); else the portable 8.  Measured
#: inside the decode step of the 0.9B model at context 4096, 8 -> 16 splits: batch 1 1.003 -> 0.938 ms a step,
#: batch 2 1.022 -> 0.977, batch 4 1.080 -> 1.051; at batch 8 (384 CTAs) 16 splits cost (17.6 -> 28.4 us a launch).
#: TIS_ATTN_MAX_SPLITS overrides.
ATTN_MAX_SPLITS_KEYS = int(os.environ.get("TIS_ATTN_MAX_SPLITS", "16"))
ATTN_DECODE_RESIDENT_CTAS = 148 * 2


def plan_splits(num_tiles: int, kv_heads: int, max_kv: int, mode_keys: bool, resident: int = ATTN_RESIDENT_CTAS,
                min_kv: Optional[int] = None):
    """(keys per split, number of splits) for contexts of up to ``max_kv`` keys.

    One CTA walks the keys of one (tile, kv head, split), 64 at a time.  With few tiles the
    SMs idle unless the keys are split; with too many splits every CTA is all overhead.
    Tiles of a prompt see different numbers of keys (``min_kv`` .. ``max_kv``, causal): without
    splits the CTA of the last tile works long after the others are done.  The number of
    splits minimises an estimate of the time: CTAs that have keys at all, each costing
    overhead + its tiles, spread over the CTAs that are resident at a time, but never less
    than the longest CTA; plus the cost of merging."""
    total_tiles = max(1, (max_kv + 63) // 64)
    lo_tiles = total_tiles if min_kv is None else max(1, (min(min_kv, max_kv) + 63) // 64)
    # the splits are one thread-block cluster: at most 8 CTAs, or 16 for decode tiles (a cluster size
    # that the device allows on request)
    limit = min(total_tiles, ATTN_MAX_SPLITS_KEYS if mode_keys else 8)
    if not mode_keys and lo_tiles < 0.75 * total_tiles:
        # a prompt from its start: tiles see very different numbers of keys.  The CTAs of a cluster
        # leave together, so a split without keys would hold its place until the longest one is
        # done: splitting gains nothing there (measured: a 2048-token prompt gets slower).
        limit = 1
    best, best_cost = 1, None
    for s in range(1, limit + 1):
        per_tiles = (total_tiles + s - 1) // s
        if (total_tiles + per_tiles - 1) // per_tiles != s:
            continue
        if s > 8 and (s != 16 or num_tiles * kv_heads * s > ATTN_DECODE_RESIDENT_CTAS):
            continue                   # above the portable cluster size only 16, and only while all CTAs are resident
        # tiles with key counts spread evenly from lo_tiles to total_tiles
        work, ctas = 0.0, 0.0
        samples = min(num_tiles, 16)
        for i in range(samples):
            kv = lo_tiles + (total_tiles - lo_tiles) * (i + 0.5) / samples
            full, rest = divmod(kv, per_tiles)
            ctas += full + (1 if rest > 1e-9 else 0)
            work += full * (ATTN_CTA_OVERHEAD_TILES + per_tiles) + ((ATTN_CTA_OVERHEAD_TILES + rest) if rest > 1e-9 else 0)
        scale = num_tiles * kv_heads / samples
        ctas, work = ctas * scale, work * scale
        longest = ATTN_CTA_OVERHEAD_TILES + per_tiles
        if lo_tiles == total_tiles:
            # equal CTAs run in whole rounds: one CTA more than fit at a time costs a second round
            cost = math.ceil(ctas / resident - 1e-9) * longest
        else:
            cost = max(longest, work / min(resident, max(ctas, 1.0)))
        if s > 1:
            cost += ATTN_MERGE_PER_SPLIT_TILES * s
            if not mode_keys:
                cost += 1.0            # 64 rows of partial outputs go through shared memory of the cluster
        if best_cost is None or cost < best_cost - 1e-9:
            best, best_cost = s, cost
    per = ((total_tiles + best - 1) // best) * 64
    return per, max(1, (max_kv + per - 1) // per)


#: decode steps: the attention kernel rotates queries and keys and writes the cache itself
#: (TIS_ATTN_ROTARY=0: the rope_kv_write kernel does, in a launch of its own, as for every other step)
ATTN_ROTARY = os.environ.get("TIS_ATTN_ROTARY", "1") != "0"


def _window_code(window: Optional[int], chunked: bool) -> int:
    """What the attention kernels take: 0 every earlier key, W > 0 the last W, -C < 0 those of the row's chunk of C positions
    (``first_key`` in csrc/common.cuh)."""
    if not window:
        return 0
    if window < 0:
        raise KernelError(f"a window of {window} keys")
    return -int(window) if chunked else int(window)


class PairRotary:
    """A rotation of the first elements of every head, twice as many as ``cos`` and ``sin`` (positions, rot / 2; None: none)
    have columns, element 2i with 2i + 1, and (``norm_eps`` not None) the division of the head by its root mean square
    behind it: what ``paged_attention`` can do to a decode row's queries and key itself (``rotary=``)."""

    def __init__(self, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor], norm_eps: Optional[float] = None):
        self.cos, self.sin, self.norm_eps = cos, sin, norm_eps


def rotary_fusable(q: torch.Tensor, step, num_heads: int, kv_heads: int, head_dim: int, pairs: bool = False) -> bool:
    """Whether ``paged_attention`` can take rows whose queries are not rotated yet and whose keys and
    values are not in the cache yet (``rotary=``): a decode step (one row per request) in bfloat16, a head
    size the kernel rotates in registers, at most 16 query heads per kv head.  ``pairs``: the rotation is a
    ``PairRotary``, whose pairs lie in one register at any head size."""
    return (ATTN_ROTARY and q.dtype == torch.bfloat16 and step is not None and getattr(step, "decode_only", False)
            and (head_dim % 32 == 0 or pairs) and kv_heads > 0 and num_heads % kv_heads == 0 and num_heads // kv_heads <= 16)


def paged_attention(q: torch.Tensor, out: torch.Tensor, plane: torch.Tensor, block_table: torch.Tensor,
                    positions: torch.Tensor, row_slot: torch.Tensor, num_heads: int, kv_heads: int,
                    head_dim: int, page_size: int, window: Optional[int], fault: torch.Tensor,
                    step=None, rotary=None, write_kv: bool = True, scale: Optional[float] = None,
                    sink: Optional[torch.Tensor] = None, chunked: bool = False, softcap: Optional[float] = None,
                    gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of the step's rows over the cache.  ``q`` is (n, >= H*hd) with the
    queries first in each row (row stride free); ``out`` is (n, H*hd).  The row at position
    p of slot s sees keys max(0, p-window+1)..p of ``plane`` through ``block_table[s]``.

    float32: CUDA-core kernel, everything in 32-bit.  bfloat16: tensor-core kernels over
    tiles of rows (``kernels.attention_plan``), keys of long contexts split over CTAs.

    ``rotary=(cos, sin)`` (only where ``rotary_fusable``): the rows of ``q`` are the projection's output
    as it is, [queries | keys | values]; the kernel rotates queries and keys itself (half-split pairs,
    tables [positions, hd/2] float32) and, with ``write_kv``, writes the rows' keys and values into
    their pages — what ``rope_kv_write`` does in a launch of its own everywhere else.  Or ``rotary`` a ``PairRotary``:
    neighbouring elements paired, and the norm of every head (``rotate_norm_store`` everywhere else).

    ``scale`` (positive; 1 / sqrt(head_dim) unless given) multiplies the scores.  ``sink`` (H,) float32: head h's softmax
    softmax denominator also holds ``exp(sink[h])`` (unscaled; it has no key and no value).  ``chunked``: instead of the last
    ``window`` keys a row sees those of its own chunk of ``window`` positions, counted from position 0.  ``softcap`` (not with
    ``rotary``): a score s becomes ``softcap * tanh(s / softcap)``.  ``gate`` (n, H), row stride free (not with ``rotary``):
    head h's output is multiplied by ``sigmoid(gate[row, h])``."""
    lib = library()
    n = q.shape[0]
    window = _window_code(window, chunked)
    cap = float(softcap or 0.0)
    ldg = gate.stride(0) if gate is not None else 0
    if rotary is not None and (cap or gate is not None or window < 0):
        raise KernelError("paged_attention: chunks, bounded scores and gates go with rows that are rotated already")
    scale = 1.0 / math.sqrt(head_dim) if scale is None else float(scale)
    if not scale > 0:
        raise KernelError(f"paged_attention: the scores are multiplied by a positive number, not {scale}")
    pairs = isinstance(rotary, PairRotary)
    if rotary is not None and not rotary_fusable(q, step, num_heads, kv_heads, head_dim, pairs):
        raise KernelError("paged_attention: rotary encoding inside the kernel is for decode steps in bfloat16")
    if q.dtype == torch.float32:
        _check(lib.tis_paged_attention_simt(
            _dt(q), _p(q), q.stride(0), _p(out), out.stride(0), _p(plane), _p(block_table), block_table.stride(0),
            plane.shape[0], _p(positions), _p(row_slot), n, num_heads, kv_heads, head_dim, page_size,
            window, _f(scale), _f(cap), _p(gate), ldg, _p(sink), _p(fault), _stream()), lib)
        return out
    if kv_heads <= 0 or num_heads % kv_heads:
        raise KernelError(f"paged_attention: {num_heads} query heads are not a multiple of {kv_heads} kv heads")
    g = num_heads // kv_heads
    if g > 64:
        raise KernelError(f"paged_attention: {g} query heads per kv head; the bfloat16 kernels take up to 64")
    alib = attention_library(head_dim)
    min_kv = None
    from . import attention_plan
    if step is not None:
        tiles = step.plan(attention_plan.planner(g))
        max_kv = step.max_position + 1
        min_kv = getattr(step, "min_position", None)
        min_kv = None if min_kv is None else min_kv + 1
    else:
        tiles = attention_plan.infer_tiles(positions, row_slot, g)
        max_kv = int(positions.max().item()) + 1 if n else 1
    rows_tiles = tiles.rows
    # keys that the key splits share out: with a window those from the tile's first one on (a tile's rows see at most
    # 63 keys more than one of them does, and the share starts at a multiple of 64)
    split_kv = max_kv if not window else min(max_kv, abs(window) + 128)
    w0, wn, wide_count = getattr(tiles, "wide", (None, None, 0))
    # One CTA of the tcgen05 kernel walks all keys of its 128 rows (no key splits yet).  Measured at the
    # 0.9B sizes: with two or more such tiles in the step it wins (256 rows ending at 4096: 51 against
    # 84 us), a single tile deep inside a long context is faster on the mma.sync kernel, which splits
    # the keys over a cluster (128 rows ending at 4096: 51 against 34 us; ending at 1024: a tie).
    tc_pays = wide_count >= TC_ATTENTION_MIN_TILES or max_kv <= TC_ATTENTION_SHORT_CONTEXT
    if wide_count and TC_ATTENTION and tc_pays and page_size in (16, 32, 64, 128) and alib.tc_attention:
        # long portions: the tcgen05 kernel takes them as tiles of 128 rows; the others stay below
        calls["attn_tc"] += 1
        _check(alib.tis_attn_tc(_p(q), q.stride(0), n, _p(out), out.stride(0), _p(plane), _p(block_table),
                                block_table.stride(0), plane.shape[0], _p(positions), _p(row_slot), _p(w0), _p(wn),
                                wide_count, num_heads, kv_heads, page_size, window, _f(scale), _f(cap), _p(gate), ldg,
                                _p(sink), _p(fault), _stream()), alib)
        skip = tiles.rows_in_wide
        if skip == tiles.rows[2]:
            rows_tiles = (None, None, 0)
        else:
            rows_tiles = (tiles.rows[0][skip:], tiles.rows[1][skip:], tiles.rows[2] - skip)
    if rotary is not None:
        row0, rows, count = tiles.keys
        if tiles.rows[2] or wide_count or tiles.keys_max_rows != 1:
            raise KernelError("paged_attention: rotary encoding inside the kernel needs tiles of one row")
        half = int(g <= 8)
        resident = alib.resident.get((1, half))
        if resident is None:
            resident = alib.resident[(1, half)] = alib.tis_attn_resident_ctas(1, half)
        per, splits = plan_splits(count, kv_heads, split_kv, True, resident, None)
        calls["attn_keys_rotary"] += 1
        if pairs:
            cos, sin = rotary.cos, rotary.sin
            how = (2, 2 * cos.shape[1] if cos is not None else 0, int(rotary.norm_eps is not None), _f(rotary.norm_eps or 0.0))
        else:
            cos, sin = rotary
            how = (1, head_dim, 0, _f(0.0))
        if getattr(tiles, "keys_identity", False) and count == n:
            row0 = rows = None          # tile i is row i: the kernel reads no tile arrays
        _check(alib.tis_attn_decode_rope(_p(q), q.stride(0), _p(out), out.stride(0), _p(plane), _p(block_table),
                                         block_table.stride(0), plane.shape[0], _p(positions), _p(row_slot), _p(row0),
                                         _p(rows), count, n, num_heads, kv_heads, page_size, window,
                                         _f(scale), per, splits, _p(cos), _p(sin), int(bool(write_kv)), *how, _p(sink),
                                         _p(fault), _stream()), alib)
        return out
    for mode, (row0, rows, count) in ((1, tiles.keys), (0, rows_tiles)):
        if count == 0:
            continue
        max_rows = tiles.keys_max_rows if mode == 1 else 0
        half = int(mode == 1 and 0 < max_rows * g <= 8)
        resident = alib.resident.get((mode, half))
        if resident is None:
            resident = alib.resident[(mode, half)] = alib.tis_attn_resident_ctas(mode, half)
        per, splits = plan_splits(count, kv_heads, split_kv, mode == 1, resident,
                                  None if mode == 1 or min_kv is None else min(min_kv, split_kv))
        calls["attn_keys" if mode == 1 else "attn_rows"] += 1
        # at most eight splits (plan_splits): they merge inside a thread-block cluster, without scratch
        _check(alib.tis_attn_mma_sink(mode, _p(q), q.stride(0), _p(out), out.stride(0), _p(plane), _p(block_table),
                                 block_table.stride(0), plane.shape[0], _p(positions), _p(row_slot), _p(row0),
                                 _p(rows), count, max_rows, n, num_heads, kv_heads, page_size, window, _f(scale),
                                 per, splits, _p(None), _p(sink), _f(cap), _p(gate), ldg, _p(fault), _stream()), alib)
    return out


def swiglu(gu: torch.Tensor, out: torch.Tensor, block: Optional[int] = None, form: GateForm = SILU) -> torch.Tensor:
    """out[r, j] = gated(gate_j, up_j) in the form ``form`` (silu(gate_j) * up_j unless given) where a row of ``gu`` holds
    gate and up columns in alternating blocks of ``block`` (default: the hidden size, i.e. [all gates | all ups])."""
    lib = library()
    n, f = out.shape
    _check(lib.tis_swiglu(_dt(gu), _p(gu), _p(out), n, f, block or f, form, _stream()), lib)
    return out


def glu_clamped(gu: torch.Tensor, gate_bias: Optional[torch.Tensor], up_bias: Optional[torch.Tensor], limit: float,
                alpha: float, shift: float, out: torch.Tensor, hidden: int) -> torch.Tensor:
    """A row of ``gu`` holds ``hidden`` gate columns, then as many up columns.  g = min(gate + bias, limit),
    u = clamp(up + bias, -limit, limit) (``limit`` <= 0: unclamped); out[:, :hidden] = g * sigmoid(alpha * g) *
    (u + shift); the columns of ``out`` beyond ``hidden`` get 1, 0, 0, ... (a column of ones for the bias of the
    product that follows)."""
    lib = library()
    n = gu.shape[0]
    _check(lib.tis_glu_clamped(_dt(gu), _p(gu), gu.stride(0), _p(gate_bias), _p(up_bias), _f(limit), _f(alpha), _f(shift),
                               _p(out), out.stride(0), n, hidden, _stream()), lib)
    return out


def scale_f32(x: torch.Tensor, scale: float) -> torch.Tensor:
    """x *= scale in place (contiguous float32)."""
    lib = library()
    _check(lib.tis_scale_f32(_p(x), _f(scale), ctypes.c_size_t(x.numel()), _stream()), lib)
    return x


def softcap_f32(x: torch.Tensor, cap: float) -> torch.Tensor:
    """x = cap * tanh(x / cap) in place (contiguous float32)."""
    lib = library()
    _check(lib.tis_softcap_f32(_p(x), _f(cap), ctypes.c_size_t(x.numel()), _stream()), lib)
    return x


#: activations of a feed-forward without a gate
ACTIVATIONS = {"relu2": 0, "gelu_tanh": 1, "silu": 2, "tanh": 3}


def activation(x: torch.Tensor, out: torch.Tensor, kind: str) -> torch.Tensor:
    """out = act(x) element by element over (n, F) (row strides free): ``relu2`` the square of relu, ``gelu_tanh``
    0.5 x (1 + tanh(sqrt(2 / pi) (x + 0.044715 x^3))), ``silu``, ``tanh``."""
    lib = library()
    if kind not in ACTIVATIONS:
        raise KernelError(f"activation {kind!r}: known are {sorted(ACTIVATIONS)}")
    n, f = x.shape
    _check(lib.tis_activation(_dt(x), _p(x), x.stride(0), _p(out), out.stride(0), n, f, ACTIVATIONS[kind], _stream()), lib)
    return out


def gemm_act(a, w: torch.Tensor, kind: str) -> torch.Tensor:
    """``act(a @ w)``: few bfloat16 rows: a weight-streaming product with the activation in its epilogue; else the
    product, then the activation kernel.  ``a`` may be ``ScaledRows``."""
    return gemm(a, w, act=kind)


def causal_conv(x: torch.Tensor, weight: torch.Tensor, state: torch.Tensor, out: torch.Tensor, row_slot: torch.Tensor,
                row_last: torch.Tensor, residual: bool = False, silu: bool = False,
                bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """A causal convolution over time on each channel: ``out[r, c] = (x[r, c] if residual) + (bias[c] if given) +
    sum_j weight[j, c] * x(t - taps + 1 + j)[c]``, through silu if asked (``bias`` (C,) float32).  ``x`` (n, C) with a free row stride; ``weight`` (taps, C)
    float32 (tap by tap, so that neighbouring channels are neighbours in memory); ``state`` (slots, taps - 1, C) float32 (a view with a free slot stride): the last inputs of every
    request, oldest first, zero before the start of a sequence; read for the rows whose history lies before this
    step and brought up to date."""
    lib = library()
    n, c = x.shape
    taps = weight.shape[0]
    if weight.shape[1] != c or not weight.is_contiguous():
        raise KernelError(f"causal_conv: weights {tuple(weight.shape)} for {c} channels (wanted contiguous (taps, channels))")
    _check(lib.tis_causal_conv(_dt(x), _p(x), x.stride(0), _p(weight), _p(state), ctypes.c_size_t(state.stride(0)),
                               _p(out), out.stride(0), _p(row_slot), _p(row_last), n, c, taps, int(residual), int(silu),
                               _p(bias), _stream()), lib)
    return out


def _page_strides(pages: torch.Tensor, width: int, free_rows: bool = False):
    """(page stride, head stride) of a view [pages, kv_heads, page_size, width] whose rows are dense; with
    ``free_rows`` also the stride from row to row, which may then exceed the width (a slice of wider rows)."""
    if pages.stride(3) != 1 or (pages.stride(2) != width if not free_rows else pages.stride(2) < width):
        raise KernelError("cache pages: the rows of a kv head must lie one after the other")
    if free_rows:
        return ctypes.c_size_t(pages.stride(0)), ctypes.c_size_t(pages.stride(1)), int(pages.stride(2))
    return ctypes.c_size_t(pages.stride(0)), ctypes.c_size_t(pages.stride(1))


def norm_mix_store(qkv: torch.Tensor, nq: int, nk: int, nv: int, q_weight: Optional[torch.Tensor],
                   k_weight: Optional[torch.Tensor], eps: float, v_other: Optional[torch.Tensor],
                   mix: Optional[torch.Tensor], k_pages: torch.Tensor, v_pages: torch.Tensor, block_table: torch.Tensor,
                   positions: torch.Tensor, row_slot: torch.Tensor, page_size: int, fault: torch.Tensor) -> None:
    """Between the projections and the cache of an attention layer.  A row of ``qkv`` holds ``nq`` query, ``nk``
    key and ``nv`` value elements.  Queries (in place) and keys are divided by their root mean square over the
    whole row part (eps inside the root) and multiplied by ``q_weight`` / ``k_weight`` (None: left alone);
    values become ``(1 - mix) * v + mix * v_other`` (``v_other`` (n, nv), None: left alone); keys and values are
    written into the row's place of ``k_pages`` / ``v_pages`` [pages, kv_heads, page_size, width]."""
    lib = library()
    n = qkv.shape[0]
    kv_heads = k_pages.shape[1]
    kps, khs = _page_strides(k_pages, nk // kv_heads)
    vps, vhs = _page_strides(v_pages, nv // kv_heads)
    _check(lib.tis_norm_mix_store(_dt(qkv), _p(qkv), qkv.stride(0), nq, nk, nv, _p(q_weight), _p(k_weight), _f(eps),
                                  _p(v_other), v_other.stride(0) if v_other is not None else 0, _p(mix), _p(k_pages), kps,
                                  khs, _p(v_pages), vps, vhs, kv_heads, page_size, k_pages.shape[0], _p(block_table),
                                  block_table.stride(0), _p(positions), _p(row_slot), _p(fault), n, _stream()), lib)


_wattn_libs = {}


def window_attention_library(k_dim: int, v_dim: int):
    """The tensor-core kernel of windowed attention for one pair of widths, compiled when first needed."""
    lib = _wattn_libs.get((k_dim, v_dim))
    if lib is None:
        library()
        lib = ctypes.CDLL(_build.build_window_attention(k_dim, v_dim))
        lib.tis_last_error.restype = ctypes.c_char_p
        kd, vd = ctypes.c_int(0), ctypes.c_int(0)
        lib.tis_window_attention_mma_dims(ctypes.byref(kd), ctypes.byref(vd))
        if (kd.value, vd.value) != (k_dim, v_dim):
            raise KernelError(f"windowed attention library built for widths {kd.value}/{vd.value}, wanted {k_dim}/{v_dim}")
        _wattn_libs[(k_dim, v_dim)] = lib
    return lib


#: bfloat16 steps run windowed attention on the tensor cores;
#: TIS_WINDOW_ATTENTION_MMA=0 keeps every step on the CUDA-core kernel
WINDOW_ATTENTION_MMA = os.environ.get("TIS_WINDOW_ATTENTION_MMA", "1") != "0"
#: CTAs that the key splits of a decode step's tiles aim at (two per SM)
WINDOW_ATTENTION_CTAS = 2 * 148


def window_attention_mma_usable(q: torch.Tensor, gate, out: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                                gate_per_head: bool = False) -> bool:
    k_dim, v_dim = k_pages.shape[3], v_pages.shape[3]
    return (WINDOW_ATTENTION_MMA and v_pages.stride(2) % 8 == 0 and q.dtype == torch.bfloat16 and k_dim % 16 == 0 and v_dim % 16 == 0
            and 16 <= k_dim <= 256 and 16 <= v_dim <= 256 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0
            and out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0
            and (gate is None or gate_per_head or (gate.stride(0) % 2 == 0 and gate.data_ptr() % 4 == 0))
            and all(s % 8 == 0 for s in (k_pages.stride(0), k_pages.stride(1), v_pages.stride(0), v_pages.stride(1)))
            and k_pages.data_ptr() % 16 == 0 and v_pages.data_ptr() % 16 == 0)


def window_attention(q: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor, k_pages: torch.Tensor,
                     v_pages: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor, row_slot: torch.Tensor,
                     num_heads: int, page_size: int, window: Optional[int], scale: float,
                     bias_slope: Optional[torch.Tensor], bias_rate: Optional[torch.Tensor], fault: torch.Tensor,
                     step=None, sink: Optional[torch.Tensor] = None, gate_per_head: bool = False,
                     chunked: bool = False, softcap: Optional[float] = None) -> torch.Tensor:
    """Attention of the step's rows over the paged cache with keys and values of any widths:
    ``score = q . k * scale - bias_slope[h] * ln(1 + bias_rate[h] * distance)``, softmax over the keys
    ``max(0, p - window + 1) .. p``, the result times ``sigmoid(gate)`` element by element.  ``q`` (n, H * k_dim),
    ``gate`` (n, H * v_dim) or None, ``out`` (n, H * v_dim); row strides free.  ``sink`` (H,) float32: the softmax's
    denominator of head h also holds ``exp(sink[h])`` (unscaled; it has no value).  ``gate_per_head``: ``gate`` is (n, H),
    one number per head for all of the head's elements.  ``chunked`` and ``softcap`` (on ``q . k * scale``, before the bias) as in
    ``paged_attention``.  The value rows may be a slice of
    wider rows (``v_pages`` with a row stride above its width, for instance the first elements of the key rows).

    float32, and widths that are not multiples of 16: a CUDA-core kernel, a CTA per row and head.  bfloat16 inside
    a step (``step`` given, with the tiles of ``kernels.window_plan``): the tensor-core kernel, a CTA per tile of rows
    and kv head; the warps of a decode row's CTA split its keys."""
    lib = library()
    n = q.shape[0]
    kv_heads, k_dim, v_dim = k_pages.shape[1], k_pages.shape[3], v_pages.shape[3]
    kps, khs = _page_strides(k_pages, k_dim)
    vps, vhs, v_row = _page_strides(v_pages, v_dim, free_rows=True)
    code, cap = _window_code(window, chunked), float(softcap or 0.0)
    if step is not None and num_heads // kv_heads <= 64 and window_attention_mma_usable(q, gate, out, k_pages, v_pages,
                                                                                          gate_per_head):
        from . import window_plan
        row0, rows, count = step.plan(window_plan.planner(num_heads // kv_heads))
        wlib = window_attention_library(k_dim, v_dim)
        calls["window_attention_mma"] += 1
        # a decode step has few tiles, each with many keys to walk: share the keys of a tile out over several CTAs
        # (about two CTAs per SM in all), whose partial results a second launch merges
        splits, partial = 1, None
        if getattr(step, "decode_only", False) and count > 0:
            keys = step.max_position + 1 if not window else min(int(window), step.max_position + 1)
            key_tiles = keys // 64 + 1
            splits = max(1, min(key_tiles, WINDOW_ATTENTION_CTAS // max(1, count * kv_heads), 64))
            if splits > 1:
                wlib.tis_window_attention_partial_floats.restype = ctypes.c_size_t
                partial = torch.empty(wlib.tis_window_attention_partial_floats(count, kv_heads, splits), dtype=torch.float32,
                                      device=q.device)
                global launches
                launches += 1
        _check(wlib.tis_window_attention_mma(_p(q), q.stride(0), _p(gate), gate.stride(0) if gate is not None else 0,
                                             _p(out), out.stride(0), _p(k_pages), kps, khs, _p(v_pages), vps, vhs,
                                             _p(block_table), block_table.stride(0), k_pages.shape[0], _p(positions),
                                             _p(row_slot), _p(row0), _p(rows), count, num_heads, kv_heads, page_size,
                                             code, _f(scale), _f(cap), _p(bias_slope), _p(bias_rate), splits, _p(partial),
                                             _p(sink), v_row, int(gate_per_head), _p(fault), _stream()), wlib)
        return out
    calls["window_attention"] += 1
    _check(lib.tis_window_attention(_dt(q), _p(q), q.stride(0), _p(gate), gate.stride(0) if gate is not None else 0,
                                    _p(out), out.stride(0), _p(k_pages), kps, khs, _p(v_pages), vps, vhs, _p(block_table),
                                    block_table.stride(0), k_pages.shape[0], _p(positions), _p(row_slot), n, num_heads,
                                    kv_heads, k_dim, v_dim, page_size, code, _f(scale), _f(cap), _p(bias_slope),
                                    _p(bias_rate), _p(sink), v_row, int(gate_per_head), _p(fault), _stream()), lib)
    return out


#: what a mixer's gate does to the projection it is made from
GATE_ACTS = {"sigmoid": 0, "silu": 1}

#: CTAs of 64 columns from which the delta rule keeps them (fewer: 16 columns a CTA, four times as many CTAs; fewer even of
#: those: 8 columns a CTA with sixteen lanes a column)
DELTA_WIDE_MIN_CTAS = 2 * 148


def _recurrence_spread(requests: Optional[int], num_heads: int, v_dim: int) -> int:
    """How a head's state columns are shared out over CTAs: 0 64 columns a CTA, 1 16 columns, 2 8 columns with sixteen
    lanes each; the fewer requests and heads a step holds, the finer."""
    if requests is None or requests * num_heads * max(1, v_dim // 64) >= DELTA_WIDE_MIN_CTAS:
        return 0
    # the finest geometry only where all of its CTAs are resident at once (two an SM by registers): a second wave of a
    # walk as long as the prompt would double the time
    return 2 if requests * num_heads * max(1, v_dim // 8) <= DELTA_WIDE_MIN_CTAS else 1


def delta_rule(qkv: torch.Tensor, beta: torch.Tensor, decay_in: torch.Tensor, gate: Optional[torch.Tensor],
               a_log: torch.Tensor, dt_bias: torch.Tensor, norm_weight: torch.Tensor, eps: float, unit_eps: float,
               q_scale: float, state: torch.Tensor, out: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor,
               num_heads: int, qk_heads: int, k_dim: int, v_dim: int, requests: Optional[int] = None,
               segments=None, decay_per_head: bool = False, gate_act: str = "sigmoid") -> torch.Tensor:
    """The delta rule with a decay per head and key channel (``decay_per_head``: one per head; ``decay_in`` is then
    (n, H) and ``dt_bias`` (H,)) over the rows of every request, from and into the
    requests' states ``state`` (slots, H, k_dim, v_dim) float32 (a view with a free slot stride).  A row of ``qkv``:
    queries and keys of ``qk_heads`` heads, values of ``num_heads`` heads.  Per head: q and k to unit length
    (``unit_eps`` inside the root; q times ``q_scale``), beta = sigmoid(``beta``), decay = exp(-exp(a_log) *
    softplus(``decay_in`` + dt_bias)) per key channel; S <- decay S; u = beta (v - S^T k); S <- S + k u^T;
    o = S^T q; out = o / rms(o) * norm_weight * act(gate), act = ``gate_act`` (``GATE_ACTS``).  ``requests``: how many requests the step holds, if
    the caller knows (few requests: a head's columns are shared out over more CTAs).  ``segments``: (first rows of
    the step's requests as an int32 device tensor, their number), from ``kernels.segment_plan``: the kernel then
    launches CTAs for the requests only, not for every row."""
    lib = library()
    n = qkv.shape[0]
    narrow = _recurrence_spread(requests, num_heads, v_dim)
    # widths that the kernel with a head's columns split over CTAs takes: the outputs pass through 32-bit scratch
    # and a second launch normalises them
    raw = None
    if lib.tis_delta_rule_splits(k_dim, v_dim):
        raw = torch.empty((n, num_heads * v_dim), dtype=torch.float32, device=qkv.device)
        global launches
        launches += 1
    _check(lib.tis_delta_rule(_dt(qkv), _p(qkv), qkv.stride(0), _p(beta), beta.stride(0), _p(decay_in), decay_in.stride(0),
                              _p(gate), gate.stride(0) if gate is not None else 0, _p(a_log), _p(dt_bias), _p(norm_weight),
                              _f(eps), _f(unit_eps), _f(q_scale), _p(state), ctypes.c_size_t(state.stride(0)), _p(out),
                              out.stride(0), _p(raw), _p(row_slot), _p(row_last), n, num_heads, qk_heads, k_dim, v_dim,
                              int(narrow), _p(segments[0] if segments is not None else None),
                              int(segments[1]) if segments is not None else 0, int(bool(decay_per_head)),
                              GATE_ACTS[gate_act], _stream()), lib)
    return out


def linear_attention(qkv: torch.Tensor, gate: Optional[torch.Tensor], decay: torch.Tensor, norm_weight: torch.Tensor,
                     eps: float, state: torch.Tensor, out: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor,
                     num_heads: int, k_dim: int, v_dim: int, requests: Optional[int] = None, segments=None) -> torch.Tensor:
    """Linear attention with a constant decay per head over the rows of every request, from and into the requests'
    states ``state`` (slots, H, k_dim, v_dim) float32 (a view with a free slot stride).  A row of ``qkv``: queries and
    keys of H heads (k_dim each), values of H heads (v_dim each), all before their activation.  q = silu(q),
    k = silu(k), v = silu(v); S <- decay[head] S + k v^T; o = S^T q; the row's outputs of all heads together are divided
    by their root mean square (eps inside the root), multiplied by ``norm_weight`` (H * v_dim) and by sigmoid(gate).
    ``requests`` and ``segments`` as for ``delta_rule``: the same kernels walk the recurrence."""
    lib = library()
    n = qkv.shape[0]
    narrow = _recurrence_spread(requests, num_heads, v_dim)
    raw = torch.empty((n, num_heads * v_dim), dtype=torch.float32, device=qkv.device)
    global launches
    launches += 1
    _check(lib.tis_linear_attention(_dt(qkv), _p(qkv), qkv.stride(0), _p(gate), gate.stride(0) if gate is not None else 0,
                                    _p(decay), _p(norm_weight), _f(eps), _p(state), ctypes.c_size_t(state.stride(0)),
                                    _p(out), out.stride(0), _p(raw), _p(row_slot), _p(row_last), n, num_heads, k_dim, v_dim,
                                    int(narrow), _p(segments[0] if segments is not None else None),
                                    int(segments[1]) if segments is not None else 0, _stream()), lib)
    return out


def forget_gate_recurrence(qv: torch.Tensor, f_in: torch.Tensor, lower: torch.Tensor, f_bias: torch.Tensor,
                           norm_weight: torch.Tensor, eps: float, state: torch.Tensor, out: torch.Tensor,
                           row_slot: torch.Tensor, row_last: torch.Tensor, num_heads: int, k_dim: int, v_dim: int,
                           requests: Optional[int] = None, segments=None) -> torch.Tensor:
    """A matrix state per head whose forget gate, per key channel, also is one minus the key, over the rows of every
    request, from and into ``state`` (slots, H, k_dim, v_dim) float32 (a view with a free slot stride).  A row of
    ``qv``: queries of H heads (k_dim each, before silu), values of H heads (v_dim each); ``f_in`` (n, H * k_dim) the
    gate's projection.  ``f = lower + (1 - lower) * sigmoid(f_in + f_bias)``; ``S <- diag(f) S + (1 - f) v^T``;
    ``o = S^T silu(q)``; per head ``out = o / rms(o) * norm_weight`` (v_dim weights shared by the heads).  Gate, state
    and norm are 32-bit.  ``requests`` and ``segments`` as for ``delta_rule``: the same kernels walk the recurrence."""
    lib = library()
    n = qv.shape[0]
    narrow = _recurrence_spread(requests, num_heads, v_dim)
    raw = None
    if lib.tis_delta_rule_splits(k_dim, v_dim):
        raw = torch.empty((n, num_heads * v_dim), dtype=torch.float32, device=qv.device)
        global launches
        launches += 1
    _check(lib.tis_forget_gate_recurrence(_dt(qv), _p(qv), qv.stride(0), _p(f_in), f_in.stride(0), _p(lower), _p(f_bias),
                                          _p(norm_weight), _f(eps), _p(state), ctypes.c_size_t(state.stride(0)), _p(out),
                                          out.stride(0), _p(raw), _p(row_slot), _p(row_last), n, num_heads, k_dim, v_dim,
                                          int(narrow), _p(segments[0] if segments is not None else None),
                                          int(segments[1]) if segments is not None else 0, _stream()), lib)
    return out


def head_norm_store(qkv: torch.Tensor, num_heads: int, kv_heads: int, maps: int, dim: int, v_dim: int,
                    bias: Optional[torch.Tensor], q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor],
                    eps: float, temp_coef: float, temp_every: int, q_out: torch.Tensor, k_pages: torch.Tensor,
                    v_pages: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor, row_slot: torch.Tensor,
                    page_size: int, fault: torch.Tensor) -> None:
    """Between the projections and the cache of attention whose heads carry ``maps`` score maps over the same values.
    A row of ``qkv``: ``num_heads * maps`` query runs, ``kv_heads * maps`` key runs (``dim`` elements each, head by
    head, map by map), ``kv_heads`` value runs of ``v_dim``.  ``bias`` (float32, the row's layout; None: none) is
    added; every query and key run is divided by its root mean square (eps inside the root) and multiplied by
    ``q_weight`` / ``k_weight`` (``dim`` weights shared by all runs; None: left alone); queries are multiplied by
    ``1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)`` at position p (``temp_every`` 0: not).  Keys (a kv head's
    runs side by side: ``maps * dim`` wide) and values go to the row's place in ``k_pages`` / ``v_pages``.  ``q_out``
    (n, H * maps * maps * dim) gets ``H * maps`` query heads as wide as a key row: run (h, m) in stretch m of head
    ``h * maps + m``, zeros in its other stretches, so that it meets only map m's part of a key row."""
    lib = library()
    n = qkv.shape[0]
    kps, khs = _page_strides(k_pages, maps * dim)
    vps, vhs = _page_strides(v_pages, v_dim)
    if k_pages.shape[1] != kv_heads or v_pages.shape[1] != kv_heads or q_out.stride(1) != 1 or qkv.stride(1) != 1:
        raise KernelError("head_norm_store: the pages or the rows do not fit the sizes")
    _check(lib.tis_head_norm_store(_dt(qkv), _p(qkv), qkv.stride(0), num_heads, kv_heads, maps, dim, v_dim, _p(bias),
                                   _p(q_weight), _p(k_weight), _f(eps), _f(temp_coef), int(temp_every), _p(q_out),
                                   q_out.stride(0), _p(k_pages), kps, khs, _p(v_pages), vps, vhs, page_size,
                                   k_pages.shape[0], _p(block_table), block_table.stride(0), _p(positions), _p(row_slot),
                                   _p(fault), n, _stream()), lib)


def diff_combine(a: torch.Tensor, lam: float, eps: float, out_scale: float, out: torch.Tensor, num_heads: int,
                 v_dim: int, row_slot: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Two score maps of a head combined: a row of ``a`` holds, head by head, map 1's and map 2's outputs (``v_dim``
    each); ``out[r, h] = o / sqrt(mean(o^2) + eps) * out_scale`` with ``o = a1 - lam * a2``, in 32-bit."""
    lib = library()
    n = a.shape[0]
    _check(lib.tis_diff_combine(_dt(a), _p(a), a.stride(0), _f(lam), _f(eps), _f(out_scale), _p(out), out.stride(0),
                                _p(row_slot), n, num_heads, v_dim, _stream()), lib)
    return out


def latent_prepare(proj: torch.Tensor, dkv_at: int, num_heads: int, flat_dim: int, rot_dim: int, rank: int,
                   c_weight: torch.Tensor, eps: float, cos: torch.Tensor, sin: torch.Tensor, q_out: torch.Tensor,
                   k_pages: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor, row_slot: torch.Tensor,
                   page_size: int, fault: torch.Tensor) -> None:
    """Between the projections and the cache of attention over compressed keys and values.  A row of ``proj`` holds,
    per head, ``flat_dim + rot_dim`` query elements, and from column ``dkv_at`` on ``rank + rot_dim`` elements of the
    compressed projection.  The first ``rank`` of those, divided by their root mean square (eps inside the root) and
    multiplied by ``c_weight``, and the last ``rot_dim``, rotated by the row's position (the first ``dims`` of them, in
    pairs (i, i + dims / 2), with tables ``cos, sin`` [positions, dims / 2] float32; the rest pass unchanged), are written as the row ``[c | rotated slice]`` of the
    position's page in ``k_pages`` [pages, 1, page_size, rank + rot_dim].  The last ``rot_dim`` elements of every
    head's query, rotated the same way, go to ``q_out`` (n, H * (rank + rot_dim)) behind the ``rank`` places that
    the caller fills.  Everything is computed in 32-bit."""
    lib = library()
    n = proj.shape[0]
    dims = 0 if cos is None else 2 * cos.shape[1]          # no tables: nothing is rotated (a model without a rotated slice)
    if k_pages.shape[1] != 1 or k_pages.shape[3] != rank + rot_dim or dims > rot_dim:
        raise KernelError("latent_prepare: the cache rows or the rotation tables do not fit the sizes")
    kps, _ = _page_strides(k_pages, rank + rot_dim)
    _check(lib.tis_latent_prepare(_dt(proj), _p(proj), proj.stride(0), dkv_at, num_heads, flat_dim, rot_dim,
                                  dims, rank, _p(c_weight), _f(eps), _p(cos), _p(sin), cos.shape[0] if cos is not None else 0, _p(q_out), q_out.stride(0),
                                  _p(k_pages), kps, page_size, k_pages.shape[0], _p(block_table), block_table.stride(0),
                                  _p(positions), _p(row_slot), _p(fault), n, _stream()), lib)


def gemm_heads(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out[r, h] = a[r, h] @ w[h]`` for every head h: ``a`` (n, H, K), ``w`` (H, K, N), ``out`` (n, H, N), the first
    two with free row and head strides.  A batched library product (float32 means true float32)."""
    if a.dtype == torch.float32 and torch.backends.cuda.matmul.allow_tf32:
        raise KernelError("float32 products must not run in TF32: torch.backends.cuda.matmul.allow_tf32 is set")
    calls["gemm_heads"] += 1
    n, heads, k = a.shape
    cols = w.shape[2]
    lib = library()
    if _blas_workspace(lib, a.device) and a.stride(2) == 1 and out.stride(2) == 1 and w.is_contiguous() and a.dtype == w.dtype == out.dtype:
        status = lib.tis_gemm_library_heads(_dt(a), _p(a), a.stride(0), ctypes.c_longlong(a.stride(1)), _p(w), _p(out),
                                            out.stride(0), ctypes.c_longlong(out.stride(1)), n, cols, k, heads, _stream())
        if status != 0:
            raise KernelError(lib.tis_last_error().decode())
        return out
    out.copy_(torch.bmm(a.transpose(0, 1), w).transpose(0, 1))
    return out


def gated_linear_attention(qkv: torch.Tensor, a_in: torch.Tensor, power: torch.Tensor, a_bias: torch.Tensor,
                           gate: Optional[torch.Tensor], norm_weight: torch.Tensor, eps: float, q_scale: float,
                           state: torch.Tensor, out: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor,
                           num_heads: int, k_dim: int, v_dim: int, requests: Optional[int] = None, segments=None,
                           gate_act: str = "silu") -> torch.Tensor:
    """Linear attention with a gate per head and key channel over the rows of every request, from and into ``state``
    (slots, H, k_dim, v_dim) float32 (a view with a free slot stride).  A row of ``qkv``: queries and keys of H heads
    (k_dim each), values of H heads (v_dim each); ``a_in`` (n, H * k_dim) the gate's projection, ``a_bias`` (H * k_dim)
    its bias, ``power`` (H,) its exponent.  ``alpha = sigmoid(a_in + a_bias) ** power``; ``S <- diag(alpha) S + k v^T``;
    ``o = S^T (q * q_scale)``; per head ``out = o / rms(o) * norm_weight * act(gate)`` (v_dim weights shared by the
    heads).  Gate, state and norm are 32-bit.  ``requests`` and ``segments`` as for ``delta_rule``."""
    lib = library()
    n = qkv.shape[0]
    narrow = _recurrence_spread(requests, num_heads, v_dim)
    raw = None
    if lib.tis_delta_rule_splits(k_dim, v_dim):
        raw = torch.empty((n, num_heads * v_dim), dtype=torch.float32, device=qkv.device)
        global launches
        launches += 1
    _check(lib.tis_gated_linear_attention(_dt(qkv), _p(qkv), qkv.stride(0), _p(a_in), a_in.stride(0), _p(power), _p(a_bias),
                                          _p(gate), gate.stride(0) if gate is not None else 0, _p(norm_weight), _f(eps),
                                          _f(q_scale), _p(state), ctypes.c_size_t(state.stride(0)), _p(out), out.stride(0),
                                          _p(raw), _p(row_slot), _p(row_last), n, num_heads, k_dim, v_dim, int(narrow),
                                          _p(segments[0] if segments is not None else None),
                                          int(segments[1]) if segments is not None else 0, GATE_ACTS[gate_act], _stream()), lib)
    return out


def state_space_scan(cbx: torch.Tensor, dt_in: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor,
                     state: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor, num_heads: int, groups: int,
                     state_dim: int, v_dim: int, requests: Optional[int] = None, segments=None) -> torch.Tensor:
    """A selective state space in its recurrent form over the rows of every request, from and into ``state`` (slots, H,
    state_dim, v_dim) float32 (a view with a free slot stride).  A row of ``cbx``: the output matrices C and then the
    input matrices B of ``groups`` groups (``state_dim`` each), then the inputs x of H heads (v_dim each); ``dt_in`` (n, H).
    ``dt = softplus(dt_in + dt_bias)``; ``S <- exp(-exp(a_log) dt) S + B (dt x)^T``; returns ``S^T C`` (n, H * v_dim)
    float32.  ``requests`` and ``segments`` as for ``delta_rule``: the same kernels walk the recurrence."""
    lib = library()
    n = cbx.shape[0]
    narrow = _recurrence_spread(requests, num_heads, v_dim)
    raw = torch.empty((n, num_heads * v_dim), dtype=torch.float32, device=cbx.device)
    _check(lib.tis_state_space_scan(_dt(cbx), _p(cbx), cbx.stride(0), _p(dt_in), dt_in.stride(0), _p(a_log), _p(dt_bias),
                                    _p(state), ctypes.c_size_t(state.stride(0)), _p(raw), _p(row_slot), _p(row_last), n,
                                    num_heads, groups, state_dim, v_dim, int(narrow),
                                    _p(segments[0] if segments is not None else None),
                                    int(segments[1]) if segments is not None else 0, _stream()), lib)
    return raw


def skip_gate_group_norm(o_raw: torch.Tensor, x: torch.Tensor, skip: torch.Tensor, z: torch.Tensor, weight: torch.Tensor,
                         groups: int, eps: float, out: torch.Tensor, row_slot: torch.Tensor, num_heads: int,
                         v_dim: int) -> torch.Tensor:
    """``y = (o_raw + skip[head] * x) * silu(z)`` over rows of H heads of v_dim elements, then the row in ``groups``
    equal parts, each divided by its root mean square (eps inside the root), times ``weight``.  ``o_raw`` (n, H * v_dim)
    float32; ``x``, ``z``, ``out`` (n, H * v_dim) with free row strides."""
    lib = library()
    n = o_raw.shape[0]
    _check(lib.tis_skip_gate_group_norm(_dt(out), _p(o_raw), _p(x), x.stride(0), _p(skip), _p(z), z.stride(0), _p(weight),
                                        int(groups), _f(eps), _p(out), out.stride(0), _p(row_slot), n, num_heads, v_dim,
                                        _stream()), lib)
    return out


def token_shift(x: torch.Tensor, mu: torch.Tensor, state: torch.Tensor, row_slot: torch.Tensor,
                row_last: torch.Tensor) -> torch.Tensor:
    """``out[r, s] = x[r] + (before - x[r]) * mu[s]``: ``before`` is the row of the token before r in its request, zero for a
    sequence's first token.  ``x`` (n, d), ``mu`` (S, d) float32, ``state`` (slots, >= d) float32: every request's last row so
    far, read for its first row of the step and brought up to date.  Returns (n, S, d)."""
    lib = library()
    n, d = x.shape
    out = torch.empty((n, mu.shape[0], d), dtype=x.dtype, device=x.device)
    _check(lib.tis_token_shift(_dt(x), _p(x), x.stride(0), _p(mu), mu.shape[0], _p(state), ctypes.c_size_t(state.stride(0)),
                               _p(out), _p(row_slot), _p(row_last), n, d, _stream()), lib)
    return out


def gemm_side_by_side(a: torch.Tensor, w: torch.Tensor, w_last: torch.Tensor, act: Optional[str] = None):
    """Products of several inputs: ``a`` (n, G + 1, K), ``w`` (G, K, N), ``w_last`` (K, M).  Returns (``out`` (n, G * N) with
    ``a[:, g] @ w[g]`` side by side, ``act(a[:, G] @ w_last)`` (n, M)).  Few bfloat16 rows: one launch of the weight-streaming
    kernel for all of them; else a batched library product and one more product."""
    n, groups, k = a.shape[0], w.shape[0], a.shape[2]
    cols, last = w.shape[2], w_last.shape[1]
    total = groups * cols + last
    if (a.dtype == torch.bfloat16 and 0 < n <= SKINNY_MAX_ROWS and k % 8 == 0 and cols % 64 == 0 and last % 8 == 0
            and _ring_tiles(total, k) <= RING_MAX_TILES and a.is_contiguous() and w.is_contiguous() and w_last.is_contiguous()
            and a.data_ptr() % 16 == 0):
        lib = library()
        out = torch.empty((n, total), dtype=a.dtype, device=a.device)
        calls["gemm_skinny_groups"] += 1
        _check(lib.tis_gemm_skinny_groups(_p(a), a.stride(0), ctypes.c_size_t(a.stride(1)), _p(w), groups, cols, _p(w_last), last,
                                          EPI_GROUP_ACT[act] if act is not None else EPI_STORE, _p(out), out.stride(0), n, k,
                                          _ksplit(total, k), _p(tc_fault()), _stream()), lib)
        return out[:, :groups * cols], out[:, groups * cols:]
    out = torch.empty((n, groups * cols), dtype=a.dtype, device=a.device)
    gemm_heads(a[:, :groups], w, out.unflatten(1, (groups, cols)))
    return out, gemm(a[:, groups], w_last, act=act)


def time_mix(rkvg: torch.Tensor, w_in: torch.Tensor, u: torch.Tensor, w_bias: torch.Tensor, norm_weight: torch.Tensor, eps: float,
             state: torch.Tensor, out: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor, num_heads: int, dim: int,
             requests: Optional[int] = None, segments=None) -> torch.Tensor:
    """A matrix state per head with a decay per key channel and a bonus for the current token, over the rows of every request,
    from and into ``state`` (slots, H, dim, dim) float32 (a view with a free slot stride).  A row of ``rkvg``: r, k, v of H heads
    (``dim`` each) and the gate's projection (H * dim); ``w_in`` (n, H * dim) the decay's projection, ``w_bias`` and the bonus
    ``u`` (H * dim) float32.  Per head ``o = (S + diag(u) k v^T)^T r``, then ``S <- diag(exp(-exp(w_in + w_bias))) S + k v^T``;
    ``out = o / rms(o) * norm_weight * silu(gate)`` (H * dim weights).  ``requests`` and ``segments`` as for ``delta_rule``."""
    lib = library()
    n = rkvg.shape[0]
    if rkvg.dtype != w_in.dtype or rkvg.stride(1) != 1 or w_in.stride(1) != 1:
        raise KernelError("time_mix: the rows and the decays' projection are dense and of one type")
    narrow = _recurrence_spread(requests, num_heads, dim)
    raw = None
    if lib.tis_delta_rule_splits(dim, dim):
        raw = torch.empty((n, num_heads * dim), dtype=torch.float32, device=rkvg.device)
        global launches
        launches += 1
    _check(lib.tis_time_mix(_dt(rkvg), _p(rkvg), rkvg.stride(0), _p(w_in), w_in.stride(0), _p(u), _p(w_bias), _p(norm_weight),
                            _f(eps), _p(state), ctypes.c_size_t(state.stride(0)), _p(out), out.stride(0), _p(raw), _p(row_slot),
                            _p(row_last), n, num_heads, dim, int(narrow), _p(segments[0] if segments is not None else None),
                            int(segments[1]) if segments is not None else 0, _stream()), lib)
    return out


#: (requests x channels) of a step up to which a selective scan keeps two states a lane instead of four (twice the CTAs).
#: Measured on a B200 at 3072 channels of 16 states, 2048 rows, us with four / two: one request 212 / 160, eight requests
#: 73 / 75, sixty-four 65 / 83.
SCAN_FINE_MAX_CHANNELS = int(os.environ.get("TIS_SCAN_FINE_MAX_CHANNELS", "8192"))


def selective_scan(x: torch.Tensor, dt_in: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor, b: torch.Tensor,
                   c: torch.Tensor, skip: torch.Tensor, z: torch.Tensor, state: torch.Tensor, out: torch.Tensor,
                   row_slot: torch.Tensor, row_last: torch.Tensor, segments=None) -> torch.Tensor:
    """A selective scan with a decay per channel and state over the rows of every request, from and into ``state`` (slots,
    channels, N) float32 (a view with a free slot stride): ``dt = softplus(dt_in + dt_bias)``; ``S <- exp(-dt exp(a_log)) S +
    dt x b^T``; ``out = (S c + skip * x) * silu(z)``.  ``x, z, out`` (n, channels), ``b, c`` (n, N) with free row strides (the
    same for both), ``dt_in`` (n, channels) float32, ``a_log`` (channels, N), ``dt_bias, skip`` (channels) float32.  N at most
    256.  ``segments`` as for ``delta_rule``."""
    lib = library()
    n, channels = x.shape
    states = a_log.shape[1]
    if b.stride(0) != c.stride(0) or dt_in.dtype != torch.float32 or not (x.dtype == b.dtype == c.dtype == z.dtype == out.dtype):
        raise KernelError("selective_scan: b and c are slices of the same rows, the step sizes 32-bit, the rest of one type")
    requests = int(segments[1]) if segments is not None else n
    calls["selective_scan"] += 1
    _check(lib.tis_selective_scan(_dt(x), _p(x), x.stride(0), _p(dt_in), dt_in.stride(0), _p(dt_bias), _p(a_log), _p(b), _p(c),
                                  b.stride(0), _p(skip), _p(z), z.stride(0), _p(state), ctypes.c_size_t(state.stride(0)), _p(out),
                                  out.stride(0), _p(row_slot), _p(row_last), _p(segments[0] if segments is not None else None),
                                  requests, n, channels, states, int(requests * channels <= SCAN_FINE_MAX_CHANNELS), _stream()), lib)
    return out


def embed_pairs(table: torch.Tensor, pairs: torch.Tensor, tokens: torch.Tensor, positions: torch.Tensor,
                row_slot: torch.Tensor, row_last: torch.Tensor, prev: torch.Tensor, out: torch.Tensor, scale: float,
                buckets: int, mul_prev: int, mul_cur: int) -> torch.Tensor:
    """``out[r] = table[token] * scale + pairs[(previous * mul_prev + token * mul_cur) % buckets]``; a sequence's first
    token takes row ``buckets`` of ``pairs``.  ``prev`` (slots,) int32: every request's last token so far, read for a
    request's first row of the step and brought up to date.  ``out`` is the float32 residual stream (n, d)."""
    lib = library()
    n, d = out.shape
    _check(lib.tis_embed_pairs(_dt(table), _p(table), _p(pairs), _p(tokens), _p(positions), _p(row_slot), _p(row_last),
                               _p(prev), _p(out), n, d, _f(scale), int(buckets), ctypes.c_longlong(mul_prev),
                               ctypes.c_longlong(mul_cur), _stream()), lib)
    return out


def group_norm(residual: torch.Tensor, delta_a: Optional[torch.Tensor], delta_b: Optional[torch.Tensor], groups: int,
               eps: float, w1: Optional[torch.Tensor], out1: Optional[torch.Tensor], w2: Optional[torch.Tensor] = None,
               out2: Optional[torch.Tensor] = None, in_place: bool = False, dtype: Optional[torch.dtype] = None):
    """``residual += delta_a + delta_b`` (each None: nothing), then the RMS norm in ``groups`` equal consecutive parts of
    the sum (each part divided by its own root mean square, eps inside the root): ``out1 = normed * w1`` and, if asked,
    ``out2 = normed * w2``.  ``in_place``: ``residual`` itself becomes ``normed * w1``.  ``w1`` None: only the sum."""
    lib = library()
    n, d = residual.shape
    ref = next((t for t in (out1, out2, delta_a, delta_b) if t is not None), None)
    code = _dt(ref) if ref is not None else (0 if dtype in (None, torch.float32) else 1)
    _check(lib.tis_group_norm(code, _p(residual), _p(delta_a), _p(delta_b), int(groups), _f(eps), _p(w1), _p(out1), _p(w2),
                              _p(out2), int(in_place), n, d, _stream()), lib)
    return out1, out2


def add_layer_norm(residual: torch.Tensor, delta_a: Optional[torch.Tensor], delta_b: Optional[torch.Tensor], w: torch.Tensor,
                   b: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """``residual += delta_a + delta_b`` (each None: nothing), then ``out = (residual - mean) / sqrt(variance + eps) * w + b``
    row by row in 32-bit (the variance is the mean of the squared deviations)."""
    lib = library()
    n, d = residual.shape
    for t in (delta_a, delta_b):
        if t is not None and (t.dtype != out.dtype or not t.is_contiguous()):
            raise KernelError("add_layer_norm: the updates are contiguous and of the output's type")
    _check(lib.tis_add_layer_norm(_dt(out), _p(residual), _p(delta_a), _p(delta_b), _p(w), _p(b), _f(eps), _p(out), n, d,
                                  _stream()), lib)
    return out


def rotate_norm_store(qkv: torch.Tensor, num_heads: int, kv_heads: int, dim: int, v_dim: int, cos: Optional[torch.Tensor],
                      sin: Optional[torch.Tensor], interleaved: bool, norm: bool, eps: float, k_pages: Optional[torch.Tensor],
                      v_pages: Optional[torch.Tensor], block_table: torch.Tensor, positions: torch.Tensor,
                      row_slot: torch.Tensor, page_size: int, fault: torch.Tensor, permuted: bool = False,
                      whole_weight: Optional[torch.Tensor] = None) -> None:
    """Between the projections and the cache of an attention whose queries and keys are rotated and then normed head by
    head.  A row of ``qkv``: H query heads and G key heads of ``dim`` elements, G value heads of ``v_dim``.  The first
    elements of every query and key head, twice as many as ``cos`` and ``sin`` (positions, rot / 2; None: none) have columns,
    are rotated by the row's position (``interleaved``: element 2i with 2i + 1, else i with i + rot / 2); with ``norm`` the
    head is then divided by its root mean square (eps inside the root).  Queries in place; keys and values into the row's
    page, in the row format of ``paged_attention`` if ``permuted`` (16-byte chunks permuted by the position), else as they
    are.  ``kv_heads`` 0: the rows hold queries only and nothing is stored.  ``whole_weight`` ((H + G) * dim float32: the queries'
    weights, then the keys'): the norm comes *before* the rotation and runs over all query heads, and over all key heads, at
    once (``norm`` is then not looked at).  Everything is computed in 32-bit."""
    lib = library()
    n = qkv.shape[0]
    rot = 0 if cos is None else 2 * cos.shape[1]
    kps = khs = vps = vhs = ctypes.c_size_t(0)
    if kv_heads:
        kps, khs = _page_strides(k_pages, dim)
        vps, vhs = _page_strides(v_pages, v_dim)
        if k_pages.shape[1] != kv_heads or v_pages.shape[1] != kv_heads:
            raise KernelError("rotate_norm_store: the pages do not fit the key/value heads")
    else:
        k_pages = v_pages = None
    if qkv.stride(1) != 1:
        raise KernelError("rotate_norm_store: the rows are not dense")
    if whole_weight is not None and (whole_weight.numel() != (num_heads + kv_heads) * dim or whole_weight.dtype != torch.float32
                                     or not whole_weight.is_contiguous()):
        raise KernelError("rotate_norm_store: one 32-bit weight for every query and key element")
    _check(lib.tis_rotate_norm_store(_dt(qkv), _p(qkv), qkv.stride(0), num_heads, kv_heads, dim, v_dim, rot, int(interleaved),
                                     int(permuted), _p(cos), _p(sin), int(norm), _f(eps), _p(whole_weight), _p(k_pages), kps, khs, _p(v_pages), vps, vhs,
                                     page_size, k_pages.shape[0] if k_pages is not None else 0, _p(block_table),
                                     block_table.stride(0), _p(positions), _p(row_slot), _p(fault), n, _stream()), lib)


def scaled_sum(a: torch.Tensor, scale_a: float, b: torch.Tensor, scale_b: float) -> torch.Tensor:
    """``a * scale_a + b * scale_b`` (n, d), the sum formed in 32-bit; row strides free."""
    lib = library()
    n, d = a.shape
    out = torch.empty((n, d), dtype=a.dtype, device=a.device)
    _check(lib.tis_scaled_sum(_dt(a), _p(a), a.stride(0), _f(scale_a), _p(b), b.stride(0), _f(scale_b), _p(out), out.stride(0),
                              n, d, _stream()), lib)
    return out


def rotate_tie_store(qk: torch.Tensor, num_heads: int, kv_heads: int, dim: int, rot: int, cos: torch.Tensor,
                     sin: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, block_table: torch.Tensor,
                     positions: torch.Tensor, row_slot: torch.Tensor, page_size: int, fault: torch.Tensor) -> None:
    """Between the projections and the cache of an attention whose values are its keys before rotation.  A row of ``qk``:
    H query heads, then G key heads, ``dim`` elements each.  The first ``rot`` elements of every head are rotated by the
    row's position (element i with i + rot / 2; ``cos``, ``sin`` (positions, rot / 2) float32): queries in place, keys into
    the key rows of the row's page; the unrotated keys go into the value rows."""
    lib = library()
    n = qk.shape[0]
    kps, khs = _page_strides(k_pages, dim)
    vps, vhs = _page_strides(v_pages, dim)
    _check(lib.tis_rotate_tie_store(_dt(qk), _p(qk), qk.stride(0), num_heads, kv_heads, dim, rot, _p(cos), _p(sin),
                                    _p(k_pages), kps, khs, _p(v_pages), vps, vhs, page_size, k_pages.shape[0],
                                    _p(block_table), block_table.stride(0), _p(positions), _p(row_slot), _p(fault), n,
                                    _stream()), lib)


# ---------------------------------------------------------------------------------------
# routed experts
# ---------------------------------------------------------------------------------------

#: how a router turns logits into choices and weights
ROUTER_SCORES = {"sigmoid": 0, "softmax_chosen": 1, "softmax": 2}
#: the strength of a group of experts: the sum of its two largest choosing scores, or its largest
GROUP_SCORES = {"two_best": 0, "best": 1}


def moe_route(x: torch.Tensor, w_router: torch.Tensor, correction: Optional[torch.Tensor],
              w_shared_gate: Optional[torch.Tensor], groups: int, keep: int, top: int, weight_eps: float = 1e-20,
              scores: str = "sigmoid", group_score: str = "two_best", renorm: bool = True):
    """The router of a mixture of experts, a row at a time, in 32-bit: ``s = sigmoid(w_router x)`` (E experts);
    choosing scores ``s + correction``; with ``groups`` > 0 only the experts of the ``keep`` groups (of E / groups
    neighbours) with the largest sum of their two best choosing scores can be chosen; the ``top`` largest choosing
    scores win (the lower index on a tie); weights ``s`` of the chosen over their sum (+ ``weight_eps``).  ``scores``
    ``"softmax_chosen"``: the logits themselves choose and the weights are the softmax over the chosen logits only;
    ``"softmax"``: ``s = softmax(w_router x)`` over all experts.  ``group_score`` (``GROUP_SCORES``) ``"best"``: a group is as
    strong as its largest choosing score.  ``renorm`` False: the weights are the chosen ``s`` as they are.  Returns
    (chosen (n, top) int32, weights (n, top) float32, sigmoid(w_shared_gate . x) (n,) float32 or None)."""
    lib = library()
    n, d = x.shape
    experts = w_router.shape[0]
    chosen = torch.empty((n, top), dtype=torch.int32, device=x.device)
    weights = torch.empty((n, top), dtype=torch.float32, device=x.device)
    shared = torch.empty((n,), dtype=torch.float32, device=x.device) if w_shared_gate is not None else None
    _check(lib.tis_moe_route(_dt(x), _p(x), x.stride(0), _p(w_router), _p(correction), _p(w_shared_gate), n, d, experts,
                             int(groups), int(keep), int(top), _f(weight_eps), _p(chosen), _p(weights), _p(shared),
                             ROUTER_SCORES[scores], GROUP_SCORES[group_score], int(renorm), _stream()), lib)
    return chosen, weights, shared


def moe_gate_up(x: torch.Tensor, chosen: torch.Tensor, w_gate_up: torch.Tensor, act: Optional[str] = None,
                form: GateForm = SILU, in_weights: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``hidden[r * top + k] = gated(Wg[e] x[r], Wu[e] x[r])`` in the form ``form`` with ``e = chosen[r, k]``: ``w_gate_up`` (E, 2, F, d)
    holds every expert's gate and up matrices (out, in); the result is (n * top, F) in the dtype of ``x``.  ``act``
    (``ACTIVATIONS``): units without a gate, ``hidden = act(Wu[e] x[r])`` with ``w_gate_up`` (E, F, d).  ``in_weights`` (n, top): multiplies every unit's input."""
    lib = library()
    n, d = x.shape
    top = chosen.shape[1]
    experts, hidden = w_gate_up.shape[0], w_gate_up.shape[-2]
    out = torch.empty((n * top, hidden), dtype=x.dtype, device=x.device)
    _check(lib.tis_moe_gate_up(_dt(x), _p(x), x.stride(0), _p(chosen), _p(w_gate_up), _p(out), n, d, top, experts, hidden,
                               ACTIVATIONS[act] if act is not None else -1, form, _p(in_weights), _stream()), lib)
    return out


def moe_down(hidden: torch.Tensor, chosen: torch.Tensor, weights: Optional[torch.Tensor], w_down: torch.Tensor,
             shared: Optional[torch.Tensor], shared_gate: Optional[torch.Tensor]) -> torch.Tensor:
    """``out[r] = sum_k weights[r, k] * Wd[chosen[r, k]] hidden[r * top + k] (+ shared_gate[r] * shared[r]; the gate None: + shared[r])``:
    ``w_down`` (E, d, F) (out, in), ``hidden`` (n * top, F), ``shared`` (n, d) or None; ``weights`` None: 1; the result is (n, d)."""
    lib = library()
    n, top = chosen.shape
    experts, d, f = w_down.shape
    out = torch.empty((n, d), dtype=hidden.dtype, device=hidden.device)
    _check(lib.tis_moe_down(_dt(hidden), _p(hidden), _p(chosen), _p(weights), _p(w_down), _p(shared),
                            shared.stride(0) if shared is not None else 0, _p(shared_gate), _p(out), n, d, top, experts, f,
                            _stream()), lib)
    return out


def mtp_input(h_prev: torch.Tensor, state: torch.Tensor, row_slot: torch.Tensor, row_last: torch.Tensor,
              tokens: torch.Tensor, table: torch.Tensor, scale: torch.Tensor, eps: float,
              out: torch.Tensor) -> torch.Tensor:
    """out[r] = [h_prev of the row before r (the slot's saved row for a request's first row) |
    rmsnorm(table[tokens[r]])]; saves h_prev[row_last[r]] into the slot for the next step."""
    lib = library()
    n, d = h_prev.shape
    _check(lib.tis_mtp_input(_dt(h_prev), _p(h_prev), _p(state), _p(row_slot), _p(row_last), _p(tokens),
                             _p(table), _p(scale), _f(eps), _p(out), n, d, _stream()), lib)
    return out


# ---------------------------------------------------------------------------------------
# sampling
# ---------------------------------------------------------------------------------------

def sample_rows(logits: torch.Tensor, temps: torch.Tensor, top_ks: torch.Tensor, top_ps: torch.Tensor,
                penalties: torch.Tensor, slots: Optional[torch.Tensor], seen_bitmap: Optional[torch.Tensor],
                seeds: torch.Tensor, counters: torch.Tensor, out_tokens: torch.Tensor,
                probs_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One token per row of float32 ``logits`` (k, V); see csrc/sampling.cu for the order of
    the transformations.  ``seen_bitmap`` (slots, ceil(V/32)) int32 gets the drawn token's bit."""
    lib = library()
    k, v = logits.shape
    words = seen_bitmap.shape[1] if seen_bitmap is not None else 0
    _check(lib.tis_sample_rows(_p(logits), k, v, _p(temps), _p(top_ks), _p(top_ps), _p(penalties), _p(slots),
                               _p(seen_bitmap), words, _p(seeds), _p(counters), _p(out_tokens), _p(probs_out),
                               _stream()), lib)
    return out_tokens


def sample_stage_limit(entries: int) -> None:
    """For tests: the most entries of a row that a CTA of the sampling kernel keeps in shared memory (fewer
    means more CTAs a row; 0: none, every pass reads the logits; -1: what the device allows)."""
    _check(library().tis_sample_stage_limit(int(entries)), library())


def bitmap_set(bitmap_row: torch.Tensor, tokens: torch.Tensor) -> None:
    lib = library()
    _check(lib.tis_bitmap_set(_p(bitmap_row), _p(tokens), tokens.numel(), _stream()), lib)


#: (token, choice) pairs from which bfloat16 expert products go to the tiles on the tensor cores (rows sorted by expert on
#: the device) instead of one dot product per output element; TIS_MOE_GROUPED_MIN_PAIRS overrides (0: never)
MOE_GROUPED_MIN_PAIRS = int(os.environ.get("TIS_MOE_GROUPED_MIN_PAIRS", "96"))
#: pairs from which they go to the tcgen05 kernel (tiles of 128 rows, TMA-fed, accumulator in tensor memory) where width and
#: hidden size are multiples of 64; TIS_MOE_TC_MIN_PAIRS overrides (0: never)
MOE_TC_MIN_PAIRS = int(os.environ.get("TIS_MOE_TC_MIN_PAIRS", "1024"))


def moe_experts(x: torch.Tensor, chosen: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor,
                shared: Optional[torch.Tensor], shared_gate: Optional[torch.Tensor], act: Optional[str] = None,
                form: GateForm = SILU, weigh_input: bool = False) -> torch.Tensor:
    """``out[r] = sum_k weights[r, k] * unit(chosen[r, k])(x[r]) (+ shared_gate[r] * shared[r], or + shared[r])`` with the gated
    units ``unit(e)(x) = Wd[e] gated(Wg[e] x, Wu[e] x)`` in the form ``form``: ``w_gate_up`` (E, 2, F, d), ``w_down`` (E, d, F); or, with ``act``
    (``ACTIVATIONS``), units without a gate, ``Wd[e] act(Wu[e] x)`` and ``w_gate_up`` (E, F, d).  ``weigh_input``: ``sum_k unit(chosen[r, k])(weights[r, k] *
    x[r])`` instead (the weight multiplies both projections of the unit in 32-bit).  Few rows, and
    float32: ``moe_gate_up`` and ``moe_down`` (a dot product per output element, the weights read where they lie).  Many
    bfloat16 rows: the rows are sorted by expert on the device and every expert's rows run as tiles on the tensor
    cores; nothing is read back, so either way the step can be captured in a graph."""
    n, d = x.shape
    top = chosen.shape[1]
    experts, hidden = w_gate_up.shape[0], w_gate_up.shape[-2]
    act_code = ACTIVATIONS[act] if act is not None else -1
    grouped = (x.dtype == torch.bfloat16 and MOE_GROUPED_MIN_PAIRS > 0 and x.stride(1) == 1 and x.stride(0) % 8 == 0
               and x.data_ptr() % 16 == 0 and (shared is None or (shared.stride(1) == 1 and shared.stride(0) % 2 == 0)))
    if grouped and MOE_TC_MIN_PAIRS > 0 and n * top >= MOE_TC_MIN_PAIRS and d % 64 == 0 and hidden % 64 == 0:
        # many rows: 128-row tiles on the tcgen05 tensor cores, the stacked weights as TMA boxes where they lie
        lib = library()
        tiles = lib.tis_moe_tc_tiles(n * top, experts)
        dev = x.device
        meta = torch.empty(tiles * 128 + n * top + tiles, dtype=torch.int32, device=dev)
        sorted_pair, pair_place, tile_expert = meta[:tiles * 128], meta[tiles * 128:tiles * 128 + n * top], meta[tiles * 128 + n * top:]
        xs = torch.empty((tiles * 128, d), dtype=x.dtype, device=dev)
        hid = torch.empty((tiles * 128, hidden), dtype=x.dtype, device=dev)
        y = torch.empty((tiles * 128, d), dtype=x.dtype, device=dev)
        out = torch.empty((n, d), dtype=x.dtype, device=dev)
        calls["moe_grouped_tc"] += 1
        global launches
        launches += 4
        _check(lib.tis_moe_grouped_tc(_p(x), x.stride(0), _p(chosen), _p(weights), _p(w_gate_up), _p(w_down), _p(shared),
                                      shared.stride(0) if shared is not None else 0, _p(shared_gate), _p(out), _p(sorted_pair),
                                      _p(pair_place), _p(tile_expert), _p(xs), _p(hid), _p(y), n, d, top, experts, hidden,
                                      act_code, form, int(weigh_input), _p(tc_fault()), _stream()), lib)
        return out
    if (grouped and n * top >= MOE_GROUPED_MIN_PAIRS and d % 32 == 0
            and hidden % 32 == 0):
        lib = library()
        tiles = lib.tis_moe_grouped_tiles(n * top, experts)
        dev = x.device
        meta = torch.empty(tiles * 64 + n * top + tiles, dtype=torch.int32, device=dev)
        sorted_pair, pair_place, tile_expert = meta[:tiles * 64], meta[tiles * 64:tiles * 64 + n * top], meta[tiles * 64 + n * top:]
        hid = torch.empty((tiles * 64, hidden), dtype=x.dtype, device=dev)
        y = torch.empty((tiles * 64, d), dtype=x.dtype, device=dev)
        out = torch.empty((n, d), dtype=x.dtype, device=dev)
        calls["moe_grouped"] += 1
        launches += 3
        _check(lib.tis_moe_grouped(_p(x), x.stride(0), _p(chosen), _p(weights), _p(w_gate_up), _p(w_down), _p(shared),
                                   shared.stride(0) if shared is not None else 0, _p(shared_gate), _p(out), _p(sorted_pair),
                                   _p(pair_place), _p(tile_expert), _p(hid), _p(y), n, d, top, experts, hidden, act_code,
                                   form, int(weigh_input), _stream()), lib)
        return out
    hid = moe_gate_up(x, chosen, w_gate_up, act, form, weights if weigh_input else None)
    return moe_down(hid, chosen, None if weigh_input else weights, w_down, shared, shared_gate)
