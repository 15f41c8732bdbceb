"""Tensor-level operators over the C ABI.

`apply_delta` keeps the signature of the reference's op
(serving/vllm/delta/deltazip_marlin.py:10-19):

    y = apply_delta(x, qweight_stacked, scales_stacked, meta_stacked, indices, base_weight)

All tensors are CUDA tensors; work is enqueued on torch's current stream.
PyTorch is used for memory and streams only -- every computation below runs in
libdeltazip_b200.so, with one exception: for prefill-sized batches (more than
FUSED_MAX_TOKENS rows) the plain dense product x W^T, the reference's F.linear
(serving/vllm/model_executor/layers/linear.py:85-96), goes to the library GEMM
(torch.matmul) once, and the library's kernel then adds the delta products into
that result token block by token block.  The fused kernel streams W once per
block of 128 tokens, which is the right trade for decode batches and the wrong
one for thousands of prompt tokens.
"""
from __future__ import annotations

import ctypes
import functools
from typing import NamedTuple, Optional, Tuple

import torch

from . import _lib
from ._lib import SbmmArgs, check, lib


# Largest batch (rows of x) that takes the fused kernel for base and delta products together.
FUSED_MAX_TOKENS = 512
# In a prefill-sized, sorted batch whose host-side run list is known (Segments.host_runs), a slot
# with at least this many consecutive rows is dequantised once (dz_unpack) and multiplied by the
# library GEMM, as the reference's PyTorch path does (deltazip/nn_modules/qlinear.py:266-330);
# the SBMM kernel would expand the slot's codes once per 32-row window instead.
DENSE_RUN_TOKENS = 256


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _need_cuda(*tensors):
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise ValueError("deltazip_b200 operators take CUDA tensors only (no CPU path)")


# ---------------------------------------------------------------------------
# slot format
# ---------------------------------------------------------------------------

def slot_shapes(n: int, k: int, bits: int) -> Tuple[Tuple[int, int], Tuple[int, int], Tuple[int, int]]:
    """(qweight int32, meta int16, scales fp16) shapes of one slot of a [n, k] layer.

    Same outer shapes as the reference's stacked tensors
    (serving/vllm/delta/layers_marlin.py:311-333) for 4-bit; for 2-bit the
    metadata keeps k/16 int16 per row (the reference formula would give k/32,
    which cannot hold two 2-bit positions per group of four)."""
    return (k * bits // 128, 2 * n), (n, k // 16), (1, n)


def alloc_slots(num_slots: int, n: int, k: int, bits: int, device) -> Tuple[torch.Tensor, ...]:
    qs, ms, ss = slot_shapes(n, k, bits)
    return (torch.zeros((num_slots, *qs), dtype=torch.int32, device=device),
            torch.zeros((num_slots, *ms), dtype=torch.int16, device=device),
            torch.zeros((num_slots, *ss), dtype=torch.float16, device=device))


def convert_from_gptq(qweight: torch.Tensor, qzeros: torch.Tensor, scales: torch.Tensor, bits: int,
                      out: Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]] = None,
                      check_status: bool = True):
    """GPTQ-layout tensors of one delta layer -> (qweight, meta, scales) in slot layout."""
    _need_cuda(qweight, qzeros, scales)
    k = qweight.shape[0] * 32 // bits
    n = qweight.shape[1]
    qweight = qweight.contiguous()
    qzeros = qzeros.contiguous()
    scales = scales.contiguous()
    if out is None:
        qs, ms, ss = slot_shapes(n, k, bits)
        out = (torch.empty(qs, dtype=torch.int32, device=qweight.device),
               torch.empty(ms, dtype=torch.int16, device=qweight.device),
               torch.empty(ss, dtype=torch.float16, device=qweight.device))
    sq, sm, ss_ = out
    status = torch.zeros(1, dtype=torch.int32, device=qweight.device)
    check(lib().dz_convert_from_gptq(qweight.data_ptr(), qzeros.data_ptr(), scales.data_ptr(),
                                     n, k, bits, sq.data_ptr(), sm.data_ptr(), ss_.data_ptr(),
                                     status.data_ptr(), _stream()), "dz_convert_from_gptq")
    if check_status:
        host = ctypes.c_int(0)
        check(lib().dz_read_status(status.data_ptr(), _stream(), ctypes.byref(host)), "dz_read_status")
        check(host.value, "dz_convert_from_gptq(device)")
    return out


def unpack(slot_qweight: torch.Tensor, slot_meta: torch.Tensor, slot_scales: torch.Tensor,
           n: int, k: int, bits: int) -> torch.Tensor:
    """Dense fp16 delta [n, k] of one slot (bit-identical to QuantLinear.unpack)."""
    _need_cuda(slot_qweight, slot_meta, slot_scales)
    out = torch.empty((n, k), dtype=torch.float16, device=slot_qweight.device)
    check(lib().dz_unpack(slot_qweight.data_ptr(), slot_meta.data_ptr(), slot_scales.data_ptr(),
                          n, k, bits, out.data_ptr(), _stream()), "dz_unpack")
    return out


# ---------------------------------------------------------------------------
# batch metadata
# ---------------------------------------------------------------------------

class Segments:
    """Device-side segment table for one batch (one scheduling step).

    Built from the per-token slot indices (`base_indices` of the reference's
    convert_mapping, serving/vllm/delta/models.py:69-145) and shared by every
    layer of the step."""

    def __init__(self, max_tokens: int, num_slots: int, device):
        self.max_tokens = int(max_tokens)
        self.num_slots = int(num_slots)
        nbytes = lib().dz_segments_bytes(self.max_tokens, self.num_slots)
        self.buf = torch.zeros(nbytes, dtype=torch.uint8, device=device)
        self.m = 0
        self.sorted = False
        # [(slot, first row, end row)] of a sorted batch when the caller knows it on the host
        # (the slot manager does); None otherwise.  Only prefill-sized batches use it.
        self.host_runs = None

    def build(self, indices: torch.Tensor, sorted_hint: Optional[bool] = None) -> "Segments":
        """Builds the table on the current stream; never synchronises with the host.
        `sorted_hint=True` is the caller's promise that `indices` is non-decreasing (the
        reference's scheduler delivers batches sorted by delta id,
        serving/vllm/core/scheduler.py:101-104): x is then read in place.  Without the
        promise the SBMM first gathers x into sorted order on the device (a plain copy when
        the batch happens to be sorted), so any order is handled."""
        _need_cuda(indices)
        m = indices.numel()
        if m > self.max_tokens:
            raise ValueError(f"{m} tokens exceed the table capacity {self.max_tokens}")
        if indices.dtype == torch.int64:
            dt = _lib.DZ_INDEX_I64
        elif indices.dtype == torch.int32:
            dt = _lib.DZ_INDEX_I32
        else:
            raise ValueError("indices must be int32 or int64")
        indices = indices.contiguous()
        check(lib().dz_build_segments(indices.data_ptr(), dt, m, self.num_slots,
                                      self.buf.data_ptr(), _stream()), "dz_build_segments")
        self.m = m
        self.sorted = bool(sorted_hint)
        self.host_runs = None
        return self

    def is_sorted_on_device(self) -> bool:
        """What the device-side builder found (synchronises; for tests and diagnostics)."""
        return bool(self.header()[3])

    def header(self):
        """(M, num_slots, num_token_blocks, sorted, status, num_windows, num_active) -- syncs."""
        return tuple(self.buf[:32].view(torch.int32)[:7].tolist())


_workspaces = {}


def _workspace(device, nbytes: int) -> torch.Tensor:
    """One grow-only scratch buffer per (device, stream).  The SBMM kernel keeps
    split-K partial tiles and tile counters here; calls on one stream are
    ordered, so they can share it."""
    key = (device.index, _stream())
    ws = _workspaces.get(key)
    if ws is None or ws.numel() < nbytes:
        ws = torch.zeros(max(nbytes, 1 << 20), dtype=torch.uint8, device=device)
        _workspaces[key] = ws
    return ws


def read_status(device=None) -> int:
    """Reads and clears the status words the SBMM, window attention, latent attention and expert kernels leave in the
    current stream's workspaces (0 = ok, DZ_ERR_TIMEOUT = a bounded device-side wait ran
    out, DZ_ERR_INVALID_ARG = a wrong `tokens_sorted` promise).  Synchronises."""
    device = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    found = 0
    for ws in (_workspaces.get((device.index, _stream())),
               _scratch.get(("window_attention", device.index, _stream())),
               _scratch.get(("status", device.index, _stream()))):
        if ws is not None:
            host = ctypes.c_int(0)
            check(lib().dz_read_status(ws.data_ptr(), _stream(), ctypes.byref(host)), "dz_read_status")
            found = found or host.value
    return found


def _dtype_code(t: torch.Tensor) -> int:
    if t.dtype == torch.float16:
        return _lib.DZ_DTYPE_F16
    if t.dtype == torch.bfloat16:
        return _lib.DZ_DTYPE_BF16
    raise ValueError(f"unsupported activation dtype {t.dtype}")


def _bits_from_shapes(qweight_stacked: torch.Tensor, k: int) -> int:
    # qweight slot is [k * bits / 128, 2n] int32
    return qweight_stacked.shape[-2] * 128 // k


def sbmm(x: torch.Tensor, qweight_stacked: torch.Tensor, scales_stacked: torch.Tensor,
         meta_stacked: torch.Tensor, segments: Segments, base_weight: Optional[torch.Tensor],
         out: Optional[torch.Tensor] = None, bits: Optional[int] = None,
         _entry: str = "dz_sbmm", accumulate: bool = False, stable: bool = False,
         push=None) -> Optional[torch.Tensor]:
    """y = x W^T + x dequant(delta_slot(i))^T with a prebuilt segment table.  With
    `base_weight=None` only the delta products are computed (rows of slot -1 get 0).
    `out` may be a column slice [:, a:a+N] of a wider row-major tensor; with
    `accumulate=True` the result is added to `out` inside the kernel.  `stable=True` is the
    caller's statement that the base weight, the slot stacks and the segment table were not
    written by the operation right before this call on the stream (DZ_SBMM_INPUTS_STABLE): the
    kernel then starts loading them while its predecessor finishes.  After writing any of them
    with a torch op, call `stream_fence()` before relying on it.  With `push` (a target from
    CustomAllreduce.push_target) the output is not written locally at all: every finished tile
    goes to all tensor-parallel ranks' receive slots and `all_reduce_pushed` yields the sum;
    the call then returns None."""
    _need_cuda(x, qweight_stacked, scales_stacked, meta_stacked)
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    m, k = x2.shape
    if base_weight is None:
        n = scales_stacked.shape[-1]
    else:
        _need_cuda(base_weight)
        n = base_weight.shape[0]
        if base_weight.shape[1] != k or not base_weight.is_contiguous():
            raise ValueError("base_weight must be a contiguous [N, K] tensor matching x")
    if segments.m != m:
        raise ValueError(f"segment table was built for {segments.m} tokens, x has {m}")
    if bits is None:
        bits = _bits_from_shapes(qweight_stacked, k)
    if base_weight is not None and m > FUSED_MAX_TOKENS and push is None and _entry == "dz_sbmm":
        # prefill-sized batch: the dense product once through the library GEMM, then the
        # delta products added to it in place (not the early-start form: y is the
        # predecessor's output here)
        base = torch.matmul(x2, base_weight.t())
        if out is None:
            out = base
        else:
            o2 = out.reshape(-1, out.shape[-1]) if out.dim() != 2 else out
            if accumulate:
                o2.add_(base)
            else:
                o2.copy_(base)
        runs = segments.host_runs
        if runs is not None and segments.sorted and \
                all(e - s >= DENSE_RUN_TOKENS for slot, s, e in runs if slot >= 0):
            o2 = out.reshape(-1, out.shape[-1]) if out.dim() != 2 else out
            for slot, s, e in runs:
                if slot < 0:
                    continue
                dense = unpack(qweight_stacked[slot], meta_stacked[slot], scales_stacked[slot],
                               n, k, bits)
                o2[s:e].addmm_(x2[s:e], dense.to(x2.dtype).t())
        else:
            sbmm(x2, qweight_stacked, scales_stacked, meta_stacked, segments, None, out=out,
                 bits=bits, accumulate=True)
        return out.reshape(*x.shape[:-1], n) if out.is_contiguous() else out
    if push is not None:
        if accumulate or out is not None or m == 0:
            raise ValueError("a pushed output takes neither `out` nor `accumulate`, and needs rows")
        nbytes = lib().dz_sbmm_workspace_bytes(m, n, k, int(segments.sorted))
        ws = _workspace(x.device, nbytes)
        args = SbmmArgs(
            x=x2.data_ptr(), w_base=base_weight.data_ptr() if base_weight is not None else None,
            qweight=qweight_stacked.data_ptr(), meta=meta_stacked.data_ptr(),
            scales=scales_stacked.data_ptr(), qweight_stride=qweight_stacked.stride(0) * 4,
            meta_stride=meta_stacked.stride(0) * 2, scales_stride=scales_stacked.stride(0) * 2,
            segments=segments.buf.data_ptr(), y=None, M=m, N=n, K=k,
            num_slots=qweight_stacked.shape[0], bits=bits, dtype=_dtype_code(x),
            tokens_sorted=int(segments.sorted),
            flags=_lib.DZ_SBMM_INPUTS_STABLE if stable else 0,
            workspace=ws.data_ptr(), workspace_bytes=ws.numel(), y_stride=0,
            push=ctypes.pointer(push))
        check(getattr(lib(), _entry)(ctypes.byref(args), _stream()), _entry)
        return None
    if out is None:
        if accumulate:
            raise ValueError("accumulate=True needs the tensor to add to (out)")
        out = torch.empty((m, n), dtype=x.dtype, device=x.device)
    out2 = out.reshape(-1, out.shape[-1]) if out.dim() != 2 else out
    if out2.shape != (m, n) or out2.stride(1) != 1 or out2.dtype != x.dtype or \
            (m > 1 and out2.stride(0) < n):
        raise ValueError(f"out must be a [{m}, {n}] {x.dtype} tensor with unit column stride")
    if m == 0:
        return out.reshape(*x.shape[:-1], n) if out.is_contiguous() else out
    nbytes = lib().dz_sbmm_workspace_bytes(m, n, k, int(segments.sorted))
    ws = _workspace(x.device, nbytes)
    args = SbmmArgs(
        x=x2.data_ptr(), w_base=base_weight.data_ptr() if base_weight is not None else None,
        qweight=qweight_stacked.data_ptr(), meta=meta_stacked.data_ptr(),
        scales=scales_stacked.data_ptr(),
        qweight_stride=qweight_stacked.stride(0) * 4, meta_stride=meta_stacked.stride(0) * 2,
        scales_stride=scales_stacked.stride(0) * 2,
        segments=segments.buf.data_ptr(), y=out2.data_ptr(),
        M=m, N=n, K=k, num_slots=qweight_stacked.shape[0], bits=bits, dtype=_dtype_code(x),
        tokens_sorted=int(segments.sorted),
        flags=(_lib.DZ_SBMM_ACCUMULATE if accumulate else 0) | (_lib.DZ_SBMM_INPUTS_STABLE if stable else 0),
        workspace=ws.data_ptr(), workspace_bytes=ws.numel(),
        y_stride=max(out2.stride(0), n))
    check(getattr(lib(), _entry)(ctypes.byref(args), _stream()), _entry)
    return out.reshape(*x.shape[:-1], n) if out.is_contiguous() else out


def stream_fence() -> None:
    """Separates earlier writers on the current stream from later `stable=True` SBMM calls."""
    check(lib().dz_stream_fence(_stream()), "dz_stream_fence")


def base_gemm(x: torch.Tensor, base_weight: torch.Tensor,
              out: Optional[torch.Tensor] = None, stable: bool = False) -> torch.Tensor:
    """y = x W^T on the same kernel (every token base-only); the library GEMM for more than
    FUSED_MAX_TOKENS rows, for shapes the kernel does not tile and for 32-bit activations."""
    _need_cuda(x, base_weight)
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    m, k = x2.shape
    n = base_weight.shape[0]
    if m > FUSED_MAX_TOKENS or n % 128 or k % 64 or x.dtype == torch.float32:
        if out is None:
            return torch.matmul(x2, base_weight.t()).reshape(*x.shape[:-1], n)
        torch.matmul(x2, base_weight.t(), out=out.reshape(m, n))
        return out.reshape(*x.shape[:-1], n)
    if out is None:
        out = torch.empty((m, n), dtype=x.dtype, device=x.device)
    if m == 0:
        return out.reshape(*x.shape[:-1], n)
    ws = _workspace(x.device, lib().dz_sbmm_workspace_bytes(m, n, k, 1))
    args = SbmmArgs(x=x2.data_ptr(), w_base=base_weight.data_ptr(), y=out.data_ptr(),
                    M=m, N=n, K=k, num_slots=0, bits=4, dtype=_dtype_code(x), tokens_sorted=1,
                    flags=_lib.DZ_SBMM_INPUTS_STABLE if stable else 0,
                    workspace=ws.data_ptr(), workspace_bytes=ws.numel())
    check(lib().dz_base_gemm(ctypes.byref(args), _stream()), "dz_base_gemm")
    return out.reshape(*x.shape[:-1], n)


_segment_cache = {}


def _segments_for(indices: torch.Tensor, num_slots: int, device) -> Segments:
    """Segment table of `indices`, rebuilt only when the tensor changed: the key is the
    buffer's address and torch's version counter, which every in-place write through torch
    (the `copy_` of the reference's _set_delta_mapping, serving/vllm/delta/models.py:407-430)
    advances.  The cache keeps the tensor alive, so the address cannot be handed to another
    tensor while the entry exists.  All layers of a step therefore share one build, with no
    host synchronisation: whether the batch is sorted is left to the device (x is gathered
    through the table's permutation, which is the identity for a sorted batch)."""
    indices = indices.reshape(-1)
    m = indices.numel()
    key = (device.index, _stream(), num_slots)
    stamp = (indices.data_ptr(), indices._version, m, indices.dtype)
    ent = _segment_cache.get(key)
    if ent is None or ent[0].max_tokens < m:
        ent = [Segments(max(m, 256), num_slots, device), None, None]
        _segment_cache[key] = ent
    if ent[1] != stamp:
        ent[0].build(indices)
        ent[1] = stamp
        ent[2] = indices
    return ent[0]


def apply_delta(x: torch.Tensor, qweight_stacked: torch.Tensor, scales_stacked: torch.Tensor,
                meta_stacked: torch.Tensor, indices: torch.Tensor,
                base_weight: torch.Tensor) -> torch.Tensor:
    """Drop-in for the reference op (serving/vllm/delta/deltazip_marlin.py:10-19).  Enqueues
    device work only: no host synchronisation and no allocation besides the result, so it can
    sit inside a captured decode step as the reference's op does."""
    seg = _segments_for(indices, qweight_stacked.shape[0], x.device)
    return sbmm(x, qweight_stacked, scales_stacked, meta_stacked, seg, base_weight)


# ---------------------------------------------------------------------------
# the "separate base output" form of the op: y += x dequant(delta)^T in place
# ---------------------------------------------------------------------------

def add_delta(y: torch.Tensor, x: torch.Tensor, qweight: torch.Tensor,
              qzeros: Optional[torch.Tensor], scales: torch.Tensor,
              g_idx: Optional[torch.Tensor], indices: torch.Tensor,
              meta: Optional[torch.Tensor] = None) -> torch.Tensor:
    """In place y[i] += x[i] @ dequant(delta[indices[i]])^T, -1 = nothing added: the
    reference's add_delta (serving/vllm/delta/deltazip.py:14-38) on slot-layout stacks
    (`qweight`, `scales`, `meta` as `alloc_slots` makes them; the symmetric zero point and the
    single quantisation group are implicit, so `qzeros` and `g_idx` are accepted and ignored).
    One launch of the SBMM kernel without its base half, adding into y in its epilogue."""
    if meta is None:
        raise ValueError("slot-layout stacks need their 2:4 metadata (meta)")
    x2 = x.reshape(-1, x.shape[-1])
    y2 = y.view(-1, y.shape[-1])
    seg = _segments_for(indices, qweight.shape[0], x.device)
    sbmm(x2, qweight, scales, meta, seg, None, out=y2, accumulate=True)
    return y


def add_delta_slice(y: torch.Tensor, x: torch.Tensor, qweight: torch.Tensor,
                    qzeros: Optional[torch.Tensor], scales: torch.Tensor,
                    g_idx: Optional[torch.Tensor], indices: torch.Tensor, scale: float,
                    y_offset: int, y_slice_size: int, *, buffer: Optional[torch.Tensor] = None,
                    meta: Optional[torch.Tensor] = None) -> torch.Tensor:
    """add_delta into the columns [y_offset, y_offset + y_slice_size) of y
    (serving/vllm/delta/deltazip.py:41-78; `scale` and `buffer` are unused there too).  The
    kernel writes the slice in place through its row stride; `y_offset` must be a multiple
    of 8 elements."""
    if meta is None:
        raise ValueError("slot-layout stacks need their 2:4 metadata (meta)")
    x2 = x.reshape(-1, x.shape[-1])
    y2 = y.view(-1, y.shape[-1])
    if scales.shape[-1] != y_slice_size:
        raise ValueError(f"slice of {y_slice_size} columns, delta stack has {scales.shape[-1]}")
    seg = _segments_for(indices, qweight.shape[0], x.device)
    sbmm(x2, qweight, scales, meta, seg, None, out=y2[:, y_offset:y_offset + y_slice_size],
         accumulate=True)
    return y


def apply_delta_packed_nslice(x: torch.Tensor, qweight_stacked, qzeros_stacked, scales_stacked,
                              g_idx_stacked, indices: torch.Tensor, output: torch.Tensor,
                              output_slices, meta_stacked=None) -> torch.Tensor:
    """Merged layers (q/k/v, gate/up) whose sub-layers keep separate stacks: one add_delta_slice
    per output slice (serving/vllm/delta/deltazip.py:108-153)."""
    if meta_stacked is None:
        raise ValueError("slot-layout stacks need their 2:4 metadata (meta_stacked)")
    x2 = x.reshape(-1, x.shape[-1])
    out2 = output.view(-1, output.shape[-1])
    offset = 0
    for i, width in enumerate(output_slices):
        add_delta_slice(out2, x2, qweight_stacked[i], qzeros_stacked[i] if qzeros_stacked else None,
                        scales_stacked[i], g_idx_stacked[i] if g_idx_stacked else None,
                        indices, 1.0, offset, width, meta=meta_stacked[i])
        offset += width
    return output


# ---------------------------------------------------------------------------
# per-delta embedding / lm_head (full replacement tables, not additive deltas)
# ---------------------------------------------------------------------------

def _index_code(indices: torch.Tensor) -> int:
    if indices.dtype == torch.int64:
        return _lib.DZ_INDEX_I64
    if indices.dtype == torch.int32:
        return _lib.DZ_INDEX_I32
    raise ValueError("indices must be int32 or int64")


def apply_delta_embed(x: torch.Tensor, delta_weights: torch.Tensor, indices: torch.Tensor,
                      base_weight: torch.Tensor) -> torch.Tensor:
    """Embedding lookup with a replacement table per delta (reference:
    serving/vllm/delta/deltazip_marlin.py:56-86).  x: token ids [M]; delta_weights:
    [D, vocab, hidden]; indices: slot per token (-1 = base_weight [vocab, hidden])."""
    _need_cuda(x, delta_weights, indices, base_weight)
    tokens = x.reshape(-1).to(torch.int64).contiguous()
    indices = indices.reshape(-1).contiguous()
    m = tokens.numel()
    vocab, hidden = base_weight.shape
    out = torch.empty((m, hidden), dtype=base_weight.dtype, device=base_weight.device)
    d = delta_weights.shape[0] if delta_weights is not None and delta_weights.numel() else 0
    check(lib().dz_delta_embedding(
        tokens.data_ptr(), indices.data_ptr(), _index_code(indices), m, hidden,
        base_weight.data_ptr(), delta_weights.data_ptr() if d else None,
        delta_weights.stride(0) * delta_weights.element_size() if d else 0, d, vocab,
        out.data_ptr(), None, _stream()), "dz_delta_embedding")
    return out.reshape(*x.shape, hidden)


_gg_ws = {}


def grouped_gemm(x: torch.Tensor, delta_weights: Optional[torch.Tensor], segments: Segments,
                 base_weight: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y[i] = x[i] T^T with T = base_weight [V, K] for rows of slot -1 and delta_weights[slot]
    ([D, V, K], dense) otherwise, in one launch per 128 rows (dz_grouped_gemm)."""
    _need_cuda(x, delta_weights, base_weight)
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    m, k = x2.shape
    v = base_weight.shape[0]
    d = delta_weights.shape[0] if delta_weights is not None and delta_weights.numel() else 0
    if d and (not delta_weights.is_contiguous() or tuple(delta_weights.shape[1:]) != (v, k)):
        raise ValueError("delta_weights must be a contiguous [D, V, K] stack matching base_weight")
    if segments.m != m or segments.num_slots != d:
        raise ValueError("segment table does not match the batch / the number of slots")
    if out is None:
        out = torch.empty((m, v), dtype=x.dtype, device=x.device)
    if m == 0:
        return out.reshape(*x.shape[:-1], v)
    need = lib().dz_grouped_gemm_workspace_bytes(m, k, int(segments.sorted))
    key = (x.device.index, _stream())
    ws = _gg_ws.get(key)
    if ws is None or ws.numel() < need:
        ws = torch.zeros(max(need, 4096), dtype=torch.uint8, device=x.device)
        _gg_ws[key] = ws
    check(lib().dz_grouped_gemm(
        x2.data_ptr(), base_weight.data_ptr(), delta_weights.data_ptr() if d else None,
        v * k * 2 if d else 0, segments.buf.data_ptr(), out.data_ptr(), m, v, k, d, _dtype_code(x),
        int(segments.sorted), out.stride(0), ws.data_ptr(), ws.numel(), _stream()), "dz_grouped_gemm")
    return out.reshape(*x.shape[:-1], v)


def apply_delta_uncompressed(x: torch.Tensor, delta_weights: torch.Tensor, indices: torch.Tensor,
                             base_embedding: torch.Tensor) -> torch.Tensor:
    """lm_head with a full replacement matrix per delta: rows with slot d are multiplied by
    delta_weights[d], rows with -1 by base_embedding (reference:
    serving/vllm/delta/deltazip_marlin.py:21-53, a host loop over the distinct ids).  Here one
    grouped launch on the dense tcgen05 GEMM, no host synchronisation; the vocabulary rows must
    be a multiple of 128 (pad the matrices otherwise)."""
    _need_cuda(x, delta_weights, indices, base_embedding)
    d = delta_weights.shape[0] if delta_weights is not None and delta_weights.numel() else 0
    seg = _segments_for(indices, d, x.device)
    return grouped_gemm(x, delta_weights if d else None, seg, base_embedding.contiguous())


# ---------------------------------------------------------------------------
# the steps between the SBMM calls of a decoder layer (decode time)
# ---------------------------------------------------------------------------

def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float,
             residual: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out = rmsnorm(x) * weight; with `residual`, first residual += x (in place) and the norm is
    taken of the sum -- the reference's RMSNorm.forward with and without residual
    (serving/vllm/model_executor/layers/layernorm.py:47-66)."""
    _need_cuda(x, weight, residual)
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    if out is None:
        out = torch.empty_like(x2)
    if residual is not None and not residual.is_contiguous():
        raise ValueError("residual must be contiguous (it is updated in place)")
    check(lib().dz_rms_norm(x2.data_ptr(), residual.data_ptr() if residual is not None else None,
                            weight.data_ptr(), out.data_ptr(), x2.shape[0], x2.shape[1], float(eps),
                            _dtype_code(x), _stream()), "dz_rms_norm")
    return out.reshape(x.shape)


def silu_and_mul(x: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """silu(x[..., :I]) * x[..., I:] (serving/vllm/model_executor/layers/activation.py:17-40)."""
    _need_cuda(x)
    x2 = x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    inter = x2.shape[1] // 2
    if out is None:
        out = torch.empty((x2.shape[0], inter), dtype=x.dtype, device=x.device)
    check(lib().dz_silu_and_mul(x2.data_ptr(), out.data_ptr(), x2.shape[0], inter, _dtype_code(x),
                                _stream()), "dz_silu_and_mul")
    return out.reshape(*x.shape[:-1], inter)


def rotary_and_cache(qkv: torch.Tensor, positions: torch.Tensor, q_heads: int, kv_heads: int,
                     rope_theta: float, k_cache: Optional[torch.Tensor] = None,
                     v_cache: Optional[torch.Tensor] = None,
                     slot_mapping: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rotary embedding in place on the q and k heads of fused qkv rows [M, (q+2kv)*128] and, when
    a cache is given, the write of k / v to cache slot `slot_mapping[token]`."""
    _need_cuda(qkv, positions, k_cache, v_cache, slot_mapping)
    if not qkv.is_contiguous() or positions.dtype != torch.int64:
        raise ValueError("qkv must be contiguous and positions int64")
    m = qkv.numel() // qkv.shape[-1]
    if slot_mapping is not None and slot_mapping.dtype != torch.int64:
        raise ValueError("slot_mapping must be int64")
    check(lib().dz_rotary_and_cache(
        qkv.data_ptr(), positions.data_ptr(),
        slot_mapping.data_ptr() if slot_mapping is not None else None,
        k_cache.data_ptr() if k_cache is not None else None,
        v_cache.data_ptr() if v_cache is not None else None,
        m, q_heads, kv_heads, qkv.shape[-1] // (q_heads + 2 * kv_heads), float(rope_theta),
        _dtype_code(qkv), _stream()), "dz_rotary_and_cache")
    return qkv


_attn_ws = {}


def paged_attention_decode(qkv: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                           block_tables: torch.Tensor, seq_lens: torch.Tensor, q_heads: int,
                           kv_heads: int, block_size: int, scale: float, splits: int = 1,
                           out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One query token per sequence (the q part of fused qkv rows [B, (q+2kv)*128]) against the
    paged cache; returns [B, q_heads*128]."""
    _need_cuda(qkv, k_cache, v_cache, block_tables, seq_lens)
    b = qkv.shape[0]
    if block_tables.dtype != torch.int32 or seq_lens.dtype != torch.int32 or not block_tables.is_contiguous():
        raise ValueError("block_tables / seq_lens must be contiguous int32")
    if out is None:
        out = torch.empty((b, q_heads * 128), dtype=qkv.dtype, device=qkv.device)
    ws_ptr, ws_bytes = None, 0
    if splits > 1:
        need = lib().dz_paged_attention_workspace_bytes(b, q_heads, kv_heads, splits)
        key = (qkv.device.index, _stream())
        ws = _attn_ws.get(key)
        if ws is None or ws.numel() < need:
            ws = torch.zeros(need, dtype=torch.uint8, device=qkv.device)
            _attn_ws[key] = ws
        ws_ptr, ws_bytes = ws.data_ptr(), ws.numel()
    check(lib().dz_paged_attention_decode(
        qkv.data_ptr(), qkv.stride(0), out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
        block_tables.data_ptr(), block_tables.shape[1], seq_lens.data_ptr(), b, q_heads, kv_heads,
        128, block_size, float(scale), splits, ws_ptr, ws_bytes, _dtype_code(qkv), _stream()),
        "dz_paged_attention_decode")
    return out


# ---------------------------------------------------------------------------
# decoder steps with a 32-bit residual stream, sliding-window attention over a ring of cache
# blocks, matrix-memory recurrence.  16-bit or 32-bit activations, any sizes.
# ---------------------------------------------------------------------------

ACTIVATIONS = {"silu": _lib.DZ_ACT_SILU, "gelu_tanh": _lib.DZ_ACT_GELU_TANH, "relu2": _lib.DZ_ACT_RELU2}
_scratch = {}


def _zeroed_scratch(kind: str, device, nbytes: int) -> Optional[torch.Tensor]:
    """Grow-only scratch per (kernel, device, stream), zero-filled when it is made: the kernels
    leave their tickets at zero."""
    if nbytes == 0:
        return None
    key = (kind, device.index, _stream())
    buf = _scratch.get(key)
    if buf is None or buf.numel() < nbytes:
        buf = torch.zeros(nbytes, dtype=torch.uint8, device=device)
        _scratch[key] = buf
    return buf


def _any_dtype_code(t: torch.Tensor) -> int:
    return _lib.DZ_DTYPE_F32 if t.dtype == torch.float32 else _dtype_code(t)


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def matmul_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """x W^T with a 32-bit result (library GEMM, 32-bit accumulation)."""
    _need_cuda(x, weight)
    if x.dtype == torch.float32:
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out_dtype=torch.float32)


def embed_norm(tokens: torch.Tensor, table: torch.Tensor, weight: Optional[torch.Tensor], eps: float,
               weight_offset: float = 0.0, copy: Optional[torch.Tensor] = None, scale: float = 1.0) -> torch.Tensor:
    """norm(scale * table[tokens]) as a 32-bit residual [M, width], without the norm when `weight` is None;
    `copy`: a column slice of a wider matrix that gets the same rounded to the table's type."""
    _need_cuda(tokens, table, weight, copy)
    m, (vocab, width) = tokens.numel(), table.shape
    residual = torch.empty((m, width), dtype=torch.float32, device=table.device)
    if copy is not None and (copy.dtype != table.dtype or copy.shape != (m, width) or copy.stride(1) != 1):
        raise ValueError("copy must be a [tokens, width] slice of the table's type with unit column stride")
    check(lib().dz_embed_norm(tokens.data_ptr(), table.data_ptr(), vocab, float(scale), _ptr(weight), float(weight_offset),
                              residual.data_ptr(), _ptr(copy), copy.stride(0) if copy is not None else 0, m, width,
                              float(eps), _any_dtype_code(table), _stream()), "dz_embed_norm")
    return residual


class Update(NamedTuple):
    """What a sublayer adds to the residual: a matrix, and optionally rows `index` [M, n] (int32, negative:
    none) of a second one that are summed into each of its rows."""
    matrix: Optional[torch.Tensor]
    rows: Optional[torch.Tensor] = None
    index: Optional[torch.Tensor] = None

    def dense(self) -> torch.Tensor:
        """The whole update in 32 bits (for inspection; residual_norm sums it on its way)."""
        picked = torch.where(self.index[..., None] >= 0, self.rows[self.index.clamp(min=0).long()].float(), 0).sum(1)
        return picked if self.matrix is None else picked + self.matrix


def residual_norm(residual: torch.Tensor, delta, weight: Optional[torch.Tensor], eps: float,
                  dtype: torch.dtype, weight_offset: float = 0.0, vec: Optional[torch.Tensor] = None,
                  replace: bool = False, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """residual (32-bit, in place) += delta + vec, or = with `replace`; returns norm(residual) in
    `dtype`, or the residual rounded to it when `weight` is None.  `delta`: a matrix, an Update or None."""
    delta, rows, index = delta if isinstance(delta, Update) else (delta, None, None)
    _need_cuda(residual, delta, weight, vec, out, rows, index)
    m, width = residual.shape
    if out is None:
        out = torch.empty((m, width), dtype=dtype, device=residual.device)
    if residual.dtype != torch.float32 or not residual.is_contiguous() or out.stride(1) != 1:
        raise ValueError("the residual is a contiguous float32 matrix, out has unit column stride")
    if delta is not None and (delta.shape != residual.shape or not delta.is_contiguous()):
        raise ValueError("delta must be a contiguous matrix of the residual's shape")
    if rows is not None and (rows.dtype != out.dtype or rows.shape[1] != width or not rows.is_contiguous() or
                             index.dtype != torch.int32 or index.shape[0] != m or not index.is_contiguous()):
        raise ValueError("summed rows are contiguous, of the output's type, with an int32 index per row")
    check(lib().dz_residual_norm(residual.data_ptr(), _ptr(delta), _any_dtype_code(delta) if delta is not None else 0,
                                 int(replace), _ptr(vec), _ptr(rows), _ptr(index), index.shape[1] if rows is not None else 0,
                                 _ptr(weight), float(weight_offset), out.data_ptr(),
                                 out.stride(0) if m > 1 else max(out.stride(0), width), m, width, float(eps),
                                 _any_dtype_code(out), _stream()), "dz_residual_norm")
    return out


def act(x: torch.Tensor, activation: str, inter: Optional[int] = None) -> torch.Tensor:
    """act(x[:, :inter]); columns beyond are padding."""
    _need_cuda(x)
    inter = inter or x.shape[1]
    out = torch.empty((x.shape[0], inter), dtype=x.dtype, device=x.device)
    check(lib().dz_act(x.data_ptr(), x.stride(0), out.data_ptr(), x.shape[0], inter, ACTIVATIONS[activation],
                       _any_dtype_code(x), _stream()), "dz_act")
    return out


def gated_act(x: torch.Tensor, activation: str, inter: Optional[int] = None) -> torch.Tensor:
    """act(x[:, :inter]) * x[:, inter:2 inter]; columns beyond are padding."""
    _need_cuda(x)
    inter = inter or x.shape[1] // 2
    out = torch.empty((x.shape[0], inter), dtype=x.dtype, device=x.device)
    check(lib().dz_gated_act(x.data_ptr(), x.stride(0), out.data_ptr(), x.shape[0], inter, ACTIVATIONS[activation],
                             _any_dtype_code(x), _stream()), "dz_gated_act")
    return out


def qk_norm(qkv: torch.Tensor, wq: torch.Tensor, wk: torch.Tensor, v_width: int, eps: float,
            k_cache: Optional[torch.Tensor] = None, v_cache: Optional[torch.Tensor] = None,
            slot_mapping: Optional[torch.Tensor] = None) -> torch.Tensor:
    """RMS norm of the query row and of the key row of [q | k | v | ...] rows in place (each over all
    its heads); with `slot_mapping` the key and value also go to the cache."""
    _need_cuda(qkv, wq, wk, k_cache, v_cache, slot_mapping)
    check(lib().dz_qk_norm(qkv.data_ptr(), qkv.stride(0), wq.numel(), wk.numel(), v_width, wq.data_ptr(),
                           wk.data_ptr(), float(eps), _ptr(k_cache), _ptr(v_cache), _ptr(slot_mapping), qkv.shape[0],
                           _any_dtype_code(qkv), _stream()), "dz_qk_norm")
    return qkv


def kv_append(qkv: torch.Tensor, k_off: int, k_cache: torch.Tensor, v_cache: torch.Tensor,
              slot_mapping: torch.Tensor) -> None:
    """Copies the key and value parts of every row to its cache slot (< 0: not kept)."""
    _need_cuda(qkv, k_cache, v_cache, slot_mapping)
    check(lib().dz_kv_append(qkv.data_ptr(), qkv.stride(0), k_off, k_cache[0].numel(), v_cache[0].numel(),
                             k_cache.data_ptr(), v_cache.data_ptr(), slot_mapping.data_ptr(), qkv.shape[0],
                             _any_dtype_code(qkv), _stream()), "dz_kv_append")


def window_attention(qkv: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor,
                     q_starts: torch.Tensor, ctx_lens: torch.Tensor, max_query: int, decode: bool, heads: int,
                     block_size: int, scale: float, window: int, bias: Optional[torch.Tensor] = None,
                     splits: int = 0, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of [q | k | v | ...] rows with a sliding window and an additive bias per distance
    ([heads, distances] float32); see dz_window_attention.  `splits` 0: enough CTAs to fill the GPU.
    `sink` [heads] float32: one more score per row, without a key or a value."""
    _need_cuda(qkv, k_cache, v_cache, block_tables, q_starts, ctx_lens, bias, sink)
    kv_heads, dim, vdim = k_cache.shape[1], k_cache.shape[2], v_cache.shape[2]
    rows, seqs = qkv.shape[0], ctx_lens.shape[0]
    if any(t.dtype != torch.int32 or not t.is_contiguous() for t in (block_tables, q_starts, ctx_lens)):
        raise ValueError("block_tables / q_starts / ctx_lens must be contiguous int32")
    out = torch.empty((rows, heads * vdim), dtype=qkv.dtype, device=qkv.device)
    if not decode:
        splits = 1
    elif splits <= 0:
        ratio = heads // kv_heads
        ctas = seqs * kv_heads * ((ratio + 3) // 4 if ratio > 2 else 1)
        most = (window + 63) // 64 if window > 0 else 8
        splits = max(1, min(8, most, 296 // max(1, ctas)))
    ws = _zeroed_scratch("window_attention", qkv.device,
                         lib().dz_window_attention_workspace_bytes(seqs, heads, kv_heads, vdim, splits))
    args = _lib.WindowAttentionArgs(
        qkv=qkv.data_ptr(), row_stride=qkv.stride(0), k_off=heads * dim, v_off=(heads + kv_heads) * dim,
        out=out.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(),
        block_tables=block_tables.data_ptr(), ring_blocks=block_tables.shape[1], block_size=block_size,
        q_starts=q_starts.data_ptr(), ctx_lens=ctx_lens.data_ptr(), num_seqs=seqs, rows=rows, max_q=max_query,
        decode=int(decode), heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(scale), window=window,
        bias=_ptr(bias), bias_len=bias.shape[1] if bias is not None else 0, splits=splits,
        workspace=_ptr(ws), workspace_bytes=ws.numel() if ws is not None else 0, dtype=_any_dtype_code(qkv),
        sink=_ptr(sink))
    check(lib().dz_window_attention(ctypes.byref(args), _stream()), "dz_window_attention")
    return out


def rows_attention(q: torch.Tensor, kv: torch.Tensor, q_starts: torch.Tensor, ctx_lens: torch.Tensor,
                   kv_starts: torch.Tensor, max_query: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                   sink: Optional[torch.Tensor] = None, window: int = 0) -> torch.Tensor:
    """The same attention with every key and value of a sequence in rows [k | v | ...] of their own, its
    position t in row kv_starts[sequence] + t (dz_window_attention with `kv`)."""
    _need_cuda(q, kv, q_starts, ctx_lens, kv_starts, sink)
    if any(t.dtype != torch.int32 or not t.is_contiguous() for t in (q_starts, ctx_lens, kv_starts)):
        raise ValueError("q_starts / ctx_lens / kv_starts must be contiguous int32")
    rows, seqs = q.shape[0], ctx_lens.shape[0]
    out = torch.empty((rows, heads * vdim), dtype=q.dtype, device=q.device)
    ws = _zeroed_scratch("window_attention", q.device, lib().dz_window_attention_workspace_bytes(seqs, heads, kv_heads, vdim, 1))
    args = _lib.WindowAttentionArgs(
        qkv=q.data_ptr(), row_stride=q.stride(0), k_off=0, v_off=kv_heads * dim, out=out.data_ptr(),
        q_starts=q_starts.data_ptr(), ctx_lens=ctx_lens.data_ptr(), num_seqs=seqs, rows=rows, max_q=max_query, decode=0,
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(scale), window=window, splits=1,
        workspace=ws.data_ptr(), workspace_bytes=ws.numel(), dtype=_any_dtype_code(q), sink=_ptr(sink), kv=kv.data_ptr(),
        kv_stride=kv.stride(0), kv_starts=kv_starts.data_ptr(), kv_rows=kv.shape[0])
    check(lib().dz_window_attention(ctypes.byref(args), _stream()), "dz_window_attention")
    return out


# ---------------------------------------------------------------------------
# attention over a cached latent, one row [latent | shared rotated key part] per token
# ---------------------------------------------------------------------------

def latent_rows(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, heads: int, dim: int, rot: int, rank: int,
                q_out: Optional[torch.Tensor] = None, l_off: int = -1, norm_weight: Optional[torch.Tensor] = None,
                eps: float = 0.0, cache: Optional[torch.Tensor] = None, slot_mapping: Optional[torch.Tensor] = None) -> None:
    """Rotates the queries' last `rot` components (in place, or into the end of q_out's rows) and, with
    l_off >= 0, writes the rows' normed latent and rotated key part to the cache (dz_latent_rows)."""
    _need_cuda(x, positions, freq, q_out, norm_weight, cache, slot_mapping)
    if positions.dtype != torch.int64 or freq.dtype != torch.float64 or freq.numel() != rot // 2:
        raise ValueError("positions are int64, freq holds rot / 2 float64 values")
    if q_out is not None and (q_out.shape != (x.shape[0], heads, rank + rot) or not q_out.is_contiguous()):
        raise ValueError("q_out must be a contiguous [rows, heads, rank + rot]")
    args = _lib.LatentRowsArgs(
        x=x.data_ptr(), row_stride=x.stride(0), positions=positions.data_ptr(), freq=freq.data_ptr(), rows=x.shape[0],
        heads=heads, dim=dim, rot=rot, q_out=_ptr(q_out), l_off=l_off, rank=rank, norm_weight=_ptr(norm_weight),
        eps=float(eps), cache=_ptr(cache), slots=_ptr(slot_mapping), dtype=_any_dtype_code(x))
    check(lib().dz_latent_rows(ctypes.byref(args), _stream()), "dz_latent_rows")


def latent_gather(cache: torch.Tensor, block_tables: torch.Tensor, block_size: int, starts: torch.Tensor, total: int,
                  max_len: int) -> torch.Tensor:
    """Cached rows of positions 0, 1, ... of every sequence, sequence after sequence: [total, row size]."""
    _need_cuda(cache, block_tables, starts)
    size = cache.shape[-1]
    out = torch.empty((total, size), dtype=cache.dtype, device=cache.device)
    check(lib().dz_latent_gather(cache.data_ptr(), block_tables.data_ptr(), block_tables.shape[1], block_size,
                                 starts.data_ptr(), block_tables.shape[0], max_len, out.data_ptr(), size,
                                 _any_dtype_code(cache), _stream()), "dz_latent_gather")
    return out


@functools.lru_cache(maxsize=4096)
def _balanced_splits(ctas: int, most: int, sms: int = 148) -> int:
    """Splits of every CTA's work with the fullest last wave; fewer where that gains little."""
    best, score = 1, 0.0
    for s in range(1, max(1, most) + 1):
        full = ctas * s / (-(-ctas * s // sms) * sms)
        if full > score * 1.05:
            best, score = s, full
    return best


def latent_attention(q: torch.Tensor, cache: torch.Tensor, block_tables: torch.Tensor, q_starts: torch.Tensor,
                     ctx_lens: torch.Tensor, rank: int, block_size: int, scale: float, sink: Optional[torch.Tensor] = None,
                     splits: int = 0) -> torch.Tensor:
    """q [rows, heads, rank + rot] against the cached rows up to each row's position; returns the weighted
    latents [rows, heads, rank] (dz_latent_attention).  `splits` 0: chosen to fill the GPU."""
    _need_cuda(q, cache, block_tables, q_starts, ctx_lens, sink)
    rows, heads, size = q.shape
    if not q.is_contiguous() or cache.shape[-1] != size or not cache.is_contiguous():
        raise ValueError("q is a contiguous [rows, heads, rank + rot] with the cache's row size")
    if any(t.dtype != torch.int32 or not t.is_contiguous() for t in (block_tables, q_starts, ctx_lens)):
        raise ValueError("block_tables / q_starts / ctx_lens must be contiguous int32")
    code = _any_dtype_code(q)
    ctas = lib().dz_latent_attention_ctas(rows, heads, rank, size - rank, code)
    if ctas == 0:
        splits = 1
    elif splits <= 0:
        splits = _balanced_splits(ctas, min(16, -(-block_tables.shape[1] * block_size // 256)))
        splits = splits if ctas <= 65536 else 1
    out = torch.empty((rows, heads, rank), dtype=q.dtype, device=q.device)
    ws = _zeroed_scratch("latent_attention", q.device, lib().dz_latent_attention_workspace_bytes(rows, heads, rank, splits))
    args = _lib.LatentAttentionArgs(
        q=q.data_ptr(), cache=cache.data_ptr(), block_tables=block_tables.data_ptr(), table_width=block_tables.shape[1],
        block_size=block_size, q_starts=q_starts.data_ptr(), ctx_lens=ctx_lens.data_ptr(), num_seqs=ctx_lens.shape[0],
        rows=rows, heads=heads, rank=rank, rot=size - rank, scale=float(scale), sink=_ptr(sink), out=out.data_ptr(),
        splits=splits, workspace=_ptr(ws), workspace_bytes=ws.numel() if ws is not None else 0, dtype=code,
        cache_rows=cache.shape[0], status=_zeroed_scratch("status", q.device, 256).data_ptr())
    check(lib().dz_latent_attention(ctypes.byref(args), _stream()), "dz_latent_attention")
    return out


# ---------------------------------------------------------------------------
# recurrent layers
# ---------------------------------------------------------------------------

LIGHTNING_POWERS = 65                   # decay^0 ... decay^64 per head


def lightning_chunk_supported(dim: int, vdim: int, dtype: torch.dtype) -> bool:
    code = {torch.float16: _lib.DZ_DTYPE_F16, torch.bfloat16: _lib.DZ_DTYPE_BF16}.get(dtype, _lib.DZ_DTYPE_F32)
    return bool(lib().dz_lightning_chunk_supported(dim, vdim, code))


def lightning(x: torch.Tensor, powers: torch.Tensor, norm_weight: torch.Tensor, S: torch.Tensor, slots: torch.Tensor,
              q_starts: torch.Tensor, ctx_lens: torch.Tensor, eps: float, chunkwise: bool) -> torch.Tensor:
    """Linear attention with a constant decay, norm over all heads and output gate over rows
    [q | k | v | g | ...]; the states in slots `slots` are updated in place (dz_lightning)."""
    _need_cuda(x, powers, norm_weight, S, slots, q_starts, ctx_lens)
    heads, dim, vdim = S.shape[1:]
    rows, seqs = x.shape[0], ctx_lens.shape[0]
    if any(t.dtype != torch.int32 or not t.is_contiguous() for t in (slots, q_starts, ctx_lens)):
        raise ValueError("slots / q_starts / ctx_lens must be contiguous int32")
    if powers.shape != (heads, LIGHTNING_POWERS) or powers.dtype != torch.float32 or not powers.is_contiguous():
        raise ValueError("powers must be a contiguous float32 [heads, 65]")
    out = torch.empty((rows, heads * vdim), dtype=x.dtype, device=x.device)
    ws = _zeroed_scratch("lightning", x.device, lib().dz_lightning_workspace_bytes(rows, seqs, heads, vdim, int(chunkwise)))
    args = _lib.LightningArgs(
        x=x.data_ptr(), row_stride=x.stride(0), k_off=heads * dim, v_off=2 * heads * dim,
        g_off=2 * heads * dim + heads * vdim, powers=powers.data_ptr(), norm_weight=norm_weight.data_ptr(),
        eps=float(eps), out=out.data_ptr(), S=S.data_ptr(), slots=slots.data_ptr(), q_starts=q_starts.data_ptr(),
        ctx_lens=ctx_lens.data_ptr(), num_seqs=seqs, rows=rows, heads=heads, dim=dim, vdim=vdim, chunkwise=int(chunkwise),
        workspace=_ptr(ws), workspace_bytes=ws.numel() if ws is not None else 0, dtype=_any_dtype_code(x))
    check(lib().dz_lightning(ctypes.byref(args), _stream()), "dz_lightning")
    return out


def mlstm_chunk_supported(dim: int, vdim: int, dtype: torch.dtype) -> bool:
    code = {torch.float16: _lib.DZ_DTYPE_F16, torch.bfloat16: _lib.DZ_DTYPE_BF16}.get(dtype, _lib.DZ_DTYPE_F32)
    return bool(lib().dz_mlstm_chunk_supported(dim, vdim, code))


def mlstm(x: torch.Tensor, h: torch.Tensor, w_if: torch.Tensor, b_if: torch.Tensor, norm_weight: torch.Tensor,
          S: torch.Tensor, n: torch.Tensor, m: torch.Tensor, slots: torch.Tensor, q_starts: torch.Tensor,
          ctx_lens: torch.Tensor, gate_cap: float, scale: float, eps: float, chunkwise: bool) -> torch.Tensor:
    """Matrix-memory recurrence, head norm and output gate over rows [q | k | v | g | ...]; the states
    in slots `slots` are updated in place (dz_mlstm).  Returns [rows, heads * vdim]."""
    _need_cuda(x, h, w_if, b_if, norm_weight, S, n, m, slots, q_starts, ctx_lens)
    heads, dim, vdim = S.shape[1:]
    rows, seqs = x.shape[0], ctx_lens.shape[0]
    if any(t.dtype != torch.int32 or not t.is_contiguous() for t in (slots, q_starts, ctx_lens)):
        raise ValueError("slots / q_starts / ctx_lens must be contiguous int32")
    out = torch.empty((rows, heads * vdim), dtype=x.dtype, device=x.device)
    pre = matmul_f32(h, w_if) if chunkwise else None
    ws = _zeroed_scratch("mlstm", x.device, lib().dz_mlstm_workspace_bytes(seqs, heads)) if chunkwise else None
    args = _lib.MlstmArgs(
        x=x.data_ptr(), row_stride=x.stride(0), k_off=heads * dim, v_off=2 * heads * dim,
        g_off=2 * heads * dim + heads * vdim, h=h.data_ptr(), w_if=w_if.data_ptr(), b_if=b_if.data_ptr(),
        pre_if=_ptr(pre), width=h.shape[1], cap=float(gate_cap), scale=float(scale),
        norm_weight=norm_weight.data_ptr(), eps=float(eps), out=out.data_ptr(), S=S.data_ptr(), n=n.data_ptr(),
        m=m.data_ptr(), slots=slots.data_ptr(), q_starts=q_starts.data_ptr(), ctx_lens=ctx_lens.data_ptr(),
        num_seqs=seqs, rows=rows, heads=heads, dim=dim, vdim=vdim, chunkwise=int(chunkwise),
        workspace=_ptr(ws), workspace_bytes=ws.numel() if ws is not None else 0, dtype=_any_dtype_code(x))
    check(lib().dz_mlstm(ctypes.byref(args), _stream()), "dz_mlstm")
    return out


# ---------------------------------------------------------------------------
# routed experts
# ---------------------------------------------------------------------------

class Routing(NamedTuple):
    """Entries (token, choice) of a batch in expert order."""
    ids: torch.Tensor                   # int32 [M, top] chosen experts
    scores: torch.Tensor                # float32 [M, top]
    offsets: torch.Tensor               # int32 [experts + 1] first sorted row of every expert
    place: torch.Tensor                 # int32 [M, top] sorted row of an entry
    order: torch.Tensor                 # int32 [M * top] entry of a sorted row
    sorted_scores: torch.Tensor         # float32 [M * top]


def moe_route(logits: torch.Tensor, top: int) -> Routing:
    """The `top` experts of every token by sigmoid(logits), and the batch's entries sorted by expert."""
    _need_cuda(logits)
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise ValueError("router logits are contiguous float32")
    m, experts = logits.shape
    dev, i32 = logits.device, torch.int32
    ids, place = (torch.empty((m, top), dtype=i32, device=dev) for _ in range(2))
    scores = torch.empty((m, top), dtype=torch.float32, device=dev)
    offsets, order = torch.empty(experts + 1, dtype=i32, device=dev), torch.empty(m * top, dtype=i32, device=dev)
    by_expert = torch.empty(m * top, dtype=torch.float32, device=dev)
    check(lib().dz_moe_route(logits.data_ptr(), m, experts, top, ids.data_ptr(), scores.data_ptr(), _stream()), "dz_moe_route")
    check(lib().dz_moe_sort(ids.data_ptr(), scores.data_ptr(), m * top, experts, offsets.data_ptr(), place.data_ptr(),
                            order.data_ptr(), by_expert.data_ptr(), _stream()), "dz_moe_sort")
    return Routing(ids, scores, offsets, place, order, by_expert)


def moe_gather(x: torch.Tensor, routing: Routing) -> torch.Tensor:
    """The entries' token rows in expert order."""
    _need_cuda(x)
    entries, top = routing.order.numel(), routing.ids.shape[1]
    out = torch.empty((entries, x.shape[1]), dtype=x.dtype, device=x.device)
    check(lib().dz_moe_gather(x.data_ptr(), routing.order.data_ptr(), entries, top, out.data_ptr(), x.shape[1],
                              _any_dtype_code(x), _stream()), "dz_moe_gather")
    return out


def moe_gemm(x: torch.Tensor, weights: torch.Tensor, offsets: torch.Tensor, scale: Optional[torch.Tensor] = None,
             activation: Optional[str] = None) -> torch.Tensor:
    """act(scale * (x W_e^T)) for rows x in expert order, weights [experts, N, K]."""
    _need_cuda(x, weights, offsets, scale)
    experts, n, k = weights.shape
    rows = x.shape[0]
    if x.shape[1] != k or not x.is_contiguous() or not weights.is_contiguous() or x.dtype != weights.dtype:
        raise ValueError("x [rows, K] and weights [experts, N, K] must be contiguous and of one type")
    out = torch.empty((rows, n), dtype=x.dtype, device=x.device)
    status = _zeroed_scratch("status", x.device, 256)
    check(lib().dz_moe_gemm(x.data_ptr(), weights.data_ptr(), offsets.data_ptr(), _ptr(scale), out.data_ptr(), rows, n, k,
                            experts, ACTIVATIONS[activation] if activation else _lib.DZ_ACT_NONE, -(-rows // experts),
                            _any_dtype_code(x), status.data_ptr(), _stream()), "dz_moe_gemm")
    return out
