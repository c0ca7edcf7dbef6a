"""Products of a few rows with many small matrices, each row set with its own (``csrc/skinny_group.cu``).

* ``head_products``: every row with every head's matrix (per-head projections of a decoding step).
* ``grouped_rows``: rows sorted by group, each group with its matrix, optionally with a gated activation on
  the result (mixture of experts with few tokens).
"""

from __future__ import annotations

import ctypes
from typing import Optional

import torch

from axlearn_b200.ops.hyper_ops import _GATE_KINDS, Gate, gate_values

Tensor = torch.Tensor


class _Args(ctypes.Structure):
    """Mirrors ``axb::SkinnyArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in ("x", "w", "out", "offsets", "row_out")] + [
        (n, ctypes.c_int64) for n in ("x_row", "x_group", "w_row", "w_group", "out_row", "out_group")] + [
        (n, ctypes.c_int) for n in ("rows", "groups", "n", "k", "up_off", "gate_kind", "act_bf16")] + [
        ("limit", ctypes.c_float), ("alpha", ctypes.c_float)]


_signatures_set = False


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        h.axb_skinny_group.argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
        h.axb_skinny_group.restype = ctypes.c_int
        _signatures_set = True
    return h


def _launch(a: _Args) -> None:
    from axlearn_b200.ops import cuda_ops

    cuda_ops._check(_lib().axb_skinny_group(ctypes.byref(a), cuda_ops._stream()), "axb_skinny_group")  # pylint: disable=protected-access


def head_products(x: Tensor, w: Tensor, out: Tensor) -> None:
    """``out[r, h, :] = w[h] @ x[r, h, :]``: views ``x [R, H, K]``, ``w [H, N, K]``, ``out [R, H, N]`` whose last
    axes are contiguous (CUDA, one dtype)."""
    rows, heads, k = x.shape
    n = w.shape[1]
    assert w.shape == (heads, n, k) and out.shape == (rows, heads, n), (x.shape, w.shape, out.shape)
    if x.dtype == torch.float32:
        out.copy_(torch.einsum("rhk,hnk->rhn", x, w))
        return
    a = _Args()
    a.x, a.w, a.out = x.data_ptr(), w.data_ptr(), out.data_ptr()
    a.x_row, a.x_group, a.w_row, a.w_group = x.stride(0), x.stride(1), w.stride(1), w.stride(0)
    a.out_row, a.out_group = out.stride(0), out.stride(1)
    a.rows, a.groups, a.n, a.k, a.up_off, a.gate_kind, a.act_bf16 = rows, heads, n, k, 0, -1, 1
    _launch(a)


def grouped_rows(x: Tensor, w: Tensor, offsets: Tensor, out: Tensor, *, n: int, k: int, row_out: Optional[Tensor] = None,
                 gate: Optional[Gate] = None, up_offset: int = 0) -> Tensor:
    """Rows ``[offsets[g], offsets[g + 1])`` of ``x [R, >= k]`` times ``w[g] [>= n, >= k]`` (transposed) into
    columns ``[0, n)`` of ``out``; row r of the result goes to row ``row_out[r]`` (None: r).  With ``gate``
    the result is that activation of rows ``[0, n)`` and ``[up_offset, up_offset + n)`` of ``w[g]``."""
    a = _Args()
    a.x, a.w, a.out, a.offsets = x.data_ptr(), w.data_ptr(), out.data_ptr(), offsets.data_ptr()
    a.row_out = None if row_out is None else row_out.data_ptr()
    a.x_row, a.x_group, a.w_row, a.w_group = x.stride(0), 0, w.stride(1), w.stride(0)
    a.out_row, a.out_group = out.stride(0), 0
    a.rows, a.groups, a.n, a.k, a.up_off = x.shape[0], w.shape[0], n, k, up_offset
    a.gate_kind = -1 if gate is None else _GATE_KINDS[gate.kind]
    a.act_bf16 = int(x.dtype == torch.bfloat16)
    if gate is not None:
        a.limit, a.alpha = gate.limit, gate.alpha
    _launch(a)
    return out


def reference_grouped_rows(x, w, offsets, *, n, k, gate=None, up_offset=0):
    """The same in PyTorch statements, rows in place (reads the offsets on the host)."""
    outs, bounds = [], offsets.tolist()
    for g in range(w.shape[0]):
        rows = x[bounds[g]:bounds[g + 1], :k].float()
        y = rows @ w[g, :n, :k].float().t()
        if gate is not None:
            y = gate_values(y, rows @ w[g, up_offset:up_offset + n, :k].float().t(), gate)
        outs.append(y)
    return torch.cat(outs).to(x.dtype)
