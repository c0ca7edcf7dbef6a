"""Hyper-connections: the residual as several parallel streams, mixed around every sublayer.

A sublayer reads ``u = sum_s read[s] * x_s``, sees ``norm(u)``, and its branch ``y`` goes back as
``x_t <- sum_s mix[s, t] * x_s + multiplier * write[t] * y``.  Between two sublayers the write of the
first, the read of the second and its norm touch the same rows, so they are ONE operation here:
``hyper_step`` takes the streams and the previous branch and returns the new streams and the next
sublayer's input (``csrc/hyper.cu``: one pass, every stream element read once and written once).

Before the first sublayer all streams are equal; that state is kept as one copy ``[B, T, D]`` instead
of ``[B, T, S, D]``.  Streams are fp32; branches and outputs are in the activation dtype.

A branch may be the mean of several outputs, each RMS-normed with its own weight (two mixers side by
side): ``NormedPair`` hands the raw outputs over and their norms are computed in the same pass.
"""

from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional, Union

import torch
import torch.nn.functional as F

from axlearn_b200.ops import dispatch

Tensor = torch.Tensor
MAX_STREAMS = 16


class NormedPair(NamedTuple):
    """``weight * (rms(left) * left_scale + rms(right) * right_scale)`` over the first ``width`` columns."""

    left: Tensor
    right: Tensor
    left_scale: Tensor
    right_scale: Tensor
    eps: float
    weight: float = 0.5


class StreamWrite(NamedTuple):
    mix: Optional[Tensor]          # [S, S], indexed [from, to]; None: the identity
    out: Optional[Tensor]          # [S]; None: ones
    multiplier: float


# The write of an ordinary residual.
PLAIN_WRITE = StreamWrite(None, None, 1.0)


def padded(n: int, multiple: int) -> int:
    return -(-n // multiple) * multiple


def _rms(x: Tensor, eps: float) -> Tensor:
    return x * torch.rsqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def combine_branch(branch: Union[Tensor, NormedPair], width: int) -> Tensor:
    """The branch as one fp32 tensor ``[..., width]``."""
    if isinstance(branch, NormedPair):
        left, right = branch.left[..., :width].float(), branch.right[..., :width].float()
        return branch.weight * (_rms(left, branch.eps) * branch.left_scale.float()
                                + _rms(right, branch.eps) * branch.right_scale.float())
    return branch[..., :width].float()


def reference_hyper_step(streams, branch, write, read, norm_scale, *, eps, norm_offset, dtype, num_streams, width,
                         h_multiplier=1.0):
    x = streams.float()
    if x.dim() == 3:
        x = x[:, :, None, :].expand(-1, -1, num_streams, -1)
    if branch is not None:
        y = combine_branch(branch, width)
        out = write.out.float() if write.out is not None else torch.ones(num_streams, device=y.device)
        mixed = x if write.mix is None else torch.einsum("btsd,se->bted", x, write.mix.float())
        x = mixed + (write.multiplier * out)[:, None] * y[:, :, None, :]
        streams = x
    u = x.sum(dim=2) if read is None else torch.einsum("btsd,s->btd", x, read.float())
    if norm_scale is None:
        return streams, u
    h = (_rms(u, eps) * (norm_offset + norm_scale.float()) * h_multiplier).to(dtype)
    return streams, F.pad(h, (0, padded(width, 8) - width))


def hyper_step(streams: Tensor, branch: Optional[Union[Tensor, NormedPair]] = None, *,
               write: Optional[StreamWrite] = None, read: Optional[Tensor] = None,
               norm_scale: Optional[Tensor] = None, eps: float = 1e-6, norm_offset: float = 1.0,
               num_streams: int, dtype: torch.dtype, keep_streams: bool = True,
               h_multiplier: float = 1.0) -> tuple[Optional[Tensor], Tensor]:
    """``(new streams, next input)``.

    streams: ``[B, T, D]`` (all streams equal) or fp32 ``[B, T, S, D]``.  branch / write: the previous
    sublayer's output and how it is written (None ahead of the first sublayer).  read: ``[S]``, or None
    for the plain sum of the streams.  norm_scale: the norm's stored weight, applied as
    ``norm_offset + weight``; None returns the fp32 sum itself.  The next input is ``[B, T, D']`` with
    D' = D rounded up to 8, its padding zero (a matrix-product operand).  ``keep_streams=False`` (the
    last read of a stack) returns no streams.  ``h_multiplier`` scales the normed output."""
    width = streams.shape[-1]
    if branch is not None and write is None:
        raise ValueError("a branch needs its write weights")
    tensors = [streams, read, norm_scale]
    if write is not None:
        tensors += [write.mix, write.out]
    tensors += list(branch[:4]) if isinstance(branch, NormedPair) else [branch]
    grad = torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in tensors)
    on_gpu = dispatch._cuda(*tensors) and not grad  # pylint: disable=protected-access
    if on_gpu and dtype in (torch.bfloat16, torch.float32):
        return _cuda_hyper_step(streams, branch, write, read, norm_scale, eps=eps, norm_offset=norm_offset,
                                dtype=dtype, num_streams=num_streams, width=width, keep_streams=keep_streams,
                                h_multiplier=h_multiplier)
    new, h = reference_hyper_step(streams, branch, write, read, norm_scale, eps=eps, norm_offset=norm_offset,
                                  dtype=dtype, num_streams=num_streams, width=width, h_multiplier=h_multiplier)
    return (new if keep_streams else None), h


class _Args(ctypes.Structure):
    """Mirrors ``axb::HyperArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "streams", "branch_a", "branch_b", "scale_a", "scale_b", "mix", "out_w", "read", "norm_scale",
        "streams_out", "h")] + [
        ("rows", ctypes.c_int64), ("streams_ld", ctypes.c_int64), ("branch_ld", ctypes.c_int64),
        ("h_ld", ctypes.c_int64)] + [(n, ctypes.c_int) for n in (
            "width", "num_streams", "streams_equal", "streams_bf16", "act_bf16")] + [(n, ctypes.c_float) for n in (
                "multiplier", "pair_weight", "pair_eps", "eps", "norm_offset", "h_mult")]


_signature_set = False


def _lib():
    global _signature_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signature_set:
        h.axb_hyper_step.argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
        h.axb_hyper_step.restype = ctypes.c_int
        h.axb_gated_act.argtypes = ([ctypes.c_void_p] * 2 + [ctypes.c_int64, ctypes.c_int, ctypes.c_int]
                                    + [ctypes.c_int64] * 2 + [ctypes.c_int] * 2 + [ctypes.c_float] * 2
                                    + [ctypes.c_void_p])
        h.axb_gated_act.restype = ctypes.c_int
        _signature_set = True
    return h


def _f32(t: Optional[Tensor]) -> Optional[Tensor]:
    return None if t is None else t.float().contiguous()


def _cuda_hyper_step(streams, branch, write, read, norm_scale, *, eps, norm_offset, dtype, num_streams, width,
                     keep_streams, h_multiplier):
    from axlearn_b200.ops import cuda_ops

    if num_streams > MAX_STREAMS:
        raise ValueError(f"at most {MAX_STREAMS} residual streams")
    b, t = streams.shape[:2]
    equal = streams.dim() == 3
    if streams.stride(-1) != 1 or (equal and streams.stride(0) != t * streams.stride(1)) or (
            not equal and not streams.is_contiguous()):
        streams = streams.contiguous()
    if not equal and streams.dtype != torch.float32:
        raise ValueError("residual streams are fp32")
    if equal and streams.dtype not in (torch.float32, torch.bfloat16):
        raise ValueError(f"unsupported embedding dtype {streams.dtype}")
    a = _Args()
    keep = []

    def ptr(x):
        if x is None:
            return None
        keep.append(x)
        return x.data_ptr()

    a.streams = ptr(streams)
    if branch is not None:
        pair = isinstance(branch, NormedPair)
        first = branch.left if pair else branch
        second = branch.right if pair else None
        for x in (first, second):
            if x is not None and (x.dtype != dtype or not x.is_contiguous() or x.shape[-1] != first.shape[-1]):
                raise ValueError("branches must be contiguous and in the activation dtype")
        a.branch_a, a.branch_b, a.branch_ld = ptr(first), ptr(second), first.shape[-1]
        if pair:
            a.scale_a, a.scale_b = ptr(_f32(branch.left_scale)), ptr(_f32(branch.right_scale))
            a.pair_weight, a.pair_eps = branch.weight, branch.eps
        a.mix, a.out_w, a.multiplier = ptr(_f32(write.mix)), ptr(_f32(write.out)), write.multiplier
    a.read, a.norm_scale = ptr(_f32(read)), ptr(_f32(norm_scale))
    new = streams
    if branch is not None:
        new = None
        if keep_streams:
            new = torch.empty((b, t, num_streams, width), dtype=torch.float32, device=streams.device)
            a.streams_out = ptr(new)
    if norm_scale is None:
        h = torch.empty((b, t, width), dtype=torch.float32, device=streams.device)
    else:
        h = torch.empty((b, t, padded(width, 8)), dtype=dtype, device=streams.device)
    a.h, a.h_ld = ptr(h), h.shape[-1]
    a.rows, a.streams_ld = b * t, (streams.stride(1) if equal else num_streams * width)
    a.width, a.num_streams, a.streams_equal = width, num_streams, int(equal)
    a.streams_bf16, a.act_bf16 = int(streams.dtype == torch.bfloat16), int(dtype == torch.bfloat16)
    a.eps, a.norm_offset, a.h_mult = eps, norm_offset, h_multiplier
    cuda_ops._check(_lib().axb_hyper_step(ctypes.byref(a), cuda_ops._stream()), "axb_hyper_step")  # pylint: disable=protected-access
    return (new if keep_streams else None), h


class Gate(NamedTuple):
    """How a gated feed-forward combines its two halves ``g`` and ``u``:

    * ``silu``: ``silu(g) * u``
    * ``gelu_tanh``: ``gelu(g) * u`` with the tanh form of gelu
    * ``clamped``: ``g' sigmoid(alpha g') (u' + 1)`` with ``g' = min(g, limit)``, ``u'`` clamped to ``+-limit``
    """

    kind: str = "silu"
    limit: float = 0.0
    alpha: float = 1.702


_GATE_KINDS = {"silu": 0, "gelu_tanh": 1, "clamped": 2}


def gate_values(g: Tensor, u: Tensor, gate: Gate) -> Tensor:
    if gate.kind == "silu":
        return F.silu(g) * u
    if gate.kind == "gelu_tanh":
        return F.gelu(g, approximate="tanh") * u
    if gate.kind == "clamped":
        g, u = g.clamp(max=gate.limit), u.clamp(-gate.limit, gate.limit)
        return g * torch.sigmoid(gate.alpha * g) * (u + 1)
    raise ValueError(f"unknown gate {gate.kind!r}")


def gated_act(gu: Tensor, width: int, up_offset: int, gate: Gate = Gate()) -> Tensor:
    """``gate`` applied to a packed product: gate half in columns ``[0, width)``, up half from ``up_offset``;
    the result is ``width`` rounded up to 8 columns wide, zero-padded."""
    out_ld = padded(width, 8)
    grad = torch.is_grad_enabled() and gu.requires_grad
    if dispatch._cuda(gu) and not grad and gu.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        from axlearn_b200.ops import cuda_ops

        gu = gu.contiguous()
        out = torch.empty(gu.shape[:-1] + (out_ld,), dtype=gu.dtype, device=gu.device)
        cuda_ops._check(_lib().axb_gated_act(  # pylint: disable=protected-access
            gu.data_ptr(), out.data_ptr(), gu.numel() // gu.shape[-1], width, up_offset, gu.shape[-1], out_ld,
            int(gu.dtype == torch.bfloat16), _GATE_KINDS[gate.kind], gate.limit, gate.alpha,
            cuda_ops._stream()), "axb_gated_act")  # pylint: disable=protected-access
        return out
    y = gate_values(gu[..., :width].float(), gu[..., up_offset:up_offset + width].float(), gate)
    return F.pad(y.to(gu.dtype), (0, out_ld - width))
