"""Mixture-of-experts feed-forward for inference: every token through its chosen experts, none dropped.

``route_rows`` picks the ``top`` largest sigmoid scores of each token; ``expert_feed_forward`` computes
``sum_k expert_(e_k)(w_k * h)``: the weight multiplies the expert's INPUT.  Expert weights are packed
``gate_up [E, 2 F', D']`` (up rows from F') and ``down [E, D', F']`` with the sizes rounded up to 64.

GPU: few tokens run ``csrc/experts.cu`` (routing and gather in one launch) and ``csrc/skinny_group.cu``, which
read each chosen expert's weights once; many bf16 tokens run the tcgen05 grouped GEMM over rows sorted by
expert; 32-bit runs use the plain kernel of ``csrc/skinny_group.cu``.
"""

from __future__ import annotations

import ctypes
import functools

import torch

from axlearn_b200.ops import dispatch
from axlearn_b200.ops.hyper_ops import Gate, gate_values, gated_act, padded

Tensor = torch.Tensor
# Up to this many (token, choice) pairs the weights dominate and the skinny kernels run.
SKINNY_MAX_PAIRS = 512


def route_rows(logits: Tensor, top: int) -> tuple[Tensor, Tensor]:
    """``(experts [T, top], scores [T, top])`` of fp32 logits: the ``top`` largest sigmoid scores, as they are."""
    scores, ids = torch.sigmoid(logits.float()).topk(top, dim=-1)
    return ids, scores


def reference_expert_feed_forward(h, logits, gate_up, down, *, top, width, hidden, gate: Gate):
    shape = h.shape
    h = h.reshape(-1, shape[-1])
    ids, weight = route_rows(logits.reshape(-1, logits.shape[-1]), top)
    half = gate_up.shape[1] // 2
    out = torch.zeros((h.shape[0], width), dtype=torch.float32, device=h.device)
    for e in range(gate_up.shape[0]):
        token, choice = torch.nonzero(ids == e, as_tuple=True)
        if token.numel() == 0:
            continue
        x = (h[token, :width].float() * weight[token, choice, None]).to(h.dtype).float()
        g = x @ gate_up[e, :hidden, :width].float().t()
        u = x @ gate_up[e, half:half + hidden, :width].float().t()
        y = gate_values(g, u, gate).to(h.dtype).float() @ down[e, :width, :hidden].float().t()
        out = out.index_add(0, token, y)
    out = torch.nn.functional.pad(out.to(h.dtype), (0, padded(width, 8) - width))
    return out.reshape(shape[:-1] + (out.shape[-1],))


def expert_feed_forward(h: Tensor, logits: Tensor, gate_up: Tensor, down: Tensor, *, top: int, width: int, hidden: int,
                        gate: Gate) -> Tensor:
    """``h [..., >= width]``, fp32 router ``logits [..., E]`` -> ``[..., width rounded up to 8]``."""
    tensors = [h, logits, gate_up, down]
    grad = torch.is_grad_enabled() and any(x.requires_grad for x in tensors)
    if dispatch._cuda(*tensors) and not grad and h.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        return _cuda_expert_feed_forward(h, logits, gate_up, down, top=top, width=width, hidden=hidden, gate=gate)
    return reference_expert_feed_forward(h, logits, gate_up, down, top=top, width=width, hidden=hidden, gate=gate)


# ------------------------------------------------------------------------------------------
# CUDA.
# ------------------------------------------------------------------------------------------


class _Args(ctypes.Structure):
    """Mirrors ``axb::RouteArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "logits", "h", "ids", "weight", "place", "offsets", "block_expert", "row_pair", "rows_out", "counts")] + [
        (n, ctypes.c_int64) for n in ("logits_ld", "h_ld", "rows_ld")] + [(n, ctypes.c_int) for n in (
            "tokens", "experts", "top", "width", "block", "blocks", "act_bf16")]


_signatures_set = False


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        for name in ("axb_route_small", "axb_route_sort"):
            getattr(h, name).argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
            getattr(h, name).restype = ctypes.c_int
        h.axb_expert_combine.argtypes = [ctypes.c_void_p] * 3 + [ctypes.c_int64] * 3 + [ctypes.c_int] * 3 + [ctypes.c_void_p]
        h.axb_expert_combine.restype = ctypes.c_int
        _signatures_set = True
    return h


def _cuda_expert_feed_forward(h, logits, gate_up, down, *, top, width, hidden, gate, path=None):
    """``path``: "skinny" / "sorted" overrides the choice by the number of pairs."""
    from axlearn_b200.ops import cuda_ops, moe_ops, skinny_ops

    lib = _lib()
    shape, dev = h.shape, h.device
    h = h.reshape(-1, shape[-1])
    h = h if h.is_contiguous() else h.contiguous()
    logits = logits.reshape(h.shape[0], -1)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    experts, half, dp = gate_up.shape[0], gate_up.shape[1] // 2, gate_up.shape[2]
    assert down.shape == (experts, dp, half) and gate_up.is_contiguous() and down.is_contiguous()
    gate_up, down = gate_up.to(h.dtype), down.to(h.dtype)
    tokens = h.shape[0]
    pairs = tokens * top
    bf16 = h.dtype == torch.bfloat16
    small = path == "skinny" or (path is None and bf16 and pairs <= SKINNY_MAX_PAIRS)
    block = moe_ops.GROUP_BLOCK if bf16 and not small else 1
    rows = pairs if block == 1 else padded(pairs + experts * (block - 1), block)
    a = _Args()
    ints = torch.empty(2 * pairs + experts + 1 + rows // block + experts, dtype=torch.int32, device=dev)
    place, row_pair, offsets, block_expert, counts = torch.split(
        ints, [pairs, pairs, experts + 1, rows // block, experts])
    x = torch.empty((rows, dp), dtype=h.dtype, device=dev)
    a.logits, a.h, a.rows_out = logits.data_ptr(), h.data_ptr(), x.data_ptr()
    a.place, a.offsets, a.row_pair = place.data_ptr(), offsets.data_ptr(), row_pair.data_ptr()
    a.logits_ld, a.h_ld, a.rows_ld = logits.stride(0), h.stride(0), dp
    a.tokens, a.experts, a.top, a.width, a.block, a.act_bf16 = tokens, experts, top, width, block, int(bf16)
    stream = cuda_ops._stream()  # pylint: disable=protected-access
    check = cuda_ops._check  # pylint: disable=protected-access
    out_ld = padded(width, 8)
    if small:
        check(lib.axb_route_small(ctypes.byref(a), stream), "axb_route_small")
    else:
        ids = torch.empty(pairs, dtype=torch.int32, device=dev)
        weight = torch.empty(pairs, dtype=torch.float32, device=dev)
        a.ids, a.weight, a.counts = ids.data_ptr(), weight.data_ptr(), counts.data_ptr()
        a.block_expert, a.blocks = block_expert.data_ptr(), rows // block
        check(lib.axb_route_sort(ctypes.byref(a), stream), "axb_route_sort")
    if block == 1:
        act = torch.empty((pairs, half), dtype=h.dtype, device=dev)
        skinny_ops.grouped_rows(x, gate_up, offsets, act, n=half, k=dp, gate=gate, up_offset=half)
        # Results in the order of the pairs, so that a token's choices lie next to each other.
        y = torch.empty((pairs, out_ld), dtype=h.dtype, device=dev)
        skinny_ops.grouped_rows(act, down, offsets, y, n=out_ld, k=half, row_out=row_pair)
        if top == 1:
            return y.reshape(shape[:-1] + (out_ld,))
        place = None
    else:
        # Rows between the runs hold anything; nobody reads their results.
        product = functools.partial(moe_ops._gmm_kernel, block_expert=block_expert, transpose_w=True, zero_unused=False)  # pylint: disable=protected-access
        y = product(gated_act(product(x, gate_up), half, half, gate), down)
    out = torch.empty((tokens, out_ld), dtype=h.dtype, device=dev)
    check(lib.axb_expert_combine(y.data_ptr(), None if place is None else place.data_ptr(), out.data_ptr(), tokens,
                                 y.stride(0), out_ld, top, out_ld, int(bf16), stream), "axb_expert_combine")
    return out.reshape(shape[:-1] + (out_ld,))
