"""Gated sliding-window attention over a packed projection and a ring KV cache.

``window_attention`` serves whole prompts, continued prompts and single decoding tokens with one
contract: ``proj [B, T, P]`` holds every token's q, k, v and output gate at given columns, ``start[b]``
tokens are already in the ring, ``live[b]`` of the T new ones are valid.  For query position ``i`` and key
position ``j`` with ``0 <= i - j < window``::

    score = (q . k) * scale * temperature(i) - slope_h * (i - j)

followed by an ordinary softmax, the values, and ``sigmoid(gate)``.  Temperature and distance bias are
optional.  Scores and softmax are fp32.  On the GPU: ``csrc/window_attn.cu`` (decoding, continued
prompts, fp32) and ``csrc/flash_fwd_v3.cu`` (bf16 prompts on the tensor cores); there the ring is updated
in place.
"""

from __future__ import annotations

import ctypes
import dataclasses
from typing import Optional

import torch
import torch.nn.functional as F

from axlearn_b200.ops import dispatch
from axlearn_b200.ops.hyper_ops import padded

Tensor = torch.Tensor


@dataclasses.dataclass(frozen=True)
class WindowSpec:
    """Sizes and constants of the attention; ``q_temp = (coef, every)``."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    q_temp: Optional[tuple] = None
    distance_bias: bool = False
    gated: bool = True

    @property
    def out_width(self) -> int:
        """Columns of the result: heads * vdim rounded up to a matrix-product operand, zero-padded."""
        return padded(self.heads * self.vdim, 8)


@dataclasses.dataclass(frozen=True)
class WindowColumns:
    """First column of each section in the projection (``g`` is unused without a gate)."""

    q: int
    k: int
    v: int
    g: int = -1


def distance_slopes(heads: int, *, device=None) -> Tensor:
    """``2^(-8 (h + 1) / heads)`` for every head count (no special case off the powers of two)."""
    return 2.0 ** (-8.0 * torch.arange(1, heads + 1, device=device, dtype=torch.float32) / heads)


def query_temperature(positions: Tensor, coef: float, every: int) -> Tensor:
    """``1 + coef * ln(floor((p + 1) / every) + 1)``."""
    return 1.0 + coef * torch.log(torch.div(positions + 1, every, rounding_mode="floor").float() + 1.0)


def ring_positions(slots: int, start: Tensor) -> Tensor:
    """Absolute position held by every ring slot ``[B, slots]`` when ``start`` tokens have been stored
    (position p in slot p % slots); negative = empty."""
    last = start.long()[:, None] - 1
    s = torch.arange(slots, device=start.device)[None]
    return torch.where(last >= 0, last - torch.remainder(last - s, slots), torch.full_like(s, -1))


def reference_window_attention(proj, spec: WindowSpec, cols: WindowColumns, *, start, live, cache):
    b, t, _ = proj.shape
    h, g, dk, dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    q = proj[..., cols.q:cols.q + h * dk].float().reshape(b, t, g, h // g, dk)
    k_new = proj[..., cols.k:cols.k + g * dk].reshape(b, t, g, dk)
    v_new = proj[..., cols.v:cols.v + g * dv].reshape(b, t, g, dv)
    pos = start.long()[:, None] + torch.arange(t, device=proj.device)[None]                 # [B, T]
    k_pos = torch.where(torch.arange(t, device=proj.device)[None] < live[:, None], pos, -1)
    k, v = k_new, v_new
    if cache is not None:
        k = torch.cat([cache["key"].to(k.dtype), k], dim=1)
        v = torch.cat([cache["value"].to(v.dtype), v], dim=1)
        k_pos = torch.cat([ring_positions(cache["key"].shape[1], start), k_pos], dim=1)
    if spec.q_temp is not None:
        q = q * query_temperature(pos, *spec.q_temp)[:, :, None, None, None]
    rel = pos[:, :, None] - k_pos[:, None, :]                                               # [B, T, S]
    scores = torch.einsum("btgrd,bsgd->bgrts", q, k.float()) * spec.scale
    if spec.distance_bias:
        slopes = distance_slopes(h, device=proj.device).reshape(g, h // g)
        scores = scores - slopes[None, :, :, None, None] * rel[:, None, None].float()
    seen = (rel >= 0) & (rel < spec.window) & (k_pos >= 0)[:, None, :]
    scores = scores.masked_fill(~seen[:, None, None], float("-inf"))
    # Padding queries see nothing: their softmax is replaced by zeros.
    probs = torch.softmax(scores, dim=-1).nan_to_num(0.0)
    out = torch.einsum("bgrts,bsgd->btgrd", probs, v.float()).reshape(b, t, h * dv)
    if spec.gated:
        out = out * torch.sigmoid(proj[..., cols.g:cols.g + h * dv].float())
    out = F.pad(out.to(proj.dtype), (0, spec.out_width - h * dv))
    if cache is None:
        return out, None
    slots = cache["key"].shape[1]
    keep = (torch.arange(t, device=proj.device)[None] < live[:, None]) & (
        torch.arange(t, device=proj.device)[None] >= live[:, None] - slots)
    key, value = cache["key"].clone(), cache["value"].clone()
    rows, idx = torch.nonzero(keep, as_tuple=True)
    slot = torch.remainder(pos[rows, idx], slots)
    key[rows, slot] = k_new[rows, idx].to(key.dtype)
    value[rows, slot] = v_new[rows, idx].to(value.dtype)
    return out, {"key": key, "value": value}


def window_attention(proj: Tensor, spec: WindowSpec, cols: WindowColumns, *, start: Optional[Tensor] = None,
                     live: Optional[Tensor] = None, cache: Optional[dict] = None):
    """``(out [B, T, out_width], cache)``.

    start: int32 ``[B]`` tokens already stored (None: zero); a negative value takes the row out of the
    step (its output is zero, its cache untouched).  live: int32 ``[B]`` valid new tokens (None: T).
    cache: ``{"key": [B, slots, G, dim], "value": [B, slots, G, vdim]}`` or None (nothing is stored and
    nothing before this block is seen)."""
    grad = torch.is_grad_enabled() and proj.requires_grad
    if dispatch._cuda(proj) and not grad and proj.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        return _cuda_window_attention(proj, spec, cols, start=start, live=live, cache=cache)
    b, t, _ = proj.shape
    if start is None:
        start = torch.zeros(b, dtype=torch.int32, device=proj.device)
    if live is None:
        live = torch.full((b,), t, dtype=torch.int32, device=proj.device)
    live = torch.where(start < 0, torch.zeros_like(live), live)
    return reference_window_attention(proj, spec, cols, start=start.clamp_min(0), live=live, cache=cache)


# ------------------------------------------------------------------------------------------
# CUDA.
# ------------------------------------------------------------------------------------------


class _Args(ctypes.Structure):
    """Mirrors ``axb::WindowArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "proj", "k_ring", "v_ring", "out", "start", "live", "part", "tickets")] + [
        ("ld", ctypes.c_int64), ("out_ld", ctypes.c_int64)] + [(n, ctypes.c_int) for n in (
            "B", "T", "heads", "kv_heads", "dim", "vdim", "slots", "window", "q_off", "k_off", "v_off", "g_off",
            "splits", "every", "bias", "act_bf16")] + [("scale", ctypes.c_float), ("coef", ctypes.c_float)]


_signatures_set = False
_tickets: dict = {}
# Below this many new tokens per sequence the tensor-core kernel's 128-row tiles are mostly padding.
FLASH_MIN_TOKENS = 32


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        for name in ("axb_window_decode", "axb_window_attn", "axb_window_append"):
            getattr(h, name).argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
            getattr(h, name).restype = ctypes.c_int
        h.axb_window_decode_ctas.argtypes = [ctypes.c_int] * 5
        h.axb_window_decode_ctas.restype = ctypes.c_int
        h.axb_flash_fwd_gated.argtypes = (
            [ctypes.c_void_p] * 5 + [ctypes.c_int] * 6 + [ctypes.c_int64] * 2 + [ctypes.c_float, ctypes.c_int,
                                                                               ctypes.c_float, ctypes.c_int,
                                                                               ctypes.c_int, ctypes.c_void_p,
                                                                               ctypes.c_void_p])
        h.axb_flash_fwd_gated.restype = ctypes.c_int
        _signatures_set = True
    return h


def _ticket_buffer(device: torch.device, n: int) -> Tensor:
    """Zeroed counters of the split-window merge, per (device, stream); the kernel leaves them zero."""
    from axlearn_b200.ops import cuda_ops

    key = (device.index if device.index is not None else torch.cuda.current_device(), cuda_ops._stream())  # pylint: disable=protected-access
    have = _tickets.get(key)
    if have is None or have.numel() < n:
        have = torch.zeros(max(n, 4096), dtype=torch.int32, device=device)
        _tickets[key] = have
    return have


def decode_splits(ctas: int, span: int, sms: int = 148) -> int:
    """KV splits of a decoding step: one wave of two CTAs per SM, at least 64 keys each."""
    want = max(1, (2 * sms) // max(1, ctas))
    return max(1, min(want, span // 64, 64))


def flash_supported(proj: Tensor, spec: WindowSpec, cols: WindowColumns) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes (16-byte aligned head rows up to 128)."""
    parts = [spec.dim, spec.vdim, proj.shape[-1], cols.q, cols.k, cols.v] + ([cols.g] if spec.gated else [])
    return proj.dtype == torch.bfloat16 and max(spec.dim, spec.vdim) <= 128 and all(x % 8 == 0 for x in parts)


def _int32(t: Optional[Tensor]) -> Optional[Tensor]:
    if t is None:
        return None
    return t if t.dtype == torch.int32 and t.is_contiguous() else t.to(torch.int32).contiguous()


def _cuda_window_attention(proj, spec, cols, *, start, live, cache):
    from axlearn_b200.ops import cuda_ops

    lib = _lib()
    proj = proj.contiguous()
    b, t, ld = proj.shape
    start, live = _int32(start), _int32(live)
    out = torch.empty((b, t, spec.out_width), dtype=proj.dtype, device=proj.device)
    coef, every = spec.q_temp if spec.q_temp is not None else (0.0, 1)
    a = _Args()
    a.proj, a.out, a.ld, a.out_ld = proj.data_ptr(), out.data_ptr(), ld, out.shape[-1]
    a.start = None if start is None else start.data_ptr()
    a.live = None if live is None else live.data_ptr()
    a.B, a.T, a.heads, a.kv_heads, a.dim, a.vdim = b, t, spec.heads, spec.kv_heads, spec.dim, spec.vdim
    a.window, a.slots = spec.window, 1
    if cache is not None:
        key, value = cache["key"], cache["value"]
        assert key.is_contiguous() and value.is_contiguous() and key.dtype == proj.dtype == value.dtype
        assert key.shape[2:] == (spec.kv_heads, spec.dim) and value.shape[2:] == (spec.kv_heads, spec.vdim)
        a.k_ring, a.v_ring, a.slots = key.data_ptr(), value.data_ptr(), key.shape[1]
    a.q_off, a.k_off, a.v_off, a.g_off = cols.q, cols.k, cols.v, (cols.g if spec.gated else -1)
    a.coef, a.every, a.scale, a.bias = float(coef), int(every), spec.scale, int(spec.distance_bias)
    a.act_bf16, a.splits = int(proj.dtype == torch.bfloat16), 1
    stream = cuda_ops._stream()  # pylint: disable=protected-access
    check = cuda_ops._check  # pylint: disable=protected-access
    if t == 1 and start is not None and cache is not None:
        ctas = lib.axb_window_decode_ctas(b, spec.heads, spec.kv_heads, spec.dim, spec.vdim)
        a.splits = decode_splits(ctas, min(spec.window, a.slots))
        part = None
        if a.splits > 1:
            part = torch.empty(b * spec.heads * a.splits * padded(spec.vdim + 2, 4), dtype=torch.float32, device=proj.device)
            a.part, a.tickets = part.data_ptr(), _ticket_buffer(proj.device, ctas).data_ptr()
        check(lib.axb_window_decode(ctypes.byref(a), stream), "axb_window_decode")
        return out, cache
    if start is not None and cache is None:
        raise ValueError("a continued block needs its cache")
    if start is None and t >= FLASH_MIN_TOKENS and flash_supported(proj, spec, cols):
        base, e = proj.data_ptr(), proj.element_size()
        check(lib.axb_flash_fwd_gated(
            base + cols.q * e, base + cols.k * e, base + cols.v * e, base + cols.g * e if spec.gated else None,
            out.data_ptr(), b, t, spec.heads, spec.kv_heads, spec.dim, spec.vdim, ld, out.shape[-1], spec.scale,
            spec.window, float(coef), int(every), int(spec.distance_bias),
            cuda_ops.status_word(proj.device).data_ptr(), stream), "axb_flash_fwd_gated")
    else:
        check(lib.axb_window_attn(ctypes.byref(a), stream), "axb_window_attn")
    if cache is not None:
        check(lib.axb_window_append(ctypes.byref(a), stream), "axb_window_append")
    return out, cache
