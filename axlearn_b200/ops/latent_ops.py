"""Latent attention: keys and values of all heads come from one low-rank vector per token.

A token's projection holds per-head queries ``[dim | rot_dim]`` (``q``), a latent (``c``, RMS-normed with a
weight) and one rotated key part shared by all heads (``r``).  With ``W_uk`` / ``W_uv`` per head::

    score = (q_plain . W_uk c_j + rot(q_r, i) . rot(r_j, j)) * scale,   j <= i
    out   = softmax(score) (W_uv c_j)

``rot`` turns the interleaved pairs ``(2k, 2k + 1)`` by ``position * base^(-2k / rot_dims)``.  Only the normed
latent and the rotated key part are cached, ``[B, slots, W]`` with W = both parts rounded up to 8 columns
(padding is zero).

Two forms of the same sum.  *Expanded* (prompts): keys and values of all heads are products of the latents
and a flash kernel runs over them.  *Absorbed* (decoding, continued prompts, 32-bit runs):
``q_plain . (W_uk c) = (W_uk^T q_plain) . c``, so attention runs over the cache rows themselves, as one key
head shared by all query heads, and ``W_uv`` is applied to the result.

``latent_attention`` takes ``start`` / ``live`` like the other mixers.  GPU: ``csrc/latent_attn.cu``,
``csrc/flash_fwd_v3.cu`` (expanded form), ``csrc/skinny_group.cu`` (per-head products of a decoding step); the
cache is updated in place.
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
class LatentSpec:
    heads: int
    dim: int           # unrotated query / key size of a head
    rot_dim: int       # rotated query / key size of a head
    vdim: int
    rank: int          # latent size
    rot_dims: int      # how many of the rot_dim dimensions turn (the rest pass unchanged)
    rot_base: float
    scale: float
    eps: float

    @property
    def rot_offset(self) -> int:
        """First column of the rotated part in a cache row."""
        return padded(self.rank, 8)

    @property
    def row_width(self) -> int:
        return padded(self.rank, 8) + padded(self.rot_dim, 8)

    @property
    def out_width(self) -> int:
        return padded(self.heads * self.vdim, 8)


@dataclasses.dataclass(frozen=True)
class LatentColumns:
    q: int
    c: int
    r: int


def rotation_frequencies(dims: int, base: float, *, device=None) -> Tensor:
    """``base^(-2k / dims)`` for every pair, in double precision."""
    return base ** (-torch.arange(0, dims, 2, dtype=torch.float64, device=device) / dims)


def rotate_interleaved(x: Tensor, positions: Tensor, dims: int, base: float) -> Tensor:
    """Turns the pairs (2k, 2k + 1) of the first ``dims`` entries of the last axis.  ``positions`` has the
    shape of ``x`` without the last axis, or broadcasts against it."""
    angle = positions.double()[..., None] * rotation_frequencies(dims, base, device=x.device)
    c, s = torch.cos(angle).float(), torch.sin(angle).float()
    u, v = x[..., 0:dims:2].float(), x[..., 1:dims:2].float()
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:].float()], dim=-1)


def reference_latent_attention(proj, norm_scale, uk, uv, spec: LatentSpec, cols: LatentColumns, *, start, live, cache):
    """Differentiable, expanded form.  ``uk [rank, heads * dim]``, ``uv [heads * vdim, rank]`` (stored sizes
    may be larger)."""
    b, t, _ = proj.shape
    h, dk, dr, dv, rank = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.rank
    uk, uv = uk[:rank, :h * dk].float(), uv[:h * dv, :rank].float()
    q = proj[..., cols.q:cols.q + h * (dk + dr)].float().reshape(b, t, h, dk + dr)
    c = proj[..., cols.c:cols.c + rank].float()
    c = c * torch.rsqrt(c.pow(2).mean(dim=-1, keepdim=True) + spec.eps) * norm_scale.float()
    pos = start.long()[:, None] + torch.arange(t, device=proj.device)[None]
    r = rotate_interleaved(proj[..., cols.r:cols.r + dr], pos, spec.rot_dims, spec.rot_base)
    qr = rotate_interleaved(q[..., dk:], pos[..., None], spec.rot_dims, spec.rot_base)
    row = torch.cat([F.pad(c, (0, spec.rot_offset - rank)),
                     F.pad(r, (0, spec.row_width - spec.rot_offset - dr))], dim=-1).to(proj.dtype)
    new_cache = None
    if cache is None:
        rows = row
    else:
        rows = cache["latent"].clone()
        slots = rows.shape[1]
        keep = (torch.arange(t, device=proj.device)[None] < live[:, None]) & (pos < slots)
        at, idx = torch.nonzero(keep, as_tuple=True)
        rows[at, pos[at, idx]] = row[at, idx].to(rows.dtype)
        new_cache = {"latent": rows}
    rows = rows.float()
    k = (rows[..., :rank] @ uk).reshape(b, -1, h, dk)
    v = (rows[..., :rank] @ uv.t()).reshape(b, -1, h, dv)
    kr = rows[..., spec.rot_offset:spec.rot_offset + dr]
    scores = (torch.einsum("bthd,bshd->bhts", q[..., :dk], k) + torch.einsum("bthd,bsd->bhts", qr, kr)) * spec.scale
    seen = torch.arange(rows.shape[1], device=proj.device)[None, None] <= pos[:, :, None]
    scores = scores.masked_fill(~seen[:, None], float("-inf"))
    out = torch.einsum("bhts,bshd->bthd", torch.softmax(scores, dim=-1), v).reshape(b, t, h * dv)
    dead = torch.arange(t, device=proj.device)[None] >= live[:, None]
    out = out.masked_fill(dead[..., None], 0.0)
    return F.pad(out.to(proj.dtype), (0, spec.out_width - h * dv)), new_cache


def latent_attention(proj: Tensor, norm_scale: Tensor, uk: Tensor, uv: Tensor, spec: LatentSpec, cols: LatentColumns,
                     *, start: Optional[Tensor] = None, live: Optional[Tensor] = None, cache: Optional[dict] = None):
    """``(out [B, T, out_width], cache)``.

    uk: ``[>= rank, >= heads * dim]`` (key of head h = columns ``h * dim ..`` of ``c @ uk``); uv: ``[>= heads *
    vdim, >= rank]``; surplus rows and columns are zero.  start: int32 ``[B]`` tokens already cached (None:
    zero); negative takes the row out of the step.  live: int32 ``[B]`` valid new tokens (None: T).  cache:
    ``{"latent": [B, slots, row_width]}`` or None (nothing is stored and nothing before this block is seen).
    On the GPU ``proj`` may be overwritten (queries are rotated in place)."""
    tensors = [proj, norm_scale, uk, uv]
    grad = torch.is_grad_enabled() and any(x.requires_grad for x in tensors)
    if dispatch._cuda(*tensors) and not grad and proj.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        return _cuda_latent_attention(proj, norm_scale, uk, uv, spec, cols, start=start, live=live, cache=cache)
    b, t, _ = proj.shape
    if live is None:
        live = torch.full((b,), t, dtype=torch.int32, device=proj.device)
    if start is None:
        start = torch.zeros(b, dtype=torch.int32, device=proj.device)
    elif cache is None:
        raise ValueError("a continued block needs its cache")
    live = torch.where(start < 0, torch.zeros_like(live), live)
    return reference_latent_attention(proj, norm_scale, uk, uv, spec, cols, start=start.clamp_min(0), live=live,
                                      cache=cache)


# ------------------------------------------------------------------------------------------
# CUDA.
# ------------------------------------------------------------------------------------------


class _Args(ctypes.Structure):
    """Mirrors ``axb::LatentArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "proj", "norm_w", "freq", "cache", "lat", "qbuf", "out", "part", "part_ml", "start", "live")] + [
        (n, ctypes.c_int64) for n in ("ld", "cache_ld", "lat_ld", "out_ld")] + [(n, ctypes.c_int) for n in (
            "B", "T", "heads", "dim", "rot_dim", "rot_dims", "rank", "rot_off", "row_w", "slots", "q_off", "c_off",
            "r_off", "splits", "act_bf16")] + [("scale", ctypes.c_float), ("eps", ctypes.c_float)]


_signatures_set = False
_freq_tables: dict = {}
# Below this many new tokens per sequence the tensor-core prompt kernel's 128-row tiles are mostly padding.
FLASH_MIN_TOKENS = 16


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        for name in ("axb_latent_prep", "axb_latent_attn", "axb_latent_decode"):
            getattr(h, name).argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
            getattr(h, name).restype = ctypes.c_int
        h.axb_latent_decode_supported.argtypes = [ctypes.c_int, ctypes.c_int]
        h.axb_latent_decode_supported.restype = ctypes.c_int
        h.axb_flash_fwd_latent.argtypes = (
            [ctypes.c_void_p] * 5 + [ctypes.c_int] * 6 + [ctypes.c_int64] * 6 + [ctypes.c_float] + [ctypes.c_void_p] * 2)
        h.axb_flash_fwd_latent.restype = ctypes.c_int
        _signatures_set = True
    return h


def _freq_table(dims: int, base: float, device) -> Tensor:
    key = (dims, base, str(device))
    if key not in _freq_tables:
        _freq_tables[key] = rotation_frequencies(dims, base).to(device)
    return _freq_tables[key]


def flash_supported(spec: LatentSpec, proj: Tensor, cols: LatentColumns) -> bool:
    """Sizes of the expanded tensor-core form: 16-byte aligned parts, unrotated and value heads up to 128,
    rotated up to 64."""
    parts = (spec.dim, spec.rot_dim, spec.vdim, spec.rank, proj.shape[-1], cols.q, cols.c, cols.r)
    return (proj.dtype == torch.bfloat16 and all(x % 8 == 0 for x in parts) and max(spec.dim, spec.vdim) <= 128
            and spec.rot_dim <= 64)


def decode_splits(ctas: int, keys: int, sms: int = 148) -> int:
    """Cuts of the cached rows in a decoding step: about one CTA per SM, at least one tile of 64 keys each."""
    return max(1, min(sms // max(1, ctas), -(-keys // 64), 64))


def _cuda_latent_attention(proj, norm_scale, uk, uv, spec, cols, *, start, live, cache, form: Optional[str] = None):
    """``form``: "expanded" / "absorbed" / "plain" (absorbed on the kernel without tensor cores) overrides the
    choice."""
    from axlearn_b200 import ops
    from axlearn_b200.ops import cuda_ops, skinny_ops
    from axlearn_b200.ops.window_ops import _int32

    lib = _lib()
    proj = proj.contiguous()
    norm_scale = norm_scale.float().contiguous()
    b, t, ld = proj.shape
    h, dk, dv = spec.heads, spec.dim, spec.vdim
    start, live = _int32(start), _int32(live)
    if cache is None:
        if start is not None:
            raise ValueError("a continued block needs its cache")
        rows = torch.empty((b, t, spec.row_width), dtype=proj.dtype, device=proj.device)
    else:
        rows = cache["latent"]
    assert rows.is_contiguous() and rows.dtype == proj.dtype and rows.shape[::2] == (b, spec.row_width), (rows.shape, spec)
    expanded = form == "expanded" or (
        form is None and start is None and t >= FLASH_MIN_TOKENS and flash_supported(spec, proj, cols))
    out = torch.empty((b, t, spec.out_width), dtype=proj.dtype, device=proj.device)
    a = _Args()
    freq = _freq_table(spec.rot_dims, spec.rot_base, proj.device)
    a.proj, a.norm_w, a.freq, a.cache = proj.data_ptr(), norm_scale.data_ptr(), freq.data_ptr(), rows.data_ptr()
    a.start = None if start is None else start.data_ptr()
    a.live = None if live is None else live.data_ptr()
    a.ld, a.cache_ld, a.B, a.T = ld, spec.row_width, b, t
    a.heads, a.dim, a.rot_dim, a.rot_dims, a.rank = h, dk, spec.rot_dim, spec.rot_dims, spec.rank
    a.rot_off, a.row_w, a.slots = spec.rot_offset, spec.row_width, rows.shape[1]
    a.q_off, a.c_off, a.r_off = cols.q, cols.c, cols.r
    a.act_bf16, a.splits, a.scale, a.eps = int(proj.dtype == torch.bfloat16), 1, spec.scale, spec.eps
    stream = cuda_ops._stream()  # pylint: disable=protected-access
    check = cuda_ops._check  # pylint: disable=protected-access
    if expanded:
        lat = torch.empty((b * t, spec.rot_offset), dtype=proj.dtype, device=proj.device)
        a.lat, a.lat_ld = lat.data_ptr(), spec.rot_offset
        check(lib.axb_latent_prep(ctypes.byref(a), stream), "axb_latent_prep")
        k = ops.linear(lat, uk.to(proj.dtype))
        v = ops.linear(lat, uv.to(proj.dtype).t())
        e = proj.element_size()
        check(lib.axb_flash_fwd_latent(
            proj.data_ptr() + cols.q * e, k.data_ptr(), rows.data_ptr() + spec.rot_offset * e, v.data_ptr(),
            out.data_ptr(), b, t, h, dk, spec.rot_dim, dv, ld, k.shape[-1], spec.row_width,
            rows.shape[1] * spec.row_width, v.shape[-1], out.shape[-1], spec.scale,
            cuda_ops.status_word(proj.device).data_ptr(), stream), "axb_flash_fwd_latent")
        if out.shape[-1] != h * dv:
            out[..., h * dv:] = 0
        return out, cache
    qbuf = torch.empty((b * t, h, spec.row_width), dtype=proj.dtype, device=proj.device)
    a.qbuf = qbuf.data_ptr()
    check(lib.axb_latent_prep(ctypes.byref(a), stream), "axb_latent_prep")
    # W_uk^T q per head, into the latent columns of qbuf.
    uk, uv = uk.to(proj.dtype).contiguous(), uv.to(proj.dtype).contiguous()
    skinny_ops.head_products(
        proj.as_strided((b * t, h, dk), (ld, dk + spec.rot_dim, 1), proj.storage_offset() + cols.q),
        uk.as_strided((h, spec.rot_offset, dk), (dk, uk.stride(0), 1), uk.storage_offset()), qbuf[..., :spec.rot_offset])
    lat_out = torch.empty((b * t, h, spec.rot_offset), dtype=proj.dtype, device=proj.device)
    a.out, a.out_ld = lat_out.data_ptr(), spec.rot_offset
    if form != "plain" and proj.dtype == torch.bfloat16 and lib.axb_latent_decode_supported(spec.row_width, spec.rank):
        ctas = b * t * -(-h // (32 if h > 16 else 16))
        a.splits = decode_splits(ctas, rows.shape[1])
        if a.splits > 1:
            part = torch.empty(b * t * h * a.splits * (spec.rot_offset + 2), dtype=torch.float32, device=proj.device)
            a.part, a.part_ml = part.data_ptr(), part[b * t * h * a.splits * spec.rot_offset:].data_ptr()
        check(lib.axb_latent_decode(ctypes.byref(a), stream), "axb_latent_decode")
    else:
        check(lib.axb_latent_attn(ctypes.byref(a), stream), "axb_latent_attn")
    skinny_ops.head_products(
        lat_out, uv.as_strided((h, dv, spec.rot_offset), (dv * uv.stride(0), uv.stride(0), 1), uv.storage_offset()),
        out.as_strided((b * t, h, dv), (spec.out_width, dv, 1)))
    if spec.out_width != h * dv:
        out[..., h * dv:] = 0
    return out, cache
