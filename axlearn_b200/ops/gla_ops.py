"""Gated linear attention: a recurrent matrix state whose key channels decay each at their own rate.

Per head: ``S_t = diag(alpha_t) S_(t-1) + k_t v_t^T``, ``o_t = S_t^T (q_t * q_scale)`` with
``alpha_t = sigmoid(W_a2 a1_t + b)^(1 / tau)``; then ``rms(o) * norm * silu(gate)`` over the value size.
``gated_linear_attention`` serves prompts, continued prompts and single tokens from one packed
projection (columns q, k, v, gate and the low-rank gate input a1).  State, decays and norms are fp32.
GPU: ``csrc/gla.cu``, which updates the state in place.
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
class GlaSpec:
    heads: int
    dim: int
    vdim: int
    rank: int          # width of the low-rank gate input
    tau: float
    q_scale: float
    eps: float

    @property
    def out_width(self) -> int:
        return padded(self.heads * self.vdim, 8)


@dataclasses.dataclass(frozen=True)
class GlaColumns:
    q: int
    k: int
    v: int
    g: int
    a1: int


def reference_gated_linear_attention(proj, a2, a2_bias, norm_scale, spec: GlaSpec, cols: GlaColumns, *, live, state,
                                     chunk: int = 16):
    """Differentiable chunked statement.  ``state [B, H, dim, vdim]`` or None; decays inside a chunk are
    formed as ``exp(G_i - G_j)`` per channel, which is at most one, so any decay strength is safe."""
    b, t, _ = proj.shape
    h, dk, dv = spec.heads, spec.dim, spec.vdim
    take = lambda off, n: proj[..., off:off + n].float()
    q = take(cols.q, h * dk).reshape(b, t, h, dk) * spec.q_scale
    k = take(cols.k, h * dk).reshape(b, t, h, dk)
    v = take(cols.v, h * dv).reshape(b, t, h, dv)
    z = take(cols.a1, spec.rank) @ a2.float().t() + a2_bias.float()
    log_decay = (F.logsigmoid(z) / spec.tau).reshape(b, t, h, dk)
    dead = torch.arange(t, device=proj.device)[None] >= live[:, None]                       # [B, T]
    k = k.masked_fill(dead[:, :, None, None], 0.0)
    log_decay = log_decay.masked_fill(dead[:, :, None, None], 0.0)
    s = torch.zeros((b, h, dk, dv), dtype=torch.float32, device=proj.device) if state is None else state.float()
    outs = []
    for lo in range(0, t, chunk):
        qc, kc, vc = q[:, lo:lo + chunk], k[:, lo:lo + chunk], v[:, lo:lo + chunk]
        gc = log_decay[:, lo:lo + chunk].cumsum(dim=1)
        c = qc.shape[1]
        causal = torch.tril(torch.ones(c, c, dtype=torch.bool, device=proj.device))
        diff = (gc[:, :, None] - gc[:, None, :]).masked_fill(~causal[None, :, :, None, None], float("-inf"))
        scores = torch.einsum("bihd,bjhd,bijhd->bhij", qc, kc, diff.exp())
        outs.append(torch.einsum("bhij,bjhv->bihv", scores, vc) + torch.einsum("bihd,bhdv->bihv", qc * gc.exp(), s))
        end = gc[:, -1:]
        s = s * end[:, 0].exp()[..., None] + torch.einsum("bjhd,bjhv->bhdv", kc * (end - gc).exp(), vc)
    o = torch.cat(outs, dim=1)
    o = o * torch.rsqrt(o.pow(2).mean(dim=-1, keepdim=True) + spec.eps) * norm_scale.float()
    o = o.reshape(b, t, h * dv) * F.silu(take(cols.g, h * dv))
    o = o.masked_fill(dead[:, :, None], 0.0)
    return F.pad(o.to(proj.dtype), (0, spec.out_width - h * dv)), s


def gated_linear_attention(proj: Tensor, a2: Tensor, a2_bias: Tensor, norm_scale: Tensor, spec: GlaSpec,
                           cols: GlaColumns, *, start: Optional[Tensor] = None, live: Optional[Tensor] = None,
                           state: Optional[Tensor] = None):
    """``(out [B, T, out_width], state [B, H, dim, vdim])``.  start: int32 ``[B]``, only its sign matters
    here (negative: the row is not in this step).  live: int32 ``[B]`` valid tokens (None: T).  state: None
    starts from zero."""
    tensors = [proj, a2, a2_bias, norm_scale]
    grad = torch.is_grad_enabled() and any(x.requires_grad for x in tensors)
    if dispatch._cuda(*tensors) and not grad and proj.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        return _cuda_gla(proj, a2, a2_bias, norm_scale, spec, cols, start=start, live=live, state=state)
    b, t, _ = proj.shape
    if live is None:
        live = torch.full((b,), t, dtype=torch.int32, device=proj.device)
    if start is not None:
        live = torch.where(start < 0, torch.zeros_like(live), live)
    return reference_gated_linear_attention(proj, a2, a2_bias, norm_scale, spec, cols, live=live, state=state)


# ------------------------------------------------------------------------------------------
# CUDA.
# ------------------------------------------------------------------------------------------


class _Args(ctypes.Structure):
    """Mirrors ``axb::GlaArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "proj", "a2", "a2_bias", "norm_w", "state", "out", "o_raw", "seg_state", "seg_decay", "start", "live")] + [
        ("ld", ctypes.c_int64), ("out_ld", ctypes.c_int64)] + [(n, ctypes.c_int) for n in (
            "B", "T", "heads", "dim", "vdim", "rank", "q_off", "k_off", "v_off", "g_off", "a1_off", "act_bf16",
            "segments", "seg_tokens")] + [(n, ctypes.c_float) for n in ("inv_tau", "q_scale", "eps")]


_signatures_set = False
CHUNK_TOKENS = 64


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        for name in ("axb_gla_decode", "axb_gla_scan", "axb_gla_chunk"):
            getattr(h, name).argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
            getattr(h, name).restype = ctypes.c_int
        _signatures_set = True
    return h


def prompt_segments(b: int, t: int, heads: int, vdim: int, sms: int = 148) -> tuple[int, int]:
    """``(segments, tokens per segment)`` of a prompt pass: cut the prompt until about two CTAs per SM
    run at once, no shorter than 256 tokens; one segment when the sequences alone fill the GPU (a cut
    costs a second pass over k, v and the decays)."""
    ctas = b * heads * (-(-vdim // 128))
    want = min((2 * sms) // max(1, ctas), t // 256)
    if want < 3:        # two halves cost as much as they win
        return 1, padded(t, CHUNK_TOKENS)
    tokens = padded(-(-t // want), CHUNK_TOKENS)
    return -(-t // tokens), tokens


def _cuda_gla(proj, a2, a2_bias, norm_scale, spec, cols, *, start, live, state, segments: Optional[tuple] = None,
              kernel: Optional[str] = None):
    """``kernel``: "chunk" / "scan" overrides the choice for prompts; ``segments`` that of
    ``prompt_segments``."""
    from axlearn_b200.ops import cuda_ops
    from axlearn_b200.ops.window_ops import _int32

    lib = _lib()
    proj, a2 = proj.contiguous(), a2.to(proj.dtype).contiguous()
    a2_bias, norm_scale = a2_bias.float().contiguous(), norm_scale.float().contiguous()
    b, t, ld = proj.shape
    start, live = _int32(start), _int32(live)
    if state is None:
        state = torch.zeros((b, spec.heads, spec.dim, spec.vdim), dtype=torch.float32, device=proj.device)
    assert state.dtype == torch.float32 and state.is_contiguous()
    assert state.shape == (b, spec.heads, spec.dim, spec.vdim), (state.shape, spec)
    assert a2.shape == (spec.heads * spec.dim, spec.rank), (a2.shape, spec)
    out = torch.empty((b, t, spec.out_width), dtype=proj.dtype, device=proj.device)
    a = _Args()
    a.proj, a.a2, a.a2_bias, a.norm_w = proj.data_ptr(), a2.data_ptr(), a2_bias.data_ptr(), norm_scale.data_ptr()
    a.state, a.out = state.data_ptr(), out.data_ptr()
    a.start = None if start is None else start.data_ptr()
    a.live = None if live is None else live.data_ptr()
    a.ld, a.out_ld, a.B, a.T = ld, out.shape[-1], b, t
    a.heads, a.dim, a.vdim, a.rank = spec.heads, spec.dim, spec.vdim, spec.rank
    a.q_off, a.k_off, a.v_off, a.g_off, a.a1_off = cols.q, cols.k, cols.v, cols.g, cols.a1
    a.act_bf16 = int(proj.dtype == torch.bfloat16)
    a.inv_tau, a.q_scale, a.eps = 1.0 / spec.tau, spec.q_scale, spec.eps
    a.segments, a.seg_tokens = 1, padded(t, CHUNK_TOKENS)
    stream = cuda_ops._stream()  # pylint: disable=protected-access
    check = cuda_ops._check  # pylint: disable=protected-access
    if t == 1 and kernel is None:
        check(lib.axb_gla_decode(ctypes.byref(a), stream), "axb_gla_decode")
        return out, state
    if kernel is None:
        kernel = "chunk" if proj.dtype == torch.bfloat16 and spec.dim <= 128 and spec.rank <= 128 else "scan"
    scratch = []
    if kernel == "scan" or spec.vdim > 128:
        scratch.append(torch.empty((b, t, spec.heads, spec.vdim), dtype=torch.float32, device=proj.device))
        a.o_raw = scratch[-1].data_ptr()
    if kernel == "scan":
        check(lib.axb_gla_scan(ctypes.byref(a), stream), "axb_gla_scan")
        return out, state
    a.segments, a.seg_tokens = segments or prompt_segments(b, t, spec.heads, spec.vdim)
    if a.segments > 1:
        scratch.append(torch.empty((b, spec.heads, a.segments, spec.dim, spec.vdim), dtype=torch.float32,
                                   device=proj.device))
        scratch.append(torch.empty((b, spec.heads, a.segments, spec.dim), dtype=torch.float32, device=proj.device))
        a.seg_state, a.seg_decay = scratch[-2].data_ptr(), scratch[-1].data_ptr()
    check(lib.axb_gla_chunk(ctypes.byref(a), stream), "axb_gla_chunk")
    return out, state
