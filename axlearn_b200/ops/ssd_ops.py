"""State-space duality (Mamba-2): a matrix state per head with one scalar decay per token.

A token's projection holds an output gate ``z [inner]``, the convolved channels ``xbc`` = x ``[inner]``, B
``[G N]``, C ``[G N]``, and step sizes ``dt [H]`` (inner = H P; head h uses group ``h // (H / G)``)::

    xbc  <- silu(causal_conv(xbc))                       per channel, `taps` taps and a bias
    dt   <- softplus(dt + dt_bias)
    S_t   = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T      [N, P], fp32
    y_t   = S_t^T C_t + D x_t
    out   = rms over `norm_groups` equal parts of (y * silu(z)) * norm_w

State: ``{"ssm": fp32 [B, H, N, P], "conv": [B, taps, channels]}``; the convolution's inputs are a ring,
the input of position p in slot ``p % taps``.  ``ssd_mix`` takes ``start`` / ``live`` like the other mixers.
GPU: ``csrc/ssd.cu``, which updates the state in place.
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
class SsdSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int
    eps: float

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Convolved channels: x, B and C."""
        return self.inner + 2 * self.groups * self.state

    @property
    def out_width(self) -> int:
        return padded(self.inner, 8)


@dataclasses.dataclass(frozen=True)
class SsdColumns:
    z: int
    xbc: int
    dt: int


@dataclasses.dataclass(frozen=True)
class SsdWeights:
    """fp32 vectors; ``conv_w [taps, channels]``, last row = the token itself."""

    conv_w: Tensor
    conv_b: Tensor
    dt_bias: Tensor
    a_log: Tensor
    d: Tensor
    norm_w: Tensor


def reference_conv(x: Tensor, w: Tensor, bias: Tensor, *, start: Tensor, live: Tensor, ring: Optional[Tensor]):
    """``(silu(conv(x)), new ring)`` of fp32 ``x [B, T, C]``."""
    b, t, _ = x.shape
    taps = w.shape[0]
    pos = start.long()[:, None] + torch.arange(-(taps - 1), t, device=x.device)[None]      # [B, taps - 1 + T]
    rows = torch.arange(b, device=x.device)[:, None]
    before = x.new_zeros((b, taps - 1, x.shape[2]))
    if ring is not None and taps > 1:
        old = pos[:, :taps - 1]
        before = ring[rows, torch.remainder(old, taps)].to(x.dtype).masked_fill((old < 0)[..., None], 0.0)
    full = torch.cat([before, x], dim=1)
    y = bias + sum(w[j] * full[:, j:j + t] for j in range(taps))
    new_ring = None
    if ring is not None:
        step = torch.arange(t, device=x.device)[None]
        keep = (step < live[:, None]) & (step >= live[:, None] - taps)
        at, idx = torch.nonzero(keep, as_tuple=True)
        new_ring = ring.clone()
        new_ring[at, torch.remainder(pos[at, taps - 1 + idx], taps)] = x[at, idx].to(ring.dtype)
    return F.silu(y), new_ring


def reference_ssd(x, b, c, dt, a_log, d, s, chunk: int = 32):
    """Differentiable chunked recurrence.  ``x [B, T, H, P]``, ``b, c [B, T, G, N]``, ``dt [B, T, H]`` (zero
    where a token is dead), state ``s [B, H, N, P]`` -> ``(y, s)``; every decay is formed as an exponential
    of a non-positive number."""
    heads, groups, t = x.shape[2], b.shape[2], x.shape[1]
    b, c = (v.repeat_interleave(heads // groups, dim=2) for v in (b, c))
    log_decay = -torch.exp(a_log) * dt
    outs = []
    for lo in range(0, t, chunk):
        xc, bc, cc, dc = (v[:, lo:lo + chunk] for v in (x, b, c, dt))
        g = log_decay[:, lo:lo + chunk].cumsum(dim=1)                                       # [B, L, H]
        n = xc.shape[1]
        causal = torch.tril(torch.ones(n, n, dtype=torch.bool, device=x.device))
        diff = (g[:, :, None] - g[:, None]).masked_fill(~causal[None, :, :, None], float("-inf"))
        scores = torch.einsum("bihn,bjhn->bijh", cc, bc) * diff.exp() * dc[:, None]
        y = torch.einsum("bijh,bjhp->bihp", scores, xc)
        outs.append(y + torch.einsum("bihn,bhnp->bihp", cc * g.exp()[..., None], s))
        end = g[:, -1]
        w = (end[:, None] - g).exp() * dc
        s = s * end.exp()[:, :, None, None] + torch.einsum("bjhn,bjhp->bhnp", bc * w[..., None], xc)
    return torch.cat(outs, dim=1) + d[:, None] * x, s


def reference_ssd_mix(proj, w: SsdWeights, spec: SsdSpec, cols: SsdColumns, *, start, live, state):
    b, t, _ = proj.shape
    h, p, n, g, inner = spec.heads, spec.vdim, spec.state, spec.groups, spec.inner
    z = proj[..., cols.z:cols.z + inner].float()
    dead = torch.arange(t, device=proj.device)[None] >= live[:, None]
    xbc, ring = reference_conv(proj[..., cols.xbc:cols.xbc + spec.channels].float(), w.conv_w.float(), w.conv_b.float(),
                               start=start, live=live, ring=None if state is None else state["conv"])
    x = xbc[..., :inner].reshape(b, t, h, p)
    bb = xbc[..., inner:inner + g * n].reshape(b, t, g, n)
    cc = xbc[..., inner + g * n:].reshape(b, t, g, n)
    dt = F.softplus(proj[..., cols.dt:cols.dt + h].float() + w.dt_bias.float(), threshold=1e9)
    dt = dt.masked_fill(dead[..., None], 0.0)
    s = torch.zeros((b, h, n, p), device=proj.device) if state is None else state["ssm"].float()
    y, s = reference_ssd(x, bb, cc, dt, w.a_log.float(), w.d.float(), s)
    v = (y.reshape(b, t, inner) * F.silu(z)).reshape(b, t, spec.norm_groups, -1)
    v = (v * torch.rsqrt(v.pow(2).mean(dim=-1, keepdim=True) + spec.eps)).reshape(b, t, inner) * w.norm_w.float()
    out = F.pad(v.masked_fill(dead[..., None], 0.0).to(proj.dtype), (0, spec.out_width - inner))
    return out, (None if state is None else {"ssm": s, "conv": ring})


def ssd_mix(proj: Tensor, weights: SsdWeights, spec: SsdSpec, cols: SsdColumns, *, start: Optional[Tensor] = None,
            live: Optional[Tensor] = None, state: Optional[dict] = None):
    """``(out [B, T, out_width], state)``.  start: int32 ``[B]`` tokens the state has seen (None: zero);
    negative takes the row out of the step.  live: int32 ``[B]`` valid new tokens (None: T).  state None
    starts from zero and keeps nothing."""
    tensors = [proj] + [getattr(weights, f.name) for f in dataclasses.fields(weights)]
    grad = torch.is_grad_enabled() and any(x.requires_grad for x in tensors)
    if dispatch._cuda(*tensors) and not grad and proj.dtype in (torch.bfloat16, torch.float32):  # pylint: disable=protected-access
        return _cuda_ssd_mix(proj, weights, spec, cols, start=start, live=live, state=state)
    b, t, _ = proj.shape
    if live is None:
        live = torch.full((b,), t, dtype=torch.int32, device=proj.device)
    if start is None:
        start = torch.zeros(b, dtype=torch.int32, device=proj.device)
    live = torch.where(start < 0, torch.zeros_like(live), live)
    return reference_ssd_mix(proj, weights, spec, cols, start=start.clamp_min(0), live=live, state=state)


# ------------------------------------------------------------------------------------------
# CUDA.
# ------------------------------------------------------------------------------------------


class _Args(ctypes.Structure):
    """Mirrors ``axb::SsdArgs``."""

    _fields_ = [(n, ctypes.c_void_p) for n in (
        "proj", "conv_w", "conv_b", "dt_bias", "a_log", "d", "norm_w", "ssm", "ring", "xbc", "y", "out",
        "seg_state", "seg_decay", "start", "live")] + [(n, ctypes.c_int64) for n in (
            "ld", "xbc_ld", "out_ld")] + [(n, ctypes.c_int) for n in (
                "B", "T", "heads", "vdim", "state", "groups", "taps", "norm_groups", "z_off", "xbc_off", "dt_off",
                "act_bf16", "segments", "seg_tokens")] + [("eps", ctypes.c_float)]


_signatures_set = False
CHUNK_TOKENS = 64


def _lib():
    global _signatures_set
    from axlearn_b200.ops import cuda_ops

    h = cuda_ops.lib()
    if not _signatures_set:
        for name in ("axb_ssd_conv", "axb_ssd_decode", "axb_ssd_scan", "axb_ssd_chunk", "axb_ssd_norm"):
            getattr(h, name).argtypes = [ctypes.POINTER(_Args), ctypes.c_void_p]
            getattr(h, name).restype = ctypes.c_int
        _signatures_set = True
    return h


def prompt_segments(ctas: int, t: int, slots: int = 592) -> tuple[int, int]:
    """``(segments, tokens per segment)`` of a prompt pass that has ``ctas`` independent CTAs per segment: cut
    until ``slots`` of them run at once, no shorter than 256 tokens; a cut costs a second pass over x and B."""
    want = min(slots // max(1, ctas), t // 256)
    if want < 3:        # two halves cost as much as they win
        return 1, padded(t, CHUNK_TOKENS)
    tokens = padded(-(-t // want), CHUNK_TOKENS)
    return -(-t // tokens), tokens


def chunk_ctas(spec: SsdSpec) -> int:
    """CTAs per sequence of the chunked kernel: 64 value columns of a head each."""
    return spec.heads * -(-spec.vdim // 64)


def _cuda_ssd_mix(proj, w: SsdWeights, spec: SsdSpec, cols: SsdColumns, *, start, live, state,
                  kernel: Optional[str] = None, segments: Optional[tuple] = None):
    """``kernel``: "chunk" / "scan" overrides the choice for prompts; ``segments`` that of ``prompt_segments``."""
    from axlearn_b200.ops import cuda_ops
    from axlearn_b200.ops.window_ops import _int32

    lib = _lib()
    proj = proj.contiguous()
    b, t, ld = proj.shape
    start, live = _int32(start), _int32(live)
    decode = t == 1 and start is not None and state is not None and kernel is None
    if state is None:
        if start is not None:
            raise ValueError("a continued block needs its state")
        state = {"ssm": torch.zeros((b, spec.heads, spec.state, spec.vdim), dtype=torch.float32, device=proj.device),
                 "conv": torch.zeros((b, spec.taps, spec.channels), dtype=proj.dtype, device=proj.device)}
        keep = None
    else:
        keep = state
    ssm, ring = state["ssm"], state["conv"]
    assert ssm.dtype == torch.float32 and ssm.is_contiguous() and ring.is_contiguous() and ring.dtype == proj.dtype
    assert ssm.shape == (b, spec.heads, spec.state, spec.vdim) and ring.shape == (b, spec.taps, spec.channels)
    vectors = {name: getattr(w, name).float().contiguous() for name in (
        "conv_w", "conv_b", "dt_bias", "a_log", "d", "norm_w")}
    out = torch.empty((b, t, spec.out_width), dtype=proj.dtype, device=proj.device)
    a = _Args()
    for name, v in vectors.items():
        setattr(a, name, v.data_ptr())
    a.proj, a.ssm, a.ring, a.out = proj.data_ptr(), ssm.data_ptr(), ring.data_ptr(), out.data_ptr()
    a.start = None if start is None else start.data_ptr()
    a.live = None if live is None else live.data_ptr()
    a.ld, a.out_ld, a.xbc_ld, a.B, a.T = ld, out.shape[-1], padded(spec.channels, 8), b, t
    a.heads, a.vdim, a.state, a.groups, a.taps = spec.heads, spec.vdim, spec.state, spec.groups, spec.taps
    a.norm_groups, a.eps = spec.norm_groups, spec.eps
    a.z_off, a.xbc_off, a.dt_off = cols.z, cols.xbc, cols.dt
    a.act_bf16, a.segments, a.seg_tokens = int(proj.dtype == torch.bfloat16), 1, padded(t, CHUNK_TOKENS)
    y = torch.empty((b, t, spec.inner), dtype=proj.dtype, device=proj.device)
    a.y = y.data_ptr()
    stream = cuda_ops._stream()  # pylint: disable=protected-access
    check = cuda_ops._check  # pylint: disable=protected-access
    if decode:
        check(lib.axb_ssd_decode(ctypes.byref(a), stream), "axb_ssd_decode")
        check(lib.axb_ssd_norm(ctypes.byref(a), stream), "axb_ssd_norm")
        return out, keep
    xbc = torch.empty((b, t, a.xbc_ld), dtype=proj.dtype, device=proj.device)
    a.xbc = xbc.data_ptr()
    check(lib.axb_ssd_conv(ctypes.byref(a), stream), "axb_ssd_conv")
    if kernel is None:
        kernel = "chunk" if proj.dtype == torch.bfloat16 and spec.state <= 128 else "scan"
    if kernel == "scan":
        check(lib.axb_ssd_scan(ctypes.byref(a), stream), "axb_ssd_scan")
    else:
        a.segments, a.seg_tokens = segments or prompt_segments(b * chunk_ctas(spec), t)
        scratch = []
        if a.segments > 1:
            scratch.append(torch.empty((b, spec.heads, a.segments, spec.state, spec.vdim), dtype=torch.float32,
                                       device=proj.device))
            scratch.append(torch.empty((b, spec.heads, a.segments), dtype=torch.float32, device=proj.device))
            a.seg_state, a.seg_decay = scratch[0].data_ptr(), scratch[1].data_ptr()
        check(lib.axb_ssd_chunk(ctypes.byref(a), stream), "axb_ssd_chunk")
    check(lib.axb_ssd_norm(ctypes.byref(a), stream), "axb_ssd_norm")
    return out, keep
