"""Kernels of the latent attention, state-space and expert operations against their plain statements."""

import pytest
import torch

from axlearn_b200.ops import expert_ops, hyper_ops, latent_ops, skinny_ops, ssd_ops
from axlearn_b200.ops.dispatch import use_reference_ops
from axlearn_b200.ops.hyper_ops import padded

pytestmark = pytest.mark.gpu
BF16, F32 = torch.bfloat16, torch.float32


def _gen(seed):
    return torch.Generator(device="cuda").manual_seed(seed)


def _randn(*shape, seed, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=_gen(seed), device="cuda") * scale).to(dtype)


def _rel(got, want):
    return ((got.float() - want.float()).norm() / want.float().norm().clamp_min(1e-6)).item()


def _worst(got, want):
    """Largest difference over the reference's root mean square."""
    return ((got.float() - want.float()).abs().max() / want.float().pow(2).mean().sqrt().clamp_min(1e-6)).item()


def _ints(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------------------ latent attention
def _latent_case(spec, b, t, dtype, seed=0):
    widths = (spec.heads * (spec.dim + spec.rot_dim), spec.rank, spec.rot_dim)
    q, c = 0, padded(widths[0], 8)
    r = padded(c + widths[1], 8)
    ld = padded(r + widths[2], 32)
    proj = _randn(b, t, ld, seed=seed, dtype=dtype)
    norm = _randn(spec.rank, seed=seed + 1, scale=0.2) + 1
    uk = torch.zeros(padded(spec.rank, 8), padded(spec.heads * spec.dim, 32), device="cuda", dtype=dtype)
    uv = torch.zeros(padded(spec.heads * spec.vdim, 32), padded(spec.rank, 8), device="cuda", dtype=dtype)
    uk[:spec.rank, :spec.heads * spec.dim] = _randn(spec.rank, spec.heads * spec.dim, seed=seed + 2, scale=spec.rank ** -0.5)
    uv[:spec.heads * spec.vdim, :spec.rank] = _randn(spec.heads * spec.vdim, spec.rank, seed=seed + 3, scale=spec.rank ** -0.5)
    return proj, norm, uk, uv, latent_ops.LatentColumns(q, c, r)


def _latent_spec(heads, dim, rot, vdim, rank, rot_dims=None):
    return latent_ops.LatentSpec(heads, dim, rot, vdim, rank, rot if rot_dims is None else rot_dims, 1000.0,
                                 1.3 * (dim + rot) ** -0.5, 1e-5)


LATENT_SIZES = [(6, 64, 32, 48, 160), (16, 128, 64, 128, 512), (5, 40, 24, 72, 96), (33, 32, 8, 16, 264), (3, 7, 6, 5, 11),
                (2, 8, 8, 128, 8), (40, 128, 64, 64, 504), (2, 128, 64, 192, 640)]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("sizes", LATENT_SIZES)
@pytest.mark.parametrize("t", [1, 17, 128, 300])
def test_latent_prompt(sizes, t, dtype):
    spec = _latent_spec(*sizes)
    proj, norm, uk, uv, cols = _latent_case(spec, 2, t, dtype, seed=t)
    live = _ints(t, max(1, t - 5))
    cache = {"latent": torch.zeros(2, t + 9, spec.row_width, device="cuda", dtype=dtype)}
    with use_reference_ops():
        want, ref = latent_ops.latent_attention(proj, norm, uk, uv, spec, cols, live=live,
                                                cache={"latent": cache["latent"].clone()})
    got, _ = latent_ops.latent_attention(proj.clone(), norm, uk, uv, spec, cols, live=live, cache=cache)
    limit = 0.012 if dtype == BF16 else 3e-6
    for r in range(2):
        n = int(live[r])
        assert _rel(got[r, :n], want[r, :n]) < limit
    assert _worst(cache["latent"], ref["latent"]) < (0.04 if dtype == BF16 else 1e-5)
    alone, none = latent_ops.latent_attention(proj.clone(), norm, uk, uv, spec, cols, live=live)
    assert none is None and torch.equal(alone[0], got[0])


@pytest.mark.parametrize("dtype,form", [(BF16, None), (BF16, "plain"), (F32, None)])
@pytest.mark.parametrize("sizes", LATENT_SIZES)
@pytest.mark.parametrize("t", [1, 2, 5])
def test_latent_step(sizes, t, dtype, form):
    """New tokens after caches of unequal lengths: split edges, rows that are out, a full cache."""
    spec = _latent_spec(*sizes)
    slots, starts = 700, [0, 63, 64, 127, 128, 500, 700 - t, -1]
    b = len(starts)
    proj, norm, uk, uv, cols = _latent_case(spec, b, t, dtype, seed=7)
    rows = torch.zeros(b, slots, spec.row_width, device="cuda", dtype=dtype)
    rows[..., :spec.rank] = _randn(b, slots, spec.rank, seed=8, dtype=dtype)
    rows[..., spec.rot_offset:spec.rot_offset + spec.rot_dim] = _randn(b, slots, spec.rot_dim, seed=9, dtype=dtype)
    start, live = _ints(*starts), _ints(*[t] * (b - 2), max(1, t - 1), t)
    with use_reference_ops():
        want, ref = latent_ops.latent_attention(proj, norm, uk, uv, spec, cols, start=start, live=live,
                                                cache={"latent": rows.clone()})
    cache = {"latent": rows.clone()}
    got, _ = latent_ops._cuda_latent_attention(proj.clone(), norm, uk, uv, spec, cols, start=start, live=live, cache=cache,
                                               form=form)
    assert _worst(cache["latent"], ref["latent"]) < (0.04 if dtype == BF16 else 1e-5)
    for r in range(b - 1):
        n = int(live[r])
        assert _rel(got[r, :n], want[r, :n]) < (0.015 if dtype == BF16 else 3e-6), r
    assert got[-1].abs().max() == 0 and torch.equal(cache["latent"][-1], rows[-1])


@pytest.mark.parametrize("far", [0, 63, 64, 127, 128, 130, 191, 192, 639])
def test_one_cached_row_stands_out(far):
    """A key that outweighs hundreds of others, at the edges of tiles and splits: the output is its value."""
    spec = _latent_spec(8, 48, 24, 64, 192)
    proj, norm, uk, uv, cols = _latent_case(spec, 1, 1, BF16, seed=3)
    rows = torch.zeros(1, 640, spec.row_width, device="cuda", dtype=BF16)
    rows[..., :192] = _randn(1, 640, 192, seed=4, dtype=BF16)
    q = proj[0, 0, :8 * 72].reshape(8, 72).float()
    lat = torch.einsum("hd,rhd->hr", q[:, :48], uk[:, :8 * 48].float().reshape(192, 8, 48))
    rows[0, far, :192] = (lat[5] * 40 / lat[5].norm()).to(BF16)        # head 5 points there
    start = _ints(639)
    with use_reference_ops():
        want, _ = latent_ops.latent_attention(proj, norm, uk, uv, spec, cols, start=start, cache={"latent": rows.clone()})
    got, _ = latent_ops.latent_attention(proj.clone(), norm, uk, uv, spec, cols, start=start, cache={"latent": rows.clone()})
    value = (uv[:512].float() @ rows[0, far, :192].float()).reshape(8, 64)[5]
    if far != 639:      # the new token's own row is written by the step
        assert _rel(want[0, 0].reshape(8, 64)[5], value) < 0.05
    assert _rel(got, want) < 0.015


def test_rotated_dims_below_the_rotated_size():
    spec = _latent_spec(4, 32, 16, 32, 64, rot_dims=6)
    proj, norm, uk, uv, cols = _latent_case(spec, 1, 40, F32, seed=5)
    with use_reference_ops():
        want, _ = latent_ops.latent_attention(proj, norm, uk, uv, spec, cols)
    got, _ = latent_ops.latent_attention(proj.clone(), norm, uk, uv, spec, cols)
    assert _rel(got, want) < 3e-6


# ------------------------------------------------------------------------------ state-space mixing
def _ssd_case(spec, b, t, dtype, seed=0, slow=False):
    xbc = padded(spec.inner, 8)
    dt = padded(xbc + spec.channels, 8)
    cols = ssd_ops.SsdColumns(z=0, xbc=xbc, dt=dt)
    proj = _randn(b, t, padded(dt + spec.heads, 32), seed=seed, dtype=dtype)
    h = spec.heads
    a_log = torch.full((h,), -6.0, device="cuda") if slow else _randn(h, seed=seed + 3)
    w = ssd_ops.SsdWeights(
        conv_w=_randn(spec.taps, spec.channels, seed=seed + 1, scale=0.5), conv_b=_randn(spec.channels, seed=seed + 2, scale=0.3),
        dt_bias=_randn(h, seed=seed + 4) - 1, a_log=a_log, d=_randn(h, seed=seed + 5), norm_w=_randn(spec.inner, seed=seed + 6))
    return proj, w, cols


def _ssd_state(spec, b, dtype, seed):
    return {"ssm": _randn(b, spec.heads, spec.state, spec.vdim, seed=seed),
            "conv": _randn(b, spec.taps, spec.channels, seed=seed + 1, dtype=dtype)}


def _copy(state):
    return {k: v.clone() for k, v in state.items()}


SSD_SIZES = [(8, 64, 128, 1, 4, 1), (6, 40, 56, 2, 3, 3), (4, 16, 24, 4, 2, 2), (2, 128, 64, 1, 4, 1), (3, 5, 7, 3, 5, 3),
             (3, 80, 128, 1, 4, 2), (2, 200, 16, 2, 1, 1), (2, 32, 200, 1, 4, 1)]


def _ssd_spec(heads, vdim, state, groups, taps, norm_groups):
    return ssd_ops.SsdSpec(heads, vdim, state, groups, taps, norm_groups, 1e-5)


def _check_ssd(got, state, want, ref, live, dtype):
    for r, n in enumerate(live.tolist()):
        assert _rel(got[r, :n], want[r, :n]) < (0.01 if dtype == BF16 else 5e-6), r
        assert got[r, n:].abs().max() == 0 if n < got.shape[1] else True
    assert _rel(state["ssm"], ref["ssm"]) < (4e-3 if dtype == BF16 else 5e-6)
    assert torch.equal(state["conv"], ref["conv"])


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("sizes", SSD_SIZES)
@pytest.mark.parametrize("t", [1, 2, 63, 64, 65, 200])
def test_ssd_prompt(sizes, t, dtype):
    spec = _ssd_spec(*sizes)
    proj, w, cols = _ssd_case(spec, 3, t, dtype, seed=t)
    live = _ints(t, max(1, t - 3), max(1, t // 2))
    state = {k: torch.zeros_like(v) for k, v in _ssd_state(spec, 3, dtype, 0).items()}
    with use_reference_ops():
        want, ref = ssd_ops.ssd_mix(proj, w, spec, cols, live=live, state=_copy(state))
    got, _ = ssd_ops.ssd_mix(proj, w, spec, cols, live=live, state=state)
    _check_ssd(got, state, want, ref, live, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("sizes", SSD_SIZES)
@pytest.mark.parametrize("t", [1, 2, 3, 70])
def test_ssd_continues(sizes, t, dtype):
    """New tokens after unequal histories, shorter and longer than the convolution; one row out."""
    spec = _ssd_spec(*sizes)
    starts = [0, 1, 2, 3, 4, 777, -1]
    b = len(starts)
    proj, w, cols = _ssd_case(spec, b, t, dtype, seed=t + 1)
    state = _ssd_state(spec, b, dtype, 21)
    before, start, live = _copy(state), _ints(*starts), _ints(*[t] * (b - 2), max(1, t - 1), t)
    with use_reference_ops():
        want, ref = ssd_ops.ssd_mix(proj, w, spec, cols, start=start, live=live, state=_copy(state))
    got, _ = ssd_ops.ssd_mix(proj, w, spec, cols, start=start, live=live, state=state)
    live[-1] = 0
    _check_ssd(got, state, want, ref, live, dtype)
    assert all(torch.equal(state[k][-1], before[k][-1]) for k in state)


@pytest.mark.parametrize("sizes", SSD_SIZES[:4])
@pytest.mark.parametrize("segments", [(3, 128), (4, 64), (2, 192)])
def test_ssd_segments_and_slow_states(sizes, segments):
    """Segmented prompts equal whole ones, with states that reach from the first token to the last; the first
    segment's input stands out."""
    spec = _ssd_spec(*sizes)
    t = segments[0] * segments[1] - 30
    proj, w, cols = _ssd_case(spec, 2, t, BF16, seed=5, slow=True)
    proj[:, 2, cols.dt:cols.dt + spec.heads] = 8.0
    live = _ints(t, t // 2)
    zero = {k: torch.zeros_like(v) for k, v in _ssd_state(spec, 2, BF16, 0).items()}
    whole, cut = _copy(zero), _copy(zero)
    with use_reference_ops():
        want, ref = ssd_ops.ssd_mix(proj, w, spec, cols, live=live, state=_copy(zero))
    a, _ = ssd_ops._cuda_ssd_mix(proj, w, spec, cols, start=None, live=live, state=whole, segments=(1, padded(t, 64)))
    b, _ = ssd_ops._cuda_ssd_mix(proj, w, spec, cols, start=None, live=live, state=cut, segments=segments)
    _check_ssd(a, whole, want, ref, live, BF16)
    _check_ssd(b, cut, want, ref, live, BF16)


def test_ssd_chunk_keeps_small_differences():
    """The state is kept to fp32 accuracy: a large state that hardly decays plus small inputs."""
    spec = _ssd_spec(2, 64, 128, 1, 4, 1)
    proj, w, cols = _ssd_case(spec, 1, 256, BF16, seed=9, slow=True)
    state = _ssd_state(spec, 1, BF16, 3)
    state["ssm"].mul_(100)
    start = _ints(64)
    with use_reference_ops():
        _, ref = ssd_ops.ssd_mix(proj, w, spec, cols, start=start, state=_copy(state))
    chunk, scan = _copy(state), _copy(state)
    ssd_ops._cuda_ssd_mix(proj, w, spec, cols, start=start, live=None, state=chunk, kernel="chunk")
    ssd_ops._cuda_ssd_mix(proj, w, spec, cols, start=start, live=None, state=scan, kernel="scan")
    # The inputs' own bf16 rounding is the same in both kernels.
    assert _rel(chunk["ssm"], scan["ssm"]) < 2e-5 and _rel(chunk["ssm"], ref["ssm"]) < 1e-3


# ------------------------------------------------------------------------------ experts
EXPERT_SIZES = [(12, 1, 320, 72, 0.8), (32, 4, 512, 320, 7.0), (5, 5, 40, 24, 0.6), (300, 8, 64, 64, 2.0), (1, 1, 72, 8, 1.0),
                (7, 2, 42, 13, 1.5)]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("sizes", EXPERT_SIZES)
@pytest.mark.parametrize("tokens,path", [(1, None), (3, None), (40, None), (64, "skinny"), (700, None), (130, "sorted")])
def test_experts(sizes, tokens, path, dtype):
    experts, top, d, f, limit = sizes
    if path == "skinny" and tokens * top > 512:
        tokens = 512 // top
    dp, fp = padded(d, 64), padded(f, 64)
    h = torch.zeros(tokens, padded(d, 8), device="cuda", dtype=dtype)
    h[:, :d] = _randn(tokens, d, seed=1, dtype=dtype)
    # Logits on a grid that is far coarser than rounding: no close calls, but ties of experts that are not chosen.
    order = torch.stack([torch.randperm(experts, generator=_gen(t), device="cuda") for t in range(tokens)])
    logits = torch.where(order < top, 1.5 - 0.3 * order, -1.0).float()
    gate_up = torch.zeros(experts, 2 * fp, dp, device="cuda", dtype=dtype)
    down = torch.zeros(experts, dp, fp, device="cuda", dtype=dtype)
    gate_up[:, :f, :d] = _randn(experts, f, d, seed=2, scale=1.5 * d ** -0.5)
    gate_up[:, fp:fp + f, :d] = _randn(experts, f, d, seed=3, scale=1.5 * d ** -0.5)
    down[:, :d, :f] = _randn(experts, d, f, seed=4, scale=f ** -0.5)
    kw = dict(top=top, width=d, hidden=f, gate=hyper_ops.Gate("clamped", limit=limit))
    with use_reference_ops():
        want = expert_ops.expert_feed_forward(h, logits, gate_up, down, **kw)
    got = expert_ops._cuda_expert_feed_forward(h, logits, gate_up, down, path=path, **kw)
    assert got.shape == want.shape and _rel(got, want) < (0.01 if dtype == BF16 else 2e-6)


def test_equal_logits_choose_the_lower_experts():
    logits = torch.zeros(70, 40, device="cuda")
    logits[:, 11] = 1.0
    h = _randn(70, 64, seed=1, dtype=BF16)
    gate_up, down = _randn(40, 128, 64, seed=2, dtype=BF16, scale=0.2), _randn(40, 64, 64, seed=3, dtype=BF16, scale=0.2)
    kw = dict(width=64, hidden=64, gate=hyper_ops.Gate("clamped", limit=1.0))
    first = torch.full_like(logits, -60.0)
    first[:, 11], first[:, :2] = 1.0, 0.0
    for path in ("skinny", "sorted"):
        a = expert_ops._cuda_expert_feed_forward(h, logits, gate_up, down, top=3, path=path, **kw)
        b = expert_ops._cuda_expert_feed_forward(h, first, gate_up, down, top=3, path=path, **kw)
        assert _rel(a, b) < 1e-3


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("rows", [1, 7, 8, 9, 40, 100])
@pytest.mark.parametrize("heads,n,k", [(16, 512, 128), (5, 24, 40), (3, 7, 11), (2, 130, 72)])
def test_head_products(heads, n, k, rows, dtype):
    x, w = _randn(rows, heads, k, seed=1, dtype=dtype), _randn(heads, n, k, seed=2, dtype=dtype)
    out = torch.empty(rows, heads, n, device="cuda", dtype=dtype)
    skinny_ops.head_products(x, w, out)
    want = torch.einsum("rhk,hnk->rhn", x.double(), w.double())
    assert _rel(out, want) < (4e-3 if dtype == BF16 else 1e-6)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("kind", ["silu", "gelu_tanh", "clamped"])
@pytest.mark.parametrize("width", [96, 21])
def test_gates(kind, width, dtype):
    gate = hyper_ops.Gate(kind, limit=1.25)
    up = padded(width, 8)
    gu = _randn(33, padded(up + width, 32), seed=1, dtype=dtype, scale=3.0)
    gu[0, :8] = torch.tensor([-90.0, 90.0, -20, 20, 0, 1, -1, 5], device="cuda")
    got = hyper_ops.gated_act(gu, width, up, gate)
    want = hyper_ops.gate_values(gu[:, :width].double(), gu[:, up:up + width].double(), gate)
    assert _worst(got[:, :width], want) < (0.03 if dtype == BF16 else 2e-6) and bool(torch.isfinite(got.float()).all())


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [64, 42, 2048])
def test_plain_residual_step(width, dtype):
    x, y = _randn(2, 5, width, seed=1, dtype=dtype), _randn(2, 5, padded(width, 32), seed=2, dtype=dtype)
    kw = dict(write=hyper_ops.PLAIN_WRITE, read=None, norm_scale=_randn(width, seed=3), eps=1e-5, norm_offset=0.0,
              num_streams=1, dtype=dtype, h_multiplier=0.3)
    got_s, got_h = hyper_ops.hyper_step(x, y, **kw)
    with use_reference_ops():
        want_s, want_h = hyper_ops.hyper_step(x, y, **kw)
    assert got_s.dtype == F32 and _worst(got_s, want_s) < 1e-6 and _worst(got_h, want_h) < (0.02 if dtype == BF16 else 1e-5)
