"""CUDA kernels of the gated window attention, the gated linear attention and the hyper-connections
against plain statements, over sizes, continuations, ragged rows and extreme decays."""

import pytest
import torch

from tests import sagisun_oracle as oracle
from axlearn_b200.ops import dispatch, gla_ops, hyper_ops, window_ops

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return 2e-5 if dtype == torch.float32 else 2e-2


def _close(got, want, tol):
    err = (got.double().cpu() - want.double().cpu()).abs().max().item()
    ref = want.abs().max().item()
    assert err <= tol * max(1.0, ref), (err, ref)


# ------------------------------------------------------------------------------ hyper-connections
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,streams", [((2, 7), 96, 4), ((1, 1), 256, 1), ((3, 5), 50, 2), ((2, 9), 1000, 3),
                                                ((1, 700), 512, 4), ((2, 3), 72, 5), ((1, 4), 64, 8), ((1, 2), 33, 16)])
@pytest.mark.parametrize("pair", [False, True])
def test_hyper_step(dtype, rows, width, streams, pair):
    g = torch.Generator().manual_seed(width + streams)
    rnd = lambda *s: torch.randn(*s, generator=g)
    ld = hyper_ops.padded(width, 32)
    x = rnd(*rows, streams, width)
    outs = [rnd(*rows, ld).to(dtype) * 3 for _ in range(2)]
    mix, out, read, norm = rnd(streams, streams), rnd(streams), rnd(streams), rnd(width)
    sa, sb = rnd(width), rnd(width)
    dev = lambda t: t.cuda()
    branch = (hyper_ops.NormedPair(dev(outs[0]), dev(outs[1]), dev(sa), dev(sb), 1e-5) if pair else dev(outs[0]))
    new, h = hyper_ops.hyper_step(
        dev(x), branch, write=hyper_ops.StreamWrite(dev(mix), dev(out), 0.7), read=dev(read), norm_scale=dev(norm),
        eps=1e-5, norm_offset=1.0, num_streams=streams, dtype=dtype)
    f = [o[..., :width].double() for o in outs]
    y = 0.5 * (oracle.rms(f[0], 1e-5) * sa.double() + oracle.rms(f[1], 1e-5) * sb.double()) if pair else f[0]
    want = oracle.hyper_write(x.double().movedim(2, 0), y, mix.double(), out.double(), 0.7)
    u = oracle.hyper_read(want, read.double())
    _close(new, want.movedim(0, 2), 1e-5)
    _close(h[..., :width], oracle.one_plus_norm(u, norm.double(), 1e-5), _tol(dtype) / 2)
    assert h.shape[-1] % 8 == 0 and (h[..., width:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_hyper_first_read_and_last_sum(dtype):
    x = torch.randn(2, 3, 40).to(dtype)
    read, norm = torch.randn(3), torch.randn(40)
    same, h = hyper_ops.hyper_step(x.cuda(), read=read.cuda(), norm_scale=norm.cuda(), eps=1e-6, num_streams=3,
                                   dtype=dtype)
    assert same.dim() == 3
    _close(h, oracle.one_plus_norm(x.double() * read.double().sum(), norm.double(), 1e-6), _tol(dtype))
    streams = torch.randn(2, 3, 3, 40)
    y = torch.randn(2, 3, 64).to(dtype)
    mix, out = torch.randn(3, 3), torch.randn(3)
    none, total = hyper_ops.hyper_step(streams.cuda(), y.cuda(), write=hyper_ops.StreamWrite(mix.cuda(), out.cuda(), 1.0),
                                       num_streams=3, dtype=dtype, keep_streams=False)
    assert none is None and total.dtype == torch.float32
    want = oracle.hyper_write(streams.double().movedim(2, 0), y[..., :40].double(), mix.double(), out.double(), 1.0)
    _close(total, want.sum(0), 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,up", [(64, 64), (50, 56), (1024, 1024)])
def test_gated_act(dtype, width, up):
    gu = torch.randn(5, hyper_ops.padded(up + width, 32)).to(dtype)
    got = hyper_ops.gated_act(gu.cuda(), width, up)
    want = oracle.silu(gu[:, :width].double()) * gu[:, up:up + width].double()
    _close(got[:, :width], want, _tol(dtype) / 2)
    assert (got[:, width:] == 0).all()


# ------------------------------------------------------------------------------ window attention
def _window_case(dtype, heads, kv, dim, vdim, b, t, seed=0):
    g = torch.Generator().manual_seed(seed)
    parts = {"q": heads * dim, "k": kv * dim, "v": kv * vdim, "g": heads * vdim}
    cols, at = {}, 0
    for name, n in parts.items():
        cols[name] = at
        at = hyper_ops.padded(at + n, 8)
    at = hyper_ops.padded(at, 32)
    proj = torch.randn(b, t, at, generator=g).to(dtype)
    return proj, window_ops.WindowColumns(**cols)


def _window_oracle(row, spec, cols):
    """One sequence ``[T, P]``."""
    t = row.shape[0]
    cut = lambda off, n, d: row[:, off:off + n * d].double().reshape(t, n, d)
    o = oracle.window_attention(cut(cols.q, spec.heads, spec.dim), cut(cols.k, spec.kv_heads, spec.dim),
                                cut(cols.v, spec.kv_heads, spec.vdim), scale=spec.scale, window=spec.window,
                                temperature=spec.q_temp, bias=spec.distance_bias)
    o = o.reshape(t, -1)
    return o * oracle.sigmoid(row[:, cols.g:cols.g + o.shape[1]].double()) if spec.gated else o


WINDOW_SIZES = [  # heads, kv heads, dim, value dim, window
    (4, 2, 56, 32, 20), (2, 2, 64, 64, 33), (8, 1, 128, 128, 64), (4, 4, 128, 64, 300), (3, 1, 40, 72, 17),
    (6, 3, 20, 12, 9), (2, 1, 96, 128, 1), (4, 1, 160, 144, 50), (5, 5, 7, 5, 11), (4, 2, 64, 128, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", WINDOW_SIZES)
@pytest.mark.parametrize("t", [5, 150])
def test_window_prompt_then_single_tokens(dtype, sizes, t):
    heads, kv, dim, vdim, window = sizes
    spec = window_ops.WindowSpec(heads, kv, dim, vdim, window, scale=dim ** -0.5, q_temp=(0.7, 16), distance_bias=True)
    b, extra = 3, 40
    proj, cols = _window_case(dtype, heads, kv, dim, vdim, b, t + extra)
    live = torch.tensor([t, max(1, t - 3), max(1, t // 2)], dtype=torch.int32)
    slots = min(window, t + extra)
    cache = {"key": torch.zeros(b, slots, kv, dim, dtype=dtype, device="cuda"),
             "value": torch.zeros(b, slots, kv, vdim, dtype=dtype, device="cuda")}
    out, cache = window_ops.window_attention(proj[:, :t].cuda().contiguous(), spec, cols, live=live.cuda(), cache=cache)
    want = []
    for r in range(b):
        n = int(live[r])
        row = torch.cat([proj[r, :n], proj[r, t:]])
        want.append(_window_oracle(row, spec, cols))
        _close(out[r, :n, :heads * vdim], want[r][:n], _tol(dtype))
    assert (out[..., heads * vdim:] == 0).all()
    start = live.cuda()
    for i in range(extra):
        skip = torch.ones(b, dtype=torch.int32, device="cuda")
        one, cache = window_ops.window_attention(proj[:, t + i:t + i + 1].cuda().contiguous(), spec, cols, start=start,
                                                 live=skip, cache=cache)
        for r in range(b):
            _close(one[r, 0, :heads * vdim], want[r][int(live[r]) + i], _tol(dtype))
        start = start + 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 3, 16, 45])
def test_window_portions(dtype, portion):
    heads, kv, dim, vdim, window, t = 4, 2, 64, 64, 24, 90
    spec = window_ops.WindowSpec(heads, kv, dim, vdim, window, scale=0.2, q_temp=(0.3, 8), distance_bias=True)
    proj, cols = _window_case(dtype, heads, kv, dim, vdim, 2, t, seed=3)
    cache = {"key": torch.zeros(2, window, kv, dim, dtype=dtype, device="cuda"),
             "value": torch.zeros(2, window, kv, vdim, dtype=dtype, device="cuda")}
    outs = []
    for lo in range(0, t, portion):
        n = min(portion, t - lo)
        start = None if lo == 0 else torch.full((2,), lo, dtype=torch.int32, device="cuda")
        o, cache = window_ops.window_attention(proj[:, lo:lo + n].cuda().contiguous(), spec, cols, start=start,
                                               cache=cache)
        outs.append(o)
    got = torch.cat(outs, dim=1)
    for r in range(2):
        _close(got[r], _window_oracle(proj[r], spec, cols), _tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 128, 56])
def test_window_edge_shows(dtype, dim):
    """One key stands out; it is the last one inside the window, then the first one outside."""
    window, t, at = 70, 200, 90
    spec = window_ops.WindowSpec(1, 1, dim, dim, window, scale=1.0, distance_bias=False, gated=False)
    proj, cols = _window_case(torch.float32, 1, 1, dim, dim, 1, t, seed=1)
    proj *= 0.01
    proj[0, :, cols.q] = 6.0
    proj[0, at, cols.k] = 6.0          # score 36 against about 0
    proj[0, at, cols.v:cols.v + dim] = 1.0
    proj = proj.to(dtype)
    out, _ = window_ops.window_attention(proj.cuda(), spec, cols)
    value = out[0, :, 0].float().cpu()
    assert (value[at:at + window] > 0.9).all() and (value[at + window:].abs() < 0.1).all() and (value[:at].abs() < 0.1).all()
    cache = {"key": torch.zeros(1, window, 1, dim, dtype=dtype, device="cuda"),
             "value": torch.zeros(1, window, 1, dim, dtype=dtype, device="cuda")}
    _, cache = window_ops.window_attention(proj[:, :at + 60].cuda().contiguous(), spec, cols, cache=cache)
    for i in range(at + 60, at + 80):
        start = torch.tensor([i], dtype=torch.int32, device="cuda")
        one, cache = window_ops.window_attention(proj[:, i:i + 1].cuda().contiguous(), spec, cols, start=start, cache=cache)
        assert (one[0, 0, 0].item() > 0.9) == (i - at < window), i


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_long_decode_splits(dtype):
    """A window long enough to be split over CTAs, ring wrapped, one row out of the step."""
    heads, kv, dim, vdim, window = 8, 2, 128, 128, 1500
    spec = window_ops.WindowSpec(heads, kv, dim, vdim, window, scale=0.09, q_temp=(0.5, 100), distance_bias=True)
    b = 3
    proj, cols = _window_case(dtype, heads, kv, dim, vdim, b, 1, seed=5)
    start = torch.tensor([4000, 37, 1499], dtype=torch.int32)
    g = torch.Generator().manual_seed(2)
    key, value = torch.randn(b, window, kv, dim, generator=g).to(dtype), torch.randn(b, window, kv, vdim, generator=g).to(dtype)
    live = torch.tensor([1, 1, 0], dtype=torch.int32)
    got, cache = window_ops.window_attention(
        proj.cuda(), spec, cols, start=start.cuda(), live=live.cuda(), cache={"key": key.cuda(), "value": value.cuda()})
    with dispatch.use_reference_ops():
        want, ref = window_ops.window_attention(proj, spec, cols, start=start, live=live, cache={"key": key, "value": value})
    _close(got[:2], want[:2], _tol(dtype))
    assert (got[2] == 0).all()
    assert torch.equal(cache["key"].cpu(), ref["key"]) and torch.equal(cache["value"].cpu(), ref["value"])


# ------------------------------------------------------------------------------ linear attention
def _gla_case(dtype, heads, dim, vdim, rank, b, t, seed=0, z_scale=1.0, z_bias=1.5):
    g = torch.Generator().manual_seed(seed)
    parts = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim, "a1": rank}
    cols, at = {}, 0
    for name, n in parts.items():
        cols[name] = at
        at = hyper_ops.padded(at + n, 8)
    proj = torch.randn(b, t, hyper_ops.padded(at, 32), generator=g).to(dtype)
    a2 = (torch.randn(heads * dim, rank, generator=g) * z_scale * rank ** -0.5).to(dtype)
    bias = torch.randn(heads * dim, generator=g) + z_bias
    norm = 1 + 0.2 * torch.randn(vdim, generator=g)
    return proj, gla_ops.GlaColumns(**cols), a2, bias, norm


def _gla_oracle(row, cols, a2, bias, norm, spec, state=None):
    t = row.shape[0]
    cut = lambda off, d: row[:, off:off + spec.heads * d].double().reshape(t, spec.heads, d)
    z = row[:, cols.a1:cols.a1 + spec.rank].double() @ a2.double().T + bias.double()
    alpha = torch.exp(-torch.nn.functional.softplus(-z) / spec.tau).reshape(t, spec.heads, spec.dim)
    o, state = oracle.gated_linear_attention(cut(cols.q, spec.dim) * spec.q_scale, cut(cols.k, spec.dim),
                                             cut(cols.v, spec.vdim), alpha, state)
    o = (oracle.rms(o, spec.eps) * norm.double()).reshape(t, -1)
    return o * oracle.silu(row[:, cols.g:cols.g + o.shape[1]].double()), state


GLA_SIZES = [(3, 56, 64, 16), (2, 64, 128, 16), (1, 128, 128, 8), (2, 128, 64, 20), (2, 32, 256, 16), (4, 24, 40, 5),
             (2, 7, 9, 3), (1, 128, 200, 48), (1, 200, 64, 16), (5, 40, 24, 40)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", GLA_SIZES)
@pytest.mark.parametrize("tau,z_bias", [(16.0, 1.5), (1.0, 0.0), (0.25, -4.0)])
def test_gla_prompt_then_single_tokens(dtype, sizes, tau, z_bias):
    heads, dim, vdim, rank = sizes
    spec = gla_ops.GlaSpec(heads, dim, vdim, rank, tau, dim ** -0.5, 1e-5)
    b, t, extra = 2, 150, 6
    proj, cols, a2, bias, norm = _gla_case(dtype, heads, dim, vdim, rank, b, t + extra, z_bias=z_bias)
    live = torch.tensor([t, 70], dtype=torch.int32)
    args = [x.cuda() for x in (a2, bias, norm)]
    out, state = gla_ops.gated_linear_attention(proj[:, :t].cuda().contiguous(), *args, spec, cols, live=live.cuda())
    want, states = [], []
    for r in range(b):
        n = int(live[r])
        w, s = _gla_oracle(proj[r, :n], cols, a2, bias, norm, spec)
        _close(out[r, :n, :heads * vdim], w, 2 * _tol(dtype))
        _close(state[r], s, 1e-4)
        states.append(s)
    assert (out[1, 70:] == 0).all() and (out[..., heads * vdim:] == 0).all()
    for i in range(extra):
        alive = torch.tensor([1, 0 if i == 2 else 1], dtype=torch.int32, device="cuda")
        one, state = gla_ops.gated_linear_attention(
            proj[:, t + i:t + i + 1].cuda().contiguous(), *args, spec, cols, start=live.cuda() + i, live=alive, state=state)
        for r in range(b):
            if alive[r] == 0:
                assert (one[r] == 0).all()
                continue
            w, states[r] = _gla_oracle(proj[r, t + i:t + i + 1], cols, a2, bias, norm, spec, states[r])
            _close(one[r, 0, :heads * vdim], w[0], 2 * _tol(dtype))
            _close(state[r], states[r], 1e-4)


@pytest.mark.parametrize("sizes", [(2, 64, 64, 16), (2, 128, 128, 16), (2, 40, 256, 16)])
@pytest.mark.parametrize("tau", [16.0, 0.5])
def test_gla_segments_and_portions_agree(sizes, tau):
    heads, dim, vdim, rank = sizes
    spec = gla_ops.GlaSpec(heads, dim, vdim, rank, tau, dim ** -0.5, 1e-5)
    t = 700
    proj, cols, a2, bias, norm = _gla_case(torch.bfloat16, heads, dim, vdim, rank, 2, t, seed=4)
    p = proj.cuda()
    args = [x.cuda() for x in (a2, bias, norm)]
    live = torch.tensor([t, 333], dtype=torch.int32, device="cuda")
    run = lambda x, **kw: gla_ops._cuda_gla(x, *args, spec, cols, start=None, **kw)  # pylint: disable=protected-access
    o1, s1 = run(p, live=live, state=None, segments=(1, 704))
    o2, s2 = run(p, live=live, state=None, segments=(3, 256))
    o3, s3 = run(p, live=live, state=None, kernel="scan")
    _close(o2, o1, 1e-2), _close(s2, s1, 1e-4), _close(o3, o1, 2e-2), _close(s3, s1, 1e-4)
    state, outs = None, []
    for lo, hi in ((0, 2), (2, 66), (66, 333), (333, t)):
        o, state = gla_ops.gated_linear_attention(p[:1, lo:hi].contiguous(), *args, spec, cols, state=state)
        outs.append(o)
    _close(torch.cat(outs, dim=1)[0], o1[0], 1e-2), _close(state[0], s1[0], 1e-4)


def test_gla_state_carries_a_far_key():
    """One key / value pair far back is found by a query that matches it when nothing decays."""
    heads, dim, vdim, rank, t = 1, 64, 64, 16, 500
    spec = gla_ops.GlaSpec(heads, dim, vdim, rank, 16.0, 1.0, 1e-5)
    proj, cols, a2, bias, norm = _gla_case(torch.float32, heads, dim, vdim, rank, 1, t)
    proj *= 0.01
    proj[0, 3, cols.k] = 8.0
    proj[0, 3, cols.v + 5] = 8.0
    proj[0, t - 1, cols.q] = 8.0
    proj[0, :, cols.g:cols.g + vdim] = 4.0
    for keep, bias_value in ((True, 40.0), (False, -40.0)):
        for dtype in DTYPES:
            out, _ = gla_ops.gated_linear_attention(
                proj.to(dtype).cuda(), (a2 * 0).to(dtype).cuda(), torch.full_like(bias, bias_value).cuda(),
                torch.ones_like(norm).cuda(), spec, cols)
            assert (out[0, -1].float().argmax().item() == 5 and out[0, -1, 5].item() > 10) == keep
