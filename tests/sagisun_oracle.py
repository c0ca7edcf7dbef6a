"""Plain statements of the Sagisun mechanisms, one function each, one sequence at a time.

Everything is written token by token or with explicit loops over heads, in the dtype of the inputs
(tests use float64), and shares no code with ``axlearn_b200``.  ``weights`` maps the checkpoint's
tensor names to tensors, ``config`` is the dictionary of ``config.json``.
"""

from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def query_temperature(position, coef, every):
    return 1 + coef * math.log((position + 1) // every + 1)


def distance_slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def visible(i, j, window):
    return 0 <= i - j < window


def window_attention(q, k, v, *, scale, window, temperature=None, bias=True):
    """``q [T, H, dim]``, ``k [T, G, dim]``, ``v [T, G, vdim]`` -> ``[T, H, vdim]``; ``temperature`` is
    ``(coef, every)``."""
    t, heads, _ = q.shape
    groups = k.shape[1]
    out = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        g = h // (heads // groups)
        slope = distance_slope(h, heads) if bias else 0.0
        for i in range(t):
            lo = max(0, i - window + 1)
            qi = q[i, h] * (query_temperature(i, *temperature) if temperature else 1.0)
            dist = i - torch.arange(lo, i + 1, dtype=q.dtype)
            s = (k[lo:i + 1, g] @ qi) * scale - slope * dist
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, g]
    return out


def left_branch(h, w, mixer):
    """The gated window-attention branch before its output norm; ``w`` maps 'q', 'k', ... to matrices."""
    t = h.shape[0]
    heads, groups, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = (h @ w["q"].T).reshape(t, heads, dim)
    k = (h @ w["k"].T).reshape(t, groups, dim)
    v = (h @ w["v"].T).reshape(t, groups, vdim)
    temp = mixer["q_temp"]
    o = window_attention(q, k, v, scale=mixer["scale"], window=mixer["mask"]["size"],
                         temperature=(temp["coef"], temp["every"]))
    o = o.reshape(t, heads * vdim) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def channel_decay(h, w, heads, dim, tau):
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    return torch.exp(-torch.log1p(torch.exp(-z)) / tau).reshape(h.shape[0], heads, dim)


def gated_linear_attention(q, k, v, alpha, state=None):
    """``q, k, alpha [T, H, dim]``, ``v [T, H, vdim]`` -> (``[T, H, vdim]``, state ``[H, dim, vdim]``)."""
    t, heads, dim = q.shape
    if state is None:
        state = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype)
    out = []
    for i in range(t):
        state = alpha[i][:, :, None] * state + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hd,hdv->hv", q[i], state))
    return torch.stack(out), state


def right_branch(h, w, mixer, eps):
    t = h.shape[0]
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    q = (h @ w["q"].T).reshape(t, heads, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(t, heads, dim)
    v = (h @ w["v"].T).reshape(t, heads, vdim)
    o, _ = gated_linear_attention(q, k, v, channel_decay(h, w, heads, dim, mixer["tau"]))
    o = (rms(o, eps) * w["norm"]).reshape(t, heads * vdim) * silu(h @ w["g"].T)
    return o @ w["o"].T


def parallel_mixer(h, w, mixer, eps):
    left = left_branch(h, sub(w, "left."), mixer["left"])
    right = right_branch(h, sub(w, "right."), mixer["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


def gated_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def hyper_read(streams, w_in):
    """``streams [S, T, D]`` -> ``[T, D]``."""
    return sum(w_in[s] * streams[s] for s in range(streams.shape[0]))


def hyper_write(streams, y, w_mix, w_out, multiplier):
    n = streams.shape[0]
    return torch.stack([sum(w_mix[s, t] * streams[s] for s in range(n)) + multiplier * w_out[t] * y
                        for t in range(n)])


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def layer_order(config):
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def forward(config, weights, tokens, *, dtype=torch.float64):
    """Logits ``[T, vocab]`` and the residual (sum of streams) after every layer run."""
    w = {k: (v if not v.is_floating_point() else v.to(dtype)) for k, v in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    streams = torch.stack([x] * config["streams"])
    residuals = []
    for i in layer_order(config):
        layer, lw = config["layers"][i], sub(w, f"l{i}.")
        u = one_plus_norm(hyper_read(streams, lw["hc1.in"]), lw["norm1"], eps)
        y = parallel_mixer(u, sub(lw, "mix."), layer["mixer"], eps)
        streams = hyper_write(streams, y, lw["hc1.mix"], lw["hc1.out"], m)
        if layer["mlp"] is not None:
            u = one_plus_norm(hyper_read(streams, lw["hc2.in"]), lw["norm2"], eps)
            streams = hyper_write(streams, gated_mlp(u, sub(lw, "mlp.")), lw["hc2.mix"], lw["hc2.out"], m)
        residuals.append(streams.sum(0))
    x = one_plus_norm(streams.sum(0), w["final.norm"], eps)
    return x @ w["embed"].T, torch.stack(residuals)
