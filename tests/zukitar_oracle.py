"""Plain statements of the Zukitar mechanisms, one function each, one sequence at a time.

Everything is written token by token or with explicit loops over heads, in the dtype of the inputs
(tests use float64), and shares no code with ``axlearn_b200``.  ``weights`` maps the checkpoint's
tensor names to tensors, ``config`` is the dictionary of ``config.json``.
"""

from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-torch.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_interleaved(x, position, dims, base):
    """Pairs (2i, 2i + 1) of the first ``dims`` entries of the last axis turn by ``position * base^(-2i/dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = position * base ** (-2 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_of(h, w, mixer, eps):
    """``(latent [T, rank], rotated shared key [T, rot_dim])`` of a sequence."""
    rank, rot = mixer["kv_rank"], mixer["rot"]
    both = h @ w["dkv"].T
    c = rms_norm(both[:, :rank], w["dkv.norm"], eps)
    kr = torch.stack([rotate_interleaved(both[t, rank:], t, rot["dims"], rot["base"]) for t in range(h.shape[0])])
    return c, kr


def latent_attention(h, w, mixer, eps):
    heads, dim, rdim, vdim = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    rot, t = mixer["rot"], h.shape[0]
    q = (h @ w["q"].T).reshape(t, heads, dim + rdim)
    c, kr = latent_of(h, w, mixer, eps)
    k = (c @ w["uk"].T).reshape(t, heads, dim)
    v = (c @ w["uv"].T).reshape(t, heads, vdim)
    out = torch.zeros(t, heads, vdim, dtype=h.dtype)
    for i in range(t):
        qr = rotate_interleaved(q[i, :, dim:], i, rot["dims"], rot["base"])
        for n in range(heads):
            s = (k[:i + 1, n] @ q[i, n, :dim] + kr[:i + 1] @ qr[n]) * mixer["scale"]
            p = torch.exp(s - s.max())
            out[i, n] = (p / p.sum()) @ v[:i + 1, n]
    return out.reshape(t, heads * vdim) @ w["o"].T


def causal_conv_silu(x, weight, bias):
    """``x [T, C]``, ``weight [C, taps]`` (last column: the token itself), zeros ahead of the start."""
    t, taps = x.shape[0], weight.shape[1]
    out = torch.zeros_like(x)
    for i in range(t):
        acc = bias.clone()
        for j in range(taps):
            if i - j >= 0:
                acc = acc + weight[:, taps - 1 - j] * x[i - j]
        out[i] = silu(acc)
    return out


def ssd_recurrence(x, b, c, dt, a_log, d):
    """``x [T, H, P]``, ``b, c [T, G, N]``, ``dt [T, H]`` (after softplus) -> ``(y [T, H, P], state [H, N, P])``."""
    t, heads, p = x.shape
    groups, n = b.shape[1:]
    s = torch.zeros(heads, n, p, dtype=x.dtype)
    y = torch.zeros_like(x)
    for i in range(t):
        for h in range(heads):
            g = h // (heads // groups)
            s[h] = torch.exp(-torch.exp(a_log[h]) * dt[i, h]) * s[h] + dt[i, h] * torch.outer(b[i, g], x[i, h])
            y[i, h] = s[h].T @ c[i, g] + d[h] * x[i, h]
    return y, s


def gated_group_norm(y, z, w, groups, eps):
    t, inner = y.shape
    v = (y * silu(z)).reshape(t, groups, inner // groups)
    return rms(v, eps).reshape(t, inner) * w


def mamba2(h, w, mixer, eps):
    heads, p, n, g = mixer["heads"], mixer["vdim"], mixer["state"], mixer["groups"]
    inner, t = heads * p, h.shape[0]
    proj = h @ w["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * g * n], proj[:, 2 * inner + 2 * g * n:]
    xbc = causal_conv_silu(xbc, w["conv"], w["conv.b"])
    x = xbc[:, :inner].reshape(t, heads, p)
    b = xbc[:, inner:inner + g * n].reshape(t, g, n)
    c = xbc[:, inner + g * n:].reshape(t, g, n)
    y, _ = ssd_recurrence(x, b, c, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_group_norm(y.reshape(t, inner), z, w["norm"], mixer["norm_groups"], eps) @ w["o"].T


def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_expert(x, gate, up, down, limit):
    g = torch.clamp(x @ gate.T, max=limit)
    u = torch.clamp(x @ up.T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, router, top):
    """``(expert ids [T, top], weights [T, top])``: largest sigmoid scores, used as they are."""
    s = sigmoid(h @ router.T)
    ids = torch.stack([torch.sort(s[t], descending=True, stable=True).indices[:top] for t in range(h.shape[0])])
    return ids, torch.gather(s, 1, ids)


def mixture(h, w, mlp):
    ids, weights = route(h, w["router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t].tolist(), weights[t]):
            out[t] += clamped_expert(p * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"],
                                     mlp["expert"]["limit"])
    return out


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def run(tokens, weights, config):
    """``(logits [T, vocab], residual after every layer [layers, T, width])``."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens)]
    after = []
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{i}.")
        mix = {"latent_attention": latent_attention, "mamba2": mamba2}[layer["type"]]
        x = x + mix(rms_norm(x, w["norm1"], eps), sub(w, "mix."), layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w["norm2"], eps)
            x = x + (dense_ff(h, sub(w, "mlp.")) if mlp["kind"] == "dense" else mixture(h, sub(w, "mlp."), mlp))
        after.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T * config["logit_scale"]
    return logits, torch.stack(after)
