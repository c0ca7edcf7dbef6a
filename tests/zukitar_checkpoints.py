"""Random Zukitar checkpoints for tests: ``config.json`` dictionaries and tensors by name.

Embeddings carry a code in their first columns, a block of columns per router, so that a token's choice of
experts is never a close call: rounding must not decide which expert a test compares."""

from __future__ import annotations

import json
import os

import torch

from axlearn_b200.common.safetensors_io import write_safetensors


def latent(heads, dim, rot_dim, vdim, rank, base=500.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, logit_scale=0.5, eps=1e-5):
    return {"architecture": "Zukitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


CONFIGS = {
    # Every layer different: groups unlike norm groups, value sizes unlike key sizes, both feed-forwards and none.
    "mixed": config(152, 80, [
        (mamba(6, 24, 20, 3, 4, 2), dense(112)),
        (latent(5, 24, 8, 40, 56), moe(40, 6, 2, 1.5)),
        (latent(3, 16, 24, 16, 24, base=2000.0), None),
        (mamba(4, 16, 40, 1, 2, 4), moe(24, 5, 3, 0.7))], logit_scale=0.6),
    # Nothing divides by eight.
    "odd": config(67, 42, [
        (latent(3, 7, 6, 5, 11), dense(31)),
        (mamba(3, 5, 7, 1, 3, 3), moe(13, 3, 1, 0.9)),
        (mamba(6, 3, 9, 2, 5, 1), None)], logit_scale=1.7, eps=1e-4),
    # One of everything.
    "ones": config(40, 16, [
        (mamba(1, 8, 8, 1, 1, 1), moe(8, 1, 1, 2.0)),
        (latent(1, 8, 2, 8, 8), dense(8))], logit_scale=1.0),
    # Tensor-core sizes.
    "wide": config(512, 320, [
        (mamba(8, 64, 128, 2, 4, 2), dense(416)),
        (latent(20, 128, 64, 128, 256), moe(160, 16, 4, 5.0)),
        (latent(4, 64, 32, 64, 192), moe(96, 8, 1, 1.0)),
        (mamba(2, 128, 64, 1, 4, 1), None)], logit_scale=0.25),
    "small": config(96, 64, [(mamba(4, 16, 16, 2, 4, 2), None), (latent(2, 16, 8, 16, 32), dense(64))]),
}


def random_tensors(cfg, *, seed=0):
    """bf16 tensors under the checkpoint's names; scaled so that every part of the model matters."""
    g = torch.Generator().manual_seed(seed)
    d, vocab, out = cfg["width"], cfg["vocab"], {}

    def normal(*shape, std=1.0):
        return torch.randn(*shape, generator=g) * std

    def linear(n, k, gain=1.0):
        return normal(n, k, std=gain * k ** -0.5)

    def near_one(*shape):
        return 1 + 0.2 * normal(*shape)

    embed, code = normal(vocab, d), {}
    experts = 0             # columns of all codes
    for i, layer in enumerate(cfg["layers"]):
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            n, top = layer["mlp"]["router"]["experts"], layer["mlp"]["router"]["top"]
            code[i] = experts
            for t in range(vocab):
                row = torch.full((n,), -3.0)
                row[torch.randperm(n, generator=g)[:top]] = 3.0
                embed[t, experts:experts + n] = row + 0.4 * normal(n)
            experts += n
    out["embed"] = embed
    out["final.norm"] = near_one(d)
    for i, layer in enumerate(cfg["layers"]):
        pre, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        out[pre + "norm1"] = near_one(d)
        if layer["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            out[pre + "mix.in"] = linear(2 * inner + 2 * gn + m["heads"], d)
            out[pre + "mix.conv"] = normal(inner + 2 * gn, m["conv"], std=0.6)
            out[pre + "mix.conv.b"] = normal(inner + 2 * gn, std=0.3)
            out[pre + "mix.dt_bias"] = normal(m["heads"]) - 1.5
            out[pre + "mix.A_log"] = normal(m["heads"]) - 1.0
            out[pre + "mix.D"] = near_one(m["heads"])
            out[pre + "mix.norm"] = near_one(inner)
            o = linear(d, inner)
        else:
            h, rank = m["heads"], m["kv_rank"]
            out[pre + "mix.q"] = linear(h * (m["dim"] + m["rot_dim"]), d, 1.5)
            out[pre + "mix.dkv"] = linear(rank + m["rot_dim"], d, 1.2)
            out[pre + "mix.dkv.norm"] = near_one(rank)
            out[pre + "mix.uk"] = linear(h * m["dim"], rank)
            out[pre + "mix.uv"] = linear(h * m["vdim"], rank)
            o = linear(d, h * m["vdim"])
        o[:experts] *= 0.1      # branches hardly write into the routers' columns
        out[pre + "mix.o"] = o
        if mlp is None:
            continue
        out[pre + "norm2"] = near_one(d)
        if mlp["kind"] == "dense":
            out[pre + "mlp.gate"], out[pre + "mlp.up"] = linear(mlp["ff"], d, 1.5), linear(mlp["ff"], d)
            out[pre + "mlp.down"] = linear(d, mlp["ff"])
            out[pre + "mlp.down"][:experts] *= 0.1
        else:
            n, f = mlp["router"]["experts"], mlp["expert"]["ff"]
            router = torch.zeros(n, d)
            router[:, code[i]:code[i] + n] = torch.eye(n)[torch.randperm(n, generator=g)]
            out[pre + "mlp.router"] = router + 0.01 * normal(n, d)
            out[pre + "norm2"][code[i]:code[i] + n] = 1.0
            for e in range(n):
                out[f"{pre}mlp.e{e}.gate"], out[f"{pre}mlp.e{e}.up"] = linear(f, d, 1.5), linear(f, d, 1.5)
                down = linear(d, f, 0.8)
                down[:experts] *= 0.1
                out[f"{pre}mlp.e{e}.down"] = down
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def save(folder, cfg, tensors) -> str:
    os.makedirs(str(folder), exist_ok=True)
    with open(os.path.join(str(folder), "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(str(folder), "model.safetensors"), tensors)
    return str(folder)
