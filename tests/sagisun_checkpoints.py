"""Random Sagisun checkpoints for tests: ``config.json`` dictionaries and tensors by name."""

from __future__ import annotations

import json
import os

import torch

from axlearn_b200.common.safetensors_io import write_safetensors


def left(heads, kv_heads, dim, vdim, window, coef=0.4, every=32, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
            "q_temp": {"coef": coef, "every": every}, "scale": dim ** -0.5 if scale is None else scale}


def right(heads, dim, vdim, tau=16.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def layer(l, r, ff):
    return {"type": "parallel", "mixer": {"left": l, "right": r},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, streams=3, loop=None, mult=0.6, eps=1e-5):
    out = {"architecture": "Sagisun", "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult,
           "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CONFIGS = {
    # Every layer different, a looped middle, a layer without feed-forward.
    "mixed": config(152, 80, [
        layer(left(4, 2, 24, 16, 12), right(3, 20, 24), 112),
        layer(left(6, 3, 16, 32, 30, coef=0.9, every=7), right(2, 40, 16, tau=4.0), None),
        layer(left(2, 1, 40, 40, 5), right(5, 8, 8, tau=1.0), 72)], streams=3, loop=(0, 2, 3), mult=0.4),
    # Nothing divides by eight; head counts are not powers of two.
    "odd": config(67, 42, [
        layer(left(3, 3, 7, 5, 9), right(2, 9, 11, tau=2.0), 31),
        layer(left(5, 1, 10, 6, 17), right(1, 6, 13), 20)], streams=2, eps=1e-4),
    # One stream, one layer, one token visible, a loop that runs once.
    "ones": config(40, 16, [layer(left(1, 1, 8, 8, 1, coef=0.0, every=1), right(1, 8, 8, tau=1.0), 24)], streams=1,
                   loop=(0, 1, 1), mult=1.0),
    # Tensor-core head sizes, wide enough for the larger product tiles.
    "wide": config(512, 320, [
        layer(left(4, 1, 64, 128, 100), right(3, 64, 128), 416),
        layer(left(4, 4, 128, 64, 64), right(2, 128, 256), 640)], streams=4, loop=(1, 2, 2)),
    "five": config(96, 64, [layer(left(2, 2, 32, 32, 48), right(2, 32, 32), 64)] * 2, streams=5),
}


def random_tensors(cfg, *, rank=12, seed=0):
    """bf16 tensors under the checkpoint's names; scaled so that every part of the model matters."""
    g = torch.Generator().manual_seed(seed)
    d, n, out = cfg["width"], cfg["streams"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain * cols ** -0.5).bfloat16()

    def vec(name, size, mean=0.0, std=0.2):
        out[name] = (mean + std * torch.randn(size, generator=g)).bfloat16()

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g).bfloat16()
    vec("final.norm", d)
    for i, entry in enumerate(cfg["layers"]):
        p = f"l{i}."
        l, r = entry["mixer"]["left"], entry["mixer"]["right"]
        for q in (1, 2) if entry["mlp"] is not None else (1,):
            vec(f"{p}norm{q}", d)
            vec(f"{p}hc{q}.in", n, 1.0 / n, 0.1)
            vec(f"{p}hc{q}.out", n, 1.0, 0.3)
            out[f"{p}hc{q}.mix"] = (torch.eye(n) * 0.9 + 0.1 * torch.randn(n, n, generator=g)).bfloat16()
        a = f"{p}mix.left."
        mat(a + "q", l["heads"] * l["dim"], d)
        mat(a + "k", l["kv_heads"] * l["dim"], d)
        mat(a + "v", l["kv_heads"] * l["vdim"], d)
        mat(a + "g", l["heads"] * l["vdim"], d)
        mat(a + "o", d, l["heads"] * l["vdim"])
        vec(a + "out", d, 1.0)
        b = f"{p}mix.right."
        mat(b + "q", r["heads"] * r["dim"], d)
        mat(b + "k", r["heads"] * r["dim"], d)
        mat(b + "v", r["heads"] * r["vdim"], d)
        mat(b + "g", r["heads"] * r["vdim"], d)
        mat(b + "o", d, r["heads"] * r["vdim"])
        mat(b + "a1", rank, d)
        mat(b + "a2", r["heads"] * r["dim"], rank, 1.5)
        vec(b + "a2.b", r["heads"] * r["dim"], 1.5, 1.5)
        vec(b + "norm", r["vdim"], 1.0)
        vec(b + "out", d, 1.0)
        if entry["mlp"] is not None:
            f = entry["mlp"]["ff"]
            mat(f"{p}mlp.gate", f, d)
            mat(f"{p}mlp.up", f, d)
            mat(f"{p}mlp.down", d, f)
    return out


def save(folder, cfg, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return str(folder)
