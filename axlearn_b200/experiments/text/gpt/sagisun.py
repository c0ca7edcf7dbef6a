"""Sagisun: a small decoder-only LM with two sequence mixers side by side in every layer.

* A layer's mixer is the mean of a gated sliding-window attention (no rotation; query temperature and a
  linear distance bias) and a gated linear attention, each RMS-normed (``common/sequence_mixer.py``).
* Several residual streams with learned read / write / mix weights instead of one residual, branches
  scaled by a constant (``common/hyper_connection.py``).
* Norm weights kept as offsets from one, SwiGLU feed-forward (a layer may lack it), a run of layers that may
  be repeated with the same weights, tied embeddings.

``model_config`` takes the dictionary of a checkpoint's ``config.json``; ``parameters`` maps its tensors to
the model's tree.  Sizes may differ from layer to layer.
"""

from __future__ import annotations

from typing import Any, Mapping, Optional, Union

import torch

from axlearn_b200.common import causal_lm
from axlearn_b200.common.config import InstantiableConfig
from axlearn_b200.common.decoder import Decoder
from axlearn_b200.common.embedding import TransformerTextEmbeddings
from axlearn_b200.common.hyper_connection import (
    GatedFeedForward,
    HyperConnection,
    HyperStackedTransformerLayer,
    HyperTransformerLayer,
    PaddedEmbedding,
)
from axlearn_b200.common.safetensors_io import TreeLoader
from axlearn_b200.common.sequence_mixer import GatedLinearAttention, GatedWindowAttention, ParallelMixer
from axlearn_b200.experiments.text.gpt.common import (
    MESH_AXIS_NAMES,
    adamw_decoupled_learner_config,
    get_trainer_config_fn,
    mesh_shape_from_axes,
)

ARCHITECTURE = "Sagisun"
Tensor = torch.Tensor
# Kernels of an inference process (a first run without a built library compiles these).
KERNEL_SOURCES = ("flash_fwd.cu", "flash_fwd_v3.cu", "gated_act.cu", "gemm.cu", "gemm_2cta.cu", "gla.cu", "hyper.cu",
                  "window_attn.cu")
# A window that never closes (a left mixer without a mask).
_NO_WINDOW = 1 << 30


def _mixer_config(entry: Mapping, *, gate_rank: int, eps: float) -> InstantiableConfig:
    if entry["type"] != "parallel":
        raise ValueError(f"unknown mixer type {entry['type']!r}")
    left, right = entry["mixer"]["left"], entry["mixer"]["right"]
    temp, mask = left.get("q_temp"), left.get("mask")
    return ParallelMixer.default_config().set(
        norm_eps=eps,
        left=GatedWindowAttention.default_config().set(
            num_heads=left["heads"], num_kv_heads=left["kv_heads"], per_head_dim=left["dim"], value_dim=left["vdim"],
            window=mask["size"] if mask else _NO_WINDOW, scale=float(left["scale"]), distance_bias=True,
            query_temp_coef=float(temp["coef"]) if temp else 0.0, query_temp_every=int(temp["every"]) if temp else 1),
        right=GatedLinearAttention.default_config().set(
            num_heads=right["heads"], per_head_dim=right["dim"], value_dim=right["vdim"], gate_rank=gate_rank,
            tau=float(right["tau"]), norm_eps=eps))


def model_config(config: Mapping[str, Any], *, gate_rank: Union[int, list] = 16,
                 scan_chunk: Optional[int] = None) -> causal_lm.Model.Config:
    """``config``: the dictionary of ``config.json``.  ``gate_rank``: width of the low-rank decay gate, of
    all layers or one per layer (a checkpoint gives it by the shape of its ``a1`` tensors)."""
    eps, streams, width = float(config["norm"]["eps"]), config["streams"], config["width"]
    ranks = gate_rank if isinstance(gate_rank, (list, tuple)) else [gate_rank] * len(config["layers"])
    layers = []
    for entry, rank in zip(config["layers"], ranks):
        mlp = entry.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        layers.append(HyperTransformerLayer.default_config().set(
            mixer=_mixer_config(entry, gate_rank=rank, eps=eps),
            feed_forward=None if mlp is None else GatedFeedForward.default_config().set(hidden_dim=mlp["ff"]),
            connection=HyperConnection.default_config().set(
                num_streams=streams, multiplier=float(config["residual_mult"]), norm_eps=eps)))
    loop = config.get("loop")
    stack = HyperStackedTransformerLayer.default_config().set(
        num_layers=len(layers), layer=layers, num_streams=streams, output_norm_eps=eps,
        loop=(loop["start"], loop["stop"], loop["times"]) if loop else None)
    decoder = Decoder.default_config().set(
        dim=width, vocab_size=config["vocab"], transformer=stack, output_norm=None,
        emb=TransformerTextEmbeddings.default_config().set(pos_emb=None, token_emb=PaddedEmbedding.default_config()))
    return causal_lm.Model.default_config().set(decoder=decoder, scan_chunk=scan_chunk)


def checkpoint_model_config(config: Mapping[str, Any], tensors: Mapping[str, Tensor]) -> causal_lm.Model.Config:
    """The model of a checkpoint: sizes from its ``config.json`` and tensor shapes."""
    ranks = [tensors[f"l{i}.mix.right.a1"].shape[0] for i in range(len(config["layers"]))]
    return model_config(config, gate_rank=ranks)


def parameters(model: causal_lm.Model, tensors: Mapping[str, Tensor], *, dtype: torch.dtype, device=None) -> dict:
    """The model's parameter tree from a checkpoint's tensors: projections packed, matrices zero-padded to
    their stored sizes and in ``dtype``, small vectors in fp32."""
    loader = TreeLoader(model, tensors, dtype=dtype)
    cfg = model.decoder.config
    d, stack = cfg.dim, model.decoder.transformer
    decoder = loader.tree["decoder"]
    loader.fill(decoder["emb"]["token_emb"]["weight"], "embed", (cfg.vocab_size, d))
    root = decoder["transformer"]
    loader.copy(root["output_norm_scale"], "final.norm", (d,))
    n = stack.config.num_streams
    for i in range(stack.config.num_layers):
        node, layer, pre = root[f"layer{i}"], getattr(stack, f"layer{i}"), f"l{i}."
        for q, name in enumerate(layer.sublayers(), start=1):
            c = node[f"{name}_connection"]
            loader.copy(c["norm_scale"], f"{pre}norm{q}", (d,))
            loader.copy(c["read"], f"{pre}hc{q}.in", (n,))
            loader.copy(c["write"], f"{pre}hc{q}.out", (n,))
            loader.copy(c["mix"], f"{pre}hc{q}.mix", (n, n))
        mixer = layer.mixer
        for side in ("left", "right"):
            sub, child, mpre = getattr(mixer, side), node["mixer"][side], f"{pre}mix.{side}."
            for name, rows in sub.sections():
                loader.fill(node["mixer"]["i_proj"]["weight"], mpre + name, (rows, d), mixer.columns()[side][name])
            s = sub.config
            loader.fill(child["o_proj"]["weight"], mpre + "o", (d, s.num_heads * s.value_dim))
            loader.copy(node["mixer"][f"{side}_norm_scale"], mpre + "out", (d,))
        s, child, mpre = mixer.right.config, node["mixer"]["right"], f"{pre}mix.right."
        keys = s.num_heads * s.per_head_dim
        loader.fill(child["gate_weight"], mpre + "a2", (keys, s.gate_rank))
        loader.copy(child["gate_bias"], mpre + "a2.b", (keys,))
        loader.copy(child["norm_scale"], mpre + "norm", (s.value_dim,))
        if "feed_forward" in layer.sublayers():
            ff, mlp = layer.feed_forward, node["feed_forward"]
            f = ff.config.hidden_dim
            loader.fill(mlp["linear1"]["weight"], f"{pre}mlp.gate", (f, d))
            loader.fill(mlp["linear1"]["weight"], f"{pre}mlp.up", (f, d), ff.up_offset())
            loader.fill(mlp["linear2"]["weight"], f"{pre}mlp.down", (d, f))
    return loader.finish(device)


# ------------------------------------------------------------------------------------------
# Named sizes.
# ------------------------------------------------------------------------------------------


def size_config(size: str, *, vocab_size: int = 32768) -> dict:
    """Configurations of the family; "1B" and "7B" have the layer widths of the Fuji models of that name."""
    sizes = {
        "test": dict(width=64, layers=3, heads=4, kv_heads=2, dim=16, rheads=2, rdim=16, rvdim=32, ff=96, window=16,
                     streams=2, loop=dict(start=1, stop=2, times=2)),
        "1B": dict(width=2048, layers=16, heads=16, kv_heads=4, dim=128, rheads=16, rdim=64, rvdim=128, ff=5632,
                   window=1024, streams=4, loop=None),
        "7B": dict(width=4096, layers=32, heads=32, kv_heads=8, dim=128, rheads=32, rdim=128, rvdim=128, ff=11008,
                   window=2048, streams=4, loop=None),
    }
    if size not in sizes:
        raise NotImplementedError(f"unknown model size {size}")
    s = sizes[size]
    layer = {
        "type": "parallel",
        "mixer": {
            "left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"],
                     "scale": s["dim"] ** -0.5, "mask": {"size": s["window"]}, "q_temp": {"coef": 0.1, "every": 8192}},
            "right": {"heads": s["rheads"], "dim": s["rdim"], "vdim": s["rvdim"], "tau": 16.0},
        },
        "mlp": {"kind": "dense", "ff": s["ff"]},
    }
    return {"architecture": ARCHITECTURE, "vocab": vocab_size, "width": s["width"], "streams": s["streams"],
            "residual_mult": 1.0, "norm": {"eps": 1e-5}, "layers": [layer] * s["layers"], "loop": s["loop"]}


def trainer_configs() -> dict:
    """``sagisun-<size>``."""

    def make(size: str, batch: int, seq: int, vocab: int):
        def fn():
            return get_trainer_config_fn(
                model_cfg=model_config(size_config(size, vocab_size=vocab)),
                learner_cfg=adamw_decoupled_learner_config(peak_lr=3e-4, max_step=10_000, weight_decay=0.1),
                max_step=10_000, train_batch_size=batch, max_sequence_length=seq, vocab_size=vocab,
                mesh_shape=mesh_shape_from_axes(data=-1), mesh_axis_names=MESH_AXIS_NAMES)()

        return fn

    return {"sagisun-test": make("test", 8, 32, 128), "sagisun-1B": make("1B", 64, 4096, 32768)}
