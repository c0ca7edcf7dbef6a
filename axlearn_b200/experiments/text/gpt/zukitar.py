"""Zukitar: a small decoder-only LM whose layers mix by latent attention or by a state-space recurrence.

* ``latent_attention``: one cached low-rank vector per token for the keys and values of all heads, and a
  rotated key part they share; ``mamba2``: short convolution, scalar-decay matrix state, gated group norm
  (``common/sequence_mixer.py``).
* Feed-forwards: gelu-gated dense, or a sigmoid-routed mixture of clamped experts whose weights scale the
  experts' inputs (``common/routed_experts.py``); a layer may lack one.
* An ordinary fp32 residual, plain RMS norms, tied embeddings with a constant logit scale.

``model_config`` takes the dictionary of a checkpoint's ``config.json``; ``parameters`` maps its tensors to
the model's tree.  Sizes and kinds may differ from layer to layer.
"""

from __future__ import annotations

from typing import Any, Mapping, Optional

import torch

from axlearn_b200.common import causal_lm
from axlearn_b200.common.config import InstantiableConfig
from axlearn_b200.common.decoder import Decoder
from axlearn_b200.common.embedding import TransformerTextEmbeddings
from axlearn_b200.common.hyper_connection import (
    GatedFeedForward,
    HyperStackedTransformerLayer,
    HyperTransformerLayer,
    PaddedEmbedding,
    ResidualConnection,
)
from axlearn_b200.common.routed_experts import RoutedFeedForward
from axlearn_b200.common.safetensors_io import TreeLoader
from axlearn_b200.common.sequence_mixer import LatentAttention, StateSpaceMixer
from axlearn_b200.experiments.text.gpt.common import (
    MESH_AXIS_NAMES,
    adamw_decoupled_learner_config,
    get_trainer_config_fn,
    mesh_shape_from_axes,
)
from axlearn_b200.ops.hyper_ops import Gate

ARCHITECTURE = "Zukitar"
Tensor = torch.Tensor
# Kernels of an inference process (a first run without a built library compiles these).
KERNEL_SOURCES = ("experts.cu", "flash_fwd.cu", "flash_fwd_v3.cu", "gated_act.cu", "gemm.cu", "gemm_2cta.cu", "hyper.cu",
                  "latent_attn.cu", "skinny_group.cu", "ssd.cu")
# The experts' gate: g sigmoid(alpha g).
_EXPERT_ALPHA = 1.702


def _mixer_config(entry: Mapping, *, eps: float) -> InstantiableConfig:
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        rot = m["rot"]
        return LatentAttention.default_config().set(
            num_heads=m["heads"], per_head_dim=m["dim"], rotated_dim=m["rot_dim"], value_dim=m["vdim"],
            kv_rank=m["kv_rank"], scale=float(m["scale"]), rope_dims=rot["dims"], rope_theta=float(rot["base"]),
            norm_eps=eps)
    if entry["type"] == "mamba2":
        return StateSpaceMixer.default_config().set(
            num_heads=m["heads"], value_dim=m["vdim"], state_dim=m["state"], num_groups=m["groups"],
            conv_taps=m["conv"], num_norm_groups=m["norm_groups"], norm_eps=eps)
    raise ValueError(f"unknown mixer type {entry['type']!r}")


def _feed_forward_config(mlp: Optional[Mapping]) -> Optional[InstantiableConfig]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return GatedFeedForward.default_config().set(hidden_dim=mlp["ff"], gate=Gate("gelu_tanh"))
    if mlp["kind"] == "moe":
        expert, router = mlp["expert"], mlp["router"]
        return RoutedFeedForward.default_config().set(
            hidden_dim=expert["ff"], num_experts=router["experts"], num_choices=router["top"],
            gate=Gate("clamped", limit=float(expert["limit"]), alpha=_EXPERT_ALPHA))
    raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")


def model_config(config: Mapping[str, Any], *, scan_chunk: Optional[int] = None) -> causal_lm.Model.Config:
    """``config``: the dictionary of ``config.json``."""
    eps = float(config["norm"]["eps"])
    layers = [
        HyperTransformerLayer.default_config().set(
            mixer=_mixer_config(entry, eps=eps), feed_forward=_feed_forward_config(entry.get("mlp")),
            connection=ResidualConnection.default_config().set(norm_eps=eps))
        for entry in config["layers"]]
    stack = HyperStackedTransformerLayer.default_config().set(
        num_layers=len(layers), layer=layers, num_streams=1, output_norm_eps=eps, output_norm_offset=0.0,
        output_multiplier=float(config["logit_scale"]))
    decoder = Decoder.default_config().set(
        dim=config["width"], vocab_size=config["vocab"], transformer=stack, output_norm=None,
        emb=TransformerTextEmbeddings.default_config().set(pos_emb=None, token_emb=PaddedEmbedding.default_config()))
    return causal_lm.Model.default_config().set(decoder=decoder, scan_chunk=scan_chunk)


def checkpoint_model_config(config: Mapping[str, Any], tensors: Mapping[str, Tensor]) -> causal_lm.Model.Config:
    """The model of a checkpoint: everything is in its ``config.json``."""
    del tensors
    return model_config(config)


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
    for i in range(stack.config.num_layers):
        node, layer, pre = root[f"layer{i}"], getattr(stack, f"layer{i}"), f"l{i}."
        for q, name in enumerate(layer.sublayers(), start=1):
            loader.copy(node[f"{name}_connection"]["norm_scale"], f"{pre}norm{q}", (d,))
        load = _load_latent if isinstance(layer.mixer, LatentAttention) else _load_state_space
        load(loader, layer.mixer, node["mixer"], f"{pre}mix.", d)
        if "feed_forward" in layer.sublayers():
            load = _load_experts if isinstance(layer.feed_forward, RoutedFeedForward) else _load_dense
            load(loader, layer.feed_forward, node["feed_forward"], f"{pre}mlp.", d)
    return loader.finish(device)


def _load_latent(loader, mixer, node, pre, d):
    c, at = mixer.config, mixer.columns()
    h, rank = c.num_heads, c.kv_rank
    loader.fill(node["i_proj"]["weight"], pre + "q", (h * (c.per_head_dim + c.rotated_dim), d), row=at["q"])
    both = loader.take(pre + "dkv", (rank + c.rotated_dim, d))
    loader.put(node["i_proj"]["weight"], both[:rank], row=at["c"])
    loader.put(node["i_proj"]["weight"], both[rank:], row=at["r"])
    loader.copy(node["latent_norm_scale"], pre + "dkv.norm", (rank,))
    loader.put(node["key_weight"], loader.take(pre + "uk", (h * c.per_head_dim, rank)).t())
    loader.fill(node["value_weight"], pre + "uv", (h * c.value_dim, rank))
    loader.fill(node["o_proj"]["weight"], pre + "o", (d, h * c.value_dim))


def _load_state_space(loader, mixer, node, pre, d):
    c, at = mixer.config, mixer.columns()
    inner = c.num_heads * c.value_dim
    channels = inner + 2 * c.num_groups * c.state_dim
    rows = loader.take(pre + "in", (inner + channels + c.num_heads, d)).split([inner, channels, c.num_heads])
    for name, part in zip(("z", "xbc", "dt"), rows):
        loader.put(node["i_proj"]["weight"], part, row=at[name])
    loader.put(node["conv_weight"], loader.take(pre + "conv", (channels, c.conv_taps)).t())
    loader.copy(node["conv_bias"], pre + "conv.b", (channels,))
    for name, key in (("dt_bias", "dt_bias"), ("a_log", "A_log"), ("d", "D")):
        loader.copy(node[name], pre + key, (c.num_heads,))
    loader.copy(node["norm_scale"], pre + "norm", (inner,))
    loader.fill(node["o_proj"]["weight"], pre + "o", (d, inner))


def _load_dense(loader, ff, node, pre, d):
    f = ff.config.hidden_dim
    loader.fill(node["linear1"]["weight"], pre + "gate", (f, d))
    loader.fill(node["linear1"]["weight"], pre + "up", (f, d), row=ff.up_offset())
    loader.fill(node["linear2"]["weight"], pre + "down", (d, f))


def _load_experts(loader, ff, node, pre, d):
    c = ff.config
    f, half = c.hidden_dim, node["gate_up_weight"].shape[1] // 2
    loader.fill(node["router"]["weight"], pre + "router", (c.num_experts, d))
    for e in range(c.num_experts):
        loader.fill(node["gate_up_weight"][e], f"{pre}e{e}.gate", (f, d))
        loader.fill(node["gate_up_weight"][e], f"{pre}e{e}.up", (f, d), row=half)
        loader.fill(node["down_weight"][e], f"{pre}e{e}.down", (d, f))


# ------------------------------------------------------------------------------------------
# Named sizes.
# ------------------------------------------------------------------------------------------


def size_config(size: str, *, vocab_size: int = 32768) -> dict:
    """Configurations of the family: two state-space layers with a dense feed-forward for every latent
    attention layer with experts.  "1B" and "7B" have the widths of the Sagisun and Fuji models of that name."""
    sizes = {
        "test": dict(width=64, layers=3, heads=4, dim=16, rot=8, vdim=16, rank=32, sheads=4, svdim=32, state=16, groups=2,
                     ff=96, eff=48, experts=4, top=2),
        "1B": dict(width=2048, layers=18, heads=16, dim=128, rot=64, vdim=128, rank=512, sheads=64, svdim=64, state=128,
                   groups=1, ff=5632, eff=1408, experts=32, top=4),
        "7B": dict(width=4096, layers=33, heads=32, dim=128, rot=64, vdim=128, rank=512, sheads=128, svdim=64, state=128,
                   groups=2, ff=11008, eff=2048, experts=32, top=4),
    }
    if size not in sizes:
        raise NotImplementedError(f"unknown model size {size}")
    s = sizes[size]
    recurrent = {
        "type": "mamba2",
        "mixer": {"heads": s["sheads"], "vdim": s["svdim"], "state": s["state"], "groups": s["groups"], "conv": 4,
                  "norm_groups": s["groups"]},
        "mlp": {"kind": "dense", "ff": s["ff"]},
    }
    attention = {
        "type": "latent_attention",
        "mixer": {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "kv_rank": s["rank"],
                  "scale": (s["dim"] + s["rot"]) ** -0.5, "rot": {"base": 10000.0, "dims": s["rot"]}},
        "mlp": {"kind": "moe", "expert": {"ff": s["eff"], "limit": 7.0},
                "router": {"experts": s["experts"], "top": s["top"]}},
    }
    layers = [attention if i % 3 == 2 else recurrent for i in range(s["layers"])]
    return {"architecture": ARCHITECTURE, "vocab": vocab_size, "width": s["width"], "norm": {"eps": 1e-5},
            "logit_scale": 1.0, "layers": layers}


def trainer_configs() -> dict:
    """``zukitar-<size>``."""

    def make(size: str, batch: int, seq: int, vocab: int):
        def fn():
            return get_trainer_config_fn(
                model_cfg=model_config(size_config(size, vocab_size=vocab)),
                learner_cfg=adamw_decoupled_learner_config(peak_lr=3e-4, max_step=10_000, weight_decay=0.1),
                max_step=10_000, train_batch_size=batch, max_sequence_length=seq, vocab_size=vocab,
                mesh_shape=mesh_shape_from_axes(data=-1), mesh_axis_names=MESH_AXIS_NAMES)()

        return fn

    return {"zukitar-test": make("test", 8, 32, 128), "zukitar-1B": make("1B", 64, 4096, 32768)}
