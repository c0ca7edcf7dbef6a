"""A drop-free mixture-of-experts feed-forward: sigmoid router, weights on the experts' inputs.

Reading side by side with ``mixture_of_experts`` (capacity, auxiliary losses, expert parallelism): this layer
keeps every (token, choice) pair, has no auxiliary loss, and runs prompts and single decoding tokens alike
(``ops/expert_ops.py``)."""

from __future__ import annotations

import torch

from axlearn_b200 import ops
from axlearn_b200.common.base_layer import BaseLayer, ParameterSpec
from axlearn_b200.common.config import REQUIRED, Required, config_class
from axlearn_b200.common.param_init import FanAxes
from axlearn_b200.common.sequence_mixer import PaddedLinear
from axlearn_b200.ops import expert_ops
from axlearn_b200.ops.hyper_ops import Gate, padded

Tensor = torch.Tensor


class RoutedFeedForward(BaseLayer):
    """``sum_k expert_(e_k)(s_k h)`` over the ``num_choices`` experts with the largest ``s = sigmoid(router h)``."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        hidden_dim: Required[int] = REQUIRED
        num_experts: Required[int] = REQUIRED
        num_choices: Required[int] = REQUIRED
        gate: Gate = Gate("silu")

    def __init__(self, cfg, *, parent=None):
        if not 1 <= cfg.num_choices <= cfg.num_experts:
            raise ValueError(f"cannot choose {cfg.num_choices} of {cfg.num_experts} experts")
        super().__init__(cfg, parent=parent)
        self._add_child("router", PaddedLinear.default_config().set(
            input_dim=cfg.input_dim, output_dim=cfg.num_experts))

    def _create_layer_parameter_specs(self):
        cfg = self._config
        d, f = padded(cfg.input_dim, 64), padded(cfg.hidden_dim, 64)
        axes = FanAxes(batch_axis=0, in_axis=-1, out_axis=-2)
        return {
            "gate_up_weight": ParameterSpec(shape=(cfg.num_experts, 2 * f, d), mesh_axes=(None,) * 3, fan_axes=axes),
            "down_weight": ParameterSpec(shape=(cfg.num_experts, d, f), mesh_axes=(None,) * 3, fan_axes=axes),
        }

    def forward(self, x: Tensor) -> Tensor:
        cfg, p = self._config, self.parameters
        logits = ops.linear_f32(x, self.state["router"]["weight"].to(x.dtype).t())[..., :cfg.num_experts]
        return expert_ops.expert_feed_forward(
            x, logits, p["gate_up_weight"].to(x.dtype), p["down_weight"].to(x.dtype), top=cfg.num_choices, width=cfg.input_dim,
            hidden=cfg.hidden_dim, gate=cfg.gate)
