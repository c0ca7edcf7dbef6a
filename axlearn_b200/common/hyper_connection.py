"""Pre-norm layers on several residual streams (hyper-connections), and stacks that loop over them.

``HyperConnection`` holds one sublayer's read, write and mix weights and its norm.
``HyperTransformerLayer`` is a sequence mixer and an optional feed-forward, each behind its own connection.
``HyperStackedTransformerLayer`` runs the layers in order; ``loop = (start, stop, times)`` runs layers
``start .. stop - 1`` that many times in a row with the same weights, every pass with its own state.

The stack walks the sublayers as one sequence: the write of one, the read of the next and the next norm are
a single operation (``hyper_ops.hyper_step``), and the last read is fused with the stack's output norm.
With one stream, a zero mix and unit weights this is the ordinary residual.
"""

from __future__ import annotations

from typing import NamedTuple, Optional, Sequence

import torch

from axlearn_b200 import ops
from axlearn_b200.common.attention import BaseStackedTransformerLayer, BaseTransformerLayer
from axlearn_b200.common.base_layer import BaseLayer, ParameterSpec
from axlearn_b200.common.config import REQUIRED, InstantiableConfig, Required, config_class
from axlearn_b200.common.layers import Embedding
from axlearn_b200.common.module import nowrap
from axlearn_b200.common.sequence_mixer import PaddedLinear, vector_spec
from axlearn_b200.ops import hyper_ops
from axlearn_b200.ops.hyper_ops import padded

Tensor = torch.Tensor


class _IdentityInitializer:
    def initialize(self, name, *, prng_key, shape, dtype, axes=None, device=None):  # pylint: disable=unused-argument
        return torch.eye(shape[0], dtype=dtype, device=device)


class HyperConnection(BaseLayer):
    """``u = sum_s read[s] x_s``, input ``norm(u)``; ``x_t <- sum_s mix[s, t] x_s + multiplier * write[t] y``.
    The norm's stored weight is an offset from ``norm_offset``."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        num_streams: Required[int] = REQUIRED
        multiplier: float = 1.0
        norm_eps: float = 1e-6
        norm_offset: float = 1.0

    class Parts(NamedTuple):
        read: Optional[Tensor]
        norm_scale: Tensor
        norm_eps: float
        norm_offset: float
        write: hyper_ops.StreamWrite

    def _create_layer_parameter_specs(self):
        cfg = self._config
        n = cfg.num_streams
        return {
            "read": vector_spec((n,), 1.0 / n),
            "write": vector_spec((n,), 1.0),
            "mix": ParameterSpec(shape=(n, n), dtype=torch.float32, mesh_axes=(None, None),
                                 initializer=_IdentityInitializer()),
            "norm_scale": vector_spec((cfg.input_dim,), 1.0 - cfg.norm_offset),
        }

    def forward(self) -> "HyperConnection.Parts":
        cfg, p = self._config, self.parameters
        return self.Parts(p["read"], p["norm_scale"], cfg.norm_eps, cfg.norm_offset,
                          hyper_ops.StreamWrite(p["mix"], p["write"], cfg.multiplier))


class ResidualConnection(BaseLayer):
    """The ordinary residual as a connection: input ``norm(x)``, ``x <- x + multiplier * y`` (one stream, fp32)."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        num_streams: int = 1
        multiplier: float = 1.0
        norm_eps: float = 1e-6
        norm_offset: float = 0.0

    def __init__(self, cfg, *, parent=None):
        if cfg.num_streams != 1:
            raise ValueError("an ordinary residual has one stream")
        super().__init__(cfg, parent=parent)

    def _create_layer_parameter_specs(self):
        cfg = self._config
        return {"norm_scale": vector_spec((cfg.input_dim,), 1.0 - cfg.norm_offset)}

    def forward(self) -> HyperConnection.Parts:
        cfg = self._config
        return HyperConnection.Parts(None, self.parameters["norm_scale"], cfg.norm_eps, cfg.norm_offset,
                                     hyper_ops.PLAIN_WRITE._replace(multiplier=cfg.multiplier))


class GatedFeedForward(BaseLayer):
    """``down(act(gate x, up x))`` with gate and up packed in one product; ``gate`` names the activation."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        hidden_dim: Required[int] = REQUIRED
        gate: hyper_ops.Gate = hyper_ops.Gate("silu")

    def __init__(self, cfg, *, parent=None):
        super().__init__(cfg, parent=parent)
        self._up = padded(cfg.hidden_dim, 8)
        self._add_child("linear1", PaddedLinear.default_config().set(
            input_dim=cfg.input_dim, output_dim=self._up + cfg.hidden_dim))
        self._add_child("linear2", PaddedLinear.default_config().set(
            input_dim=cfg.hidden_dim, output_dim=cfg.input_dim))

    @nowrap
    def up_offset(self) -> int:
        return self._up

    def forward(self, x: Tensor) -> Tensor:
        cfg = self._config
        return self.linear2(hyper_ops.gated_act(self.linear1(x), cfg.hidden_dim, self._up, cfg.gate))


class HyperTransformerLayer(BaseTransformerLayer):
    @config_class
    class Config(BaseTransformerLayer.Config):
        mixer: Required[InstantiableConfig] = REQUIRED
        feed_forward: Optional[InstantiableConfig] = None
        connection: InstantiableConfig = HyperConnection.default_config()

    def __init__(self, cfg, *, parent=None):
        super().__init__(cfg, parent=parent)
        self._names = ["mixer"] + (["feed_forward"] if cfg.feed_forward is not None else [])
        for name in self._names:
            self._add_child(name, getattr(cfg, name).clone(input_dim=cfg.input_dim))
            self._add_child(f"{name}_connection", cfg.connection.clone(input_dim=cfg.input_dim))

    @nowrap
    def sublayers(self) -> list:
        return list(self._names)

    @nowrap
    def init_layer_states(self, **kwargs) -> dict:
        return {"mixer": self._children["mixer"].init_states(**kwargs)}

    def connections(self) -> dict:
        return {name: getattr(self, f"{name}_connection")() for name in self._names}

    def run_sublayer(self, name: str, h: Tensor, *, start=None, live=None, state=None):
        """``(branch, new state)`` of one sublayer on its normed input."""
        if name == "feed_forward":
            return self.feed_forward(h), state
        branch, mixed = self.mixer(h, start=start, live=live, state=None if state is None else state["mixer"])
        return branch, (None if state is None else {"mixer": mixed})


class HyperStackedTransformerLayer(BaseStackedTransformerLayer):
    """``forward`` / ``extend_step`` return the NORMED sum of the streams: a decoder on this stack has no
    output norm of its own."""

    # The step is a fixed list of kernels on in-place states: decode engines may capture it in a graph.
    GRAPH_DECODE = True

    @config_class
    class Config(BaseStackedTransformerLayer.Config):
        num_streams: int = 1
        # (start, stop, times): layers start .. stop - 1 run `times` times in a row.
        loop: Optional[tuple] = None
        output_norm_eps: float = 1e-6
        output_norm_offset: float = 1.0
        # Constant factor of the normed output (a logit scale ahead of a linear head).
        output_multiplier: float = 1.0

    def __init__(self, cfg, *, parent=None):
        super().__init__(cfg, parent=parent)
        layers: Sequence[InstantiableConfig] = (
            cfg.layer if isinstance(cfg.layer, (list, tuple)) else [cfg.layer] * cfg.num_layers)
        if len(layers) != cfg.num_layers:
            raise ValueError("number of layer configs must equal num_layers")
        self._layers = []
        for i, lc in enumerate(layers):
            lc = lc.clone(input_dim=cfg.input_dim)
            lc.connection.num_streams = cfg.num_streams
            self._layers.append(self._add_child(f"layer{i}", lc))
        order = list(range(cfg.num_layers))
        if cfg.loop is not None:
            start, stop, times = cfg.loop
            if not 0 <= start <= stop <= cfg.num_layers or times < 0:
                raise ValueError(f"loop {cfg.loop} does not fit {cfg.num_layers} layers")
            order = order[:start] + order[start:stop] * times + order[stop:]
        self._order = order

    def _create_layer_parameter_specs(self):
        cfg = self._config
        return {"output_norm_scale": vector_spec((cfg.input_dim,), 1.0 - cfg.output_norm_offset)}

    @nowrap
    def layer_order(self) -> list:
        """Index of the layer of every run, in order."""
        return list(self._order)

    def _run(self, data: Tensor, *, start=None, live=None, states: Optional[dict] = None):
        cfg = self._config
        parts = [layer.connections() for layer in self._layers]
        step = dict(num_streams=cfg.num_streams, dtype=data.dtype)
        streams, branch, write, new_states = data, None, None, {}
        for run, index in enumerate(self._order):
            layer = self._layers[index]
            state = None if states is None else states[f"run{run}"]
            for name in layer.sublayers():
                c = parts[index][name]
                streams, h = hyper_ops.hyper_step(
                    streams, branch, write=write, read=c.read, norm_scale=c.norm_scale, eps=c.norm_eps,
                    norm_offset=c.norm_offset, **step)
                branch, state = layer.run_sublayer(name, h, start=start, live=live, state=state)
                write = c.write
            new_states[f"run{run}"] = state
        _, h = hyper_ops.hyper_step(
            streams, branch, write=write, read=None, norm_scale=self.parameters["output_norm_scale"],
            eps=cfg.output_norm_eps, norm_offset=cfg.output_norm_offset, keep_streams=False,
            h_multiplier=cfg.output_multiplier, **step)
        return new_states, self.Output(data=h)

    def forward(self, data, *, target_segment_ids=None, target_positions=None, return_aux=None, **kwargs):
        if kwargs or return_aux:
            raise NotImplementedError(f"unsupported arguments: {sorted(kwargs)} {return_aux}")
        if target_segment_ids is not None and bool((target_segment_ids != target_segment_ids[:, :1]).any()):
            raise NotImplementedError("packed sequences: recurrent states do not stop at segment borders")
        return self._run(data)[1]

    @nowrap
    def _empty_states(self, data, max_len: int) -> dict:
        b = data.shape[0]
        device = getattr(data, "device", None)
        states = {f"run{r}": self._layers[i].init_layer_states(
            batch_size=b, max_len=max_len, dtype=data.dtype or torch.float32, device=device)
            for r, i in enumerate(self._order)}
        states["time_step"] = torch.zeros(b, dtype=torch.int32, device=device)
        return states

    def init_states(self, *, time_step, data, max_len=None, page_pool=None, **kwargs):
        if page_pool is not None or kwargs:
            raise NotImplementedError(f"unsupported arguments: page_pool, {sorted(kwargs)}")
        states = self._empty_states(data, max_len or data.shape[1])
        if time_step is None:
            return states, None
        live = time_step.to(torch.int32)
        new, out = self._run(data, live=live, states=states)
        new["time_step"] = live.clone()
        return new, out

    def extend_step(self, cached_states, data, *, live_step_len=None, page_pool=None, **kwargs):
        """``data [B, steps, D]`` after the tokens seen so far; ``live_step_len [B]``: valid new tokens per
        row (0 leaves the row alone)."""
        if page_pool is not None or kwargs:
            raise NotImplementedError(f"unsupported arguments: page_pool, {sorted(kwargs)}")
        start = cached_states["time_step"]
        new, out = self._run(data, start=start, live=live_step_len, states=cached_states)
        new["time_step"] = start + (data.shape[1] if live_step_len is None else live_step_len)
        return new, out


class PaddedEmbedding(Embedding):
    """A tied embedding whose table is rounded up like ``PaddedLinear`` (rows to 32, columns to 8) so that it
    is an operand of the output product as it lies; logits are fp32."""

    def _create_layer_parameter_specs(self):
        cfg = self._config
        spec = super()._create_layer_parameter_specs()["weight"]
        spec.shape = (padded(cfg.num_embeddings, 32), padded(cfg.dim, 8))
        spec.mesh_axes = (None, None)
        return {"weight": spec}

    def _weight(self) -> Tensor:
        return self.parameters["weight"][:self._config.num_embeddings]

    def forward(self, x: Tensor) -> Tensor:
        rows = torch.nn.functional.embedding(x.long(), self.parameters["weight"])
        return rows[..., :self._config.dim]

    def attend(self, x: Tensor) -> Tensor:
        w = self.parameters["weight"]
        return ops.linear_f32(x, w.to(x.dtype).t())[..., :self._config.num_embeddings]
