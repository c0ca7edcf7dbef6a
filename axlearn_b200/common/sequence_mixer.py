"""Sequence mixers over packed projections: gated window attention, gated linear attention and the two side
by side; latent attention; state-space mixing (Mamba-2).

A mixer names the sections it needs of a token's projection (``sections``), and mixes along the sequence
given a projection that contains them (``mix``).  So several mixers that read the same input share ONE
input product (``ParallelMixer``), and a mixer alone has its own (``packed_input=False``).  One code path
serves training, prompts, continued prompts and decoding: ``start[b]`` tokens have been seen, ``live[b]``
of the T new ones are valid.

States are batch-leading tensors, so the decoding loops treat them like any KV cache.  On the GPU they are
updated in place.
"""

from __future__ import annotations

from typing import Any, Optional, Sequence

import torch

from axlearn_b200 import ops
from axlearn_b200.common.base_layer import BaseLayer, ParameterSpec
from axlearn_b200.common.config import REQUIRED, Required, config_class
from axlearn_b200.common.kv_cache import RingKVCache
from axlearn_b200.common.module import nowrap
from axlearn_b200.common.param_init import FanAxes, constant_initializer
from axlearn_b200.ops import gla_ops, hyper_ops, latent_ops, ssd_ops, window_ops
from axlearn_b200.ops.hyper_ops import padded

Tensor = torch.Tensor


def vector_spec(shape: Sequence[int], value: float) -> ParameterSpec:
    """A small fp32 parameter (norm weights, gate biases, stream mixing), replicated."""
    return ParameterSpec(shape=tuple(shape), dtype=torch.float32, mesh_axes=(None,) * len(shape),
                         initializer=constant_initializer(value))


class PaddedLinear(BaseLayer):
    """``x @ weight^T`` with ``weight [out, in]`` rounded up to what the matrix-product kernels take
    (``in`` to 8, ``out`` to 32).  Inputs are zero-padded to the rounded width by their producers; the
    surplus output columns mean nothing."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        output_dim: Required[int] = REQUIRED

    def _create_layer_parameter_specs(self):
        cfg = self._config
        return {"weight": ParameterSpec(
            shape=(padded(cfg.output_dim, 32), padded(cfg.input_dim, 8)), mesh_axes=(None, None),
            fan_axes=FanAxes(in_axis=-1, out_axis=-2))}

    def forward(self, x: Tensor) -> Tensor:
        return ops.linear(x, self.parameters["weight"].to(x.dtype).t())


_side_streams: dict = {}


def _side_stream(device: torch.device) -> "torch.cuda.Stream":
    index = device.index if device.index is not None else torch.cuda.current_device()
    if index not in _side_streams:
        _side_streams[index] = torch.cuda.Stream(device=index)
    return _side_streams[index]


class BaseSequenceMixer(BaseLayer):
    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        # The projection comes from the parent, which packs the sections of several mixers.
        packed_input: bool = False

    def __init__(self, cfg, *, parent=None):
        super().__init__(cfg, parent=parent)
        if not cfg.packed_input:
            self._columns, width = layout_sections(self.sections())
            self._add_child("i_proj", PaddedLinear.default_config().set(input_dim=cfg.input_dim, output_dim=width))

    @nowrap
    def columns(self) -> dict:
        """``{section: first column}`` of the own projection."""
        return self._columns

    @nowrap
    def sections(self) -> list:
        """``[(name, width)]`` of the projection columns this mixer reads."""
        raise NotImplementedError(type(self))

    @nowrap
    def init_states(self, *, batch_size: int, max_len: int, dtype: torch.dtype, device=None) -> dict:
        raise NotImplementedError(type(self))

    def mix(self, proj: Tensor, columns: dict, *, start=None, live=None, state=None) -> tuple[Tensor, Any]:
        """``(output projection of the mixed heads, new state)``."""
        raise NotImplementedError(type(self))

    def forward(self, x: Tensor, *, start=None, live=None, state=None) -> tuple[Any, Any]:
        return self.mix(self.i_proj(x), self._columns, start=start, live=live, state=state)


def layout_sections(sections: Sequence[tuple]) -> tuple[dict, int]:
    """``({name: first column}, total width)``; every section starts on a multiple of 8 columns."""
    columns, at = {}, 0
    for name, width in sections:
        columns[name] = at
        at = padded(at + width, 8)
    return columns, at


class GatedWindowAttention(BaseSequenceMixer):
    """Grouped-query attention inside a sliding window with an optional query temperature, linear
    distance bias and element-wise output gate (``ops/window_ops.py``)."""

    @config_class
    class Config(BaseSequenceMixer.Config):
        num_heads: Required[int] = REQUIRED
        num_kv_heads: Required[int] = REQUIRED
        per_head_dim: Required[int] = REQUIRED
        value_dim: Required[int] = REQUIRED
        window: Required[int] = REQUIRED          # positions seen, the query's own included
        scale: Required[float] = REQUIRED
        query_temp_coef: float = 0.0              # 0 = no temperature
        query_temp_every: int = 1
        distance_bias: bool = False
        output_gate: bool = True

    def __init__(self, cfg, *, parent=None):
        if cfg.num_heads % cfg.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        self._spec = window_ops.WindowSpec(
            heads=cfg.num_heads, kv_heads=cfg.num_kv_heads, dim=cfg.per_head_dim, vdim=cfg.value_dim,
            window=cfg.window, scale=cfg.scale, distance_bias=cfg.distance_bias, gated=cfg.output_gate,
            q_temp=(cfg.query_temp_coef, cfg.query_temp_every) if cfg.query_temp_coef else None)
        super().__init__(cfg, parent=parent)
        self._add_child("kv_cache", RingKVCache.default_config().set(window=cfg.window))
        self._add_child("o_proj", PaddedLinear.default_config().set(
            input_dim=cfg.num_heads * cfg.value_dim, output_dim=cfg.input_dim))

    @nowrap
    def sections(self) -> list:
        s = self._spec
        out = [("q", s.heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim)]
        return out + ([("g", s.heads * s.vdim)] if s.gated else [])

    @nowrap
    def init_states(self, *, batch_size, max_len, dtype, device=None):
        s = self._spec
        shape = RingKVCache.Shape(batch_size, max_len, s.kv_heads, s.dim, s.vdim)
        return self._children["kv_cache"].init_states(shape, dtype=dtype, device=device)

    def mix(self, proj, columns, *, start=None, live=None, state=None):
        out, state = window_ops.window_attention(proj, self._spec, window_ops.WindowColumns(**columns),
                                                 start=start, live=live, cache=state)
        return self.o_proj(out), state


class GatedLinearAttention(BaseSequenceMixer):
    """Linear attention with a per-channel data-dependent decay (``ops/gla_ops.py``), heads RMS-normed
    with a shared weight and gated by ``silu``."""

    @config_class
    class Config(BaseSequenceMixer.Config):
        num_heads: Required[int] = REQUIRED
        per_head_dim: Required[int] = REQUIRED
        value_dim: Required[int] = REQUIRED
        gate_rank: Required[int] = REQUIRED
        tau: float = 16.0
        query_scale: Optional[float] = None       # None = per_head_dim ** -0.5
        norm_eps: float = 1e-6

    def __init__(self, cfg, *, parent=None):
        scale = cfg.per_head_dim ** -0.5 if cfg.query_scale is None else cfg.query_scale
        self._spec = gla_ops.GlaSpec(heads=cfg.num_heads, dim=cfg.per_head_dim, vdim=cfg.value_dim,
                                     rank=cfg.gate_rank, tau=cfg.tau, q_scale=scale, eps=cfg.norm_eps)
        super().__init__(cfg, parent=parent)
        self._add_child("o_proj", PaddedLinear.default_config().set(
            input_dim=cfg.num_heads * cfg.value_dim, output_dim=cfg.input_dim))

    def _create_layer_parameter_specs(self):
        s = self._spec
        return {
            "gate_weight": ParameterSpec(shape=(s.heads * s.dim, s.rank), mesh_axes=(None, None),
                                         fan_axes=FanAxes(in_axis=-1, out_axis=-2)),
            "gate_bias": vector_spec((s.heads * s.dim,), 0.0),
            "norm_scale": vector_spec((s.vdim,), 1.0),
        }

    @nowrap
    def sections(self) -> list:
        s = self._spec
        return [("q", s.heads * s.dim), ("k", s.heads * s.dim), ("v", s.heads * s.vdim), ("g", s.heads * s.vdim),
                ("a1", s.rank)]

    @nowrap
    def init_states(self, *, batch_size, max_len, dtype, device=None):
        s = self._spec
        return torch.zeros((batch_size, s.heads, s.dim, s.vdim), dtype=torch.float32, device=device)

    def mix(self, proj, columns, *, start=None, live=None, state=None):
        p = self.parameters
        out, state = gla_ops.gated_linear_attention(
            proj, p["gate_weight"].to(proj.dtype), p["gate_bias"], p["norm_scale"], self._spec,
            gla_ops.GlaColumns(**columns), start=start, live=live, state=state)
        return self.o_proj(out), state


class LatentAttention(BaseSequenceMixer):
    """Attention whose keys and values come from one cached low-rank vector per token, with a rotated key
    part shared by all heads (``ops/latent_ops.py``)."""

    @config_class
    class Config(BaseSequenceMixer.Config):
        num_heads: Required[int] = REQUIRED
        per_head_dim: Required[int] = REQUIRED    # unrotated
        rotated_dim: Required[int] = REQUIRED
        value_dim: Required[int] = REQUIRED
        kv_rank: Required[int] = REQUIRED
        scale: Required[float] = REQUIRED
        rope_dims: Optional[int] = None           # None = rotated_dim
        rope_theta: float = 10000.0
        norm_eps: float = 1e-6

    def __init__(self, cfg, *, parent=None):
        rope_dims = cfg.rotated_dim if cfg.rope_dims is None else cfg.rope_dims
        if rope_dims % 2 or rope_dims > cfg.rotated_dim:
            raise ValueError(f"cannot rotate {rope_dims} of {cfg.rotated_dim} dimensions in pairs")
        self._spec = latent_ops.LatentSpec(
            heads=cfg.num_heads, dim=cfg.per_head_dim, rot_dim=cfg.rotated_dim, vdim=cfg.value_dim, rank=cfg.kv_rank,
            rot_dims=rope_dims, rot_base=cfg.rope_theta, scale=cfg.scale, eps=cfg.norm_eps)
        super().__init__(cfg, parent=parent)
        self._add_child("o_proj", PaddedLinear.default_config().set(
            input_dim=cfg.num_heads * cfg.value_dim, output_dim=cfg.input_dim))

    def _create_layer_parameter_specs(self):
        s = self._spec
        return {
            "latent_norm_scale": vector_spec((s.rank,), 1.0),
            # Keys: [rank, heads * dim], as a per-head matrix its rows are contiguous in both forms of the sum.
            "key_weight": ParameterSpec(shape=(padded(s.rank, 8), padded(s.heads * s.dim, 32)), mesh_axes=(None, None),
                                        fan_axes=FanAxes(in_axis=-2, out_axis=-1)),
            "value_weight": ParameterSpec(shape=(padded(s.heads * s.vdim, 32), padded(s.rank, 8)),
                                          mesh_axes=(None, None), fan_axes=FanAxes(in_axis=-1, out_axis=-2)),
        }

    @nowrap
    def sections(self) -> list:
        s = self._spec
        return [("q", s.heads * (s.dim + s.rot_dim)), ("c", s.rank), ("r", s.rot_dim)]

    @nowrap
    def init_states(self, *, batch_size, max_len, dtype, device=None):
        return {"latent": torch.zeros((batch_size, max_len, self._spec.row_width), dtype=dtype, device=device)}

    def mix(self, proj, columns, *, start=None, live=None, state=None):
        p = self.parameters
        out, state = latent_ops.latent_attention(
            proj, p["latent_norm_scale"], p["key_weight"], p["value_weight"], self._spec,
            latent_ops.LatentColumns(**columns), start=start, live=live, cache=state)
        return self.o_proj(out), state


class StateSpaceMixer(BaseSequenceMixer):
    """Mamba-2: a short convolution, a matrix state with a scalar decay per head, a gated group norm
    (``ops/ssd_ops.py``)."""

    @config_class
    class Config(BaseSequenceMixer.Config):
        num_heads: Required[int] = REQUIRED
        value_dim: Required[int] = REQUIRED
        state_dim: Required[int] = REQUIRED
        num_groups: int = 1
        conv_taps: int = 4
        num_norm_groups: int = 1
        norm_eps: float = 1e-6

    def __init__(self, cfg, *, parent=None):
        if cfg.num_heads % cfg.num_groups or (cfg.num_heads * cfg.value_dim) % cfg.num_norm_groups:
            raise ValueError("heads must split into groups, and channels into norm groups, evenly")
        self._spec = ssd_ops.SsdSpec(
            heads=cfg.num_heads, vdim=cfg.value_dim, state=cfg.state_dim, groups=cfg.num_groups, taps=cfg.conv_taps,
            norm_groups=cfg.num_norm_groups, eps=cfg.norm_eps)
        super().__init__(cfg, parent=parent)
        self._add_child("o_proj", PaddedLinear.default_config().set(
            input_dim=self._spec.inner, output_dim=cfg.input_dim))

    def _create_layer_parameter_specs(self):
        s = self._spec
        return {
            "conv_weight": ParameterSpec(shape=(s.taps, s.channels), dtype=torch.float32, mesh_axes=(None, None),
                                         fan_axes=FanAxes(in_axis=-2, out_axis=-1)),
            "conv_bias": vector_spec((s.channels,), 0.0),
            # Steps around 0.05 and decays around exp(-0.05) to begin with.
            "dt_bias": vector_spec((s.heads,), -3.0),
            "a_log": vector_spec((s.heads,), 0.0),
            "d": vector_spec((s.heads,), 1.0),
            "norm_scale": vector_spec((s.inner,), 1.0),
        }

    @nowrap
    def sections(self) -> list:
        s = self._spec
        return [("z", s.inner), ("xbc", s.channels), ("dt", s.heads)]

    @nowrap
    def init_states(self, *, batch_size, max_len, dtype, device=None):
        s = self._spec
        return {"ssm": torch.zeros((batch_size, s.heads, s.state, s.vdim), dtype=torch.float32, device=device),
                "conv": torch.zeros((batch_size, s.taps, s.channels), dtype=dtype, device=device)}

    def mix(self, proj, columns, *, start=None, live=None, state=None):
        p = self.parameters
        weights = ssd_ops.SsdWeights(conv_w=p["conv_weight"], conv_b=p["conv_bias"], dt_bias=p["dt_bias"],
                                     a_log=p["a_log"], d=p["d"], norm_w=p["norm_scale"])
        out, state = ssd_ops.ssd_mix(proj, weights, self._spec, ssd_ops.SsdColumns(**columns), start=start, live=live,
                                     state=state)
        return self.o_proj(out), state


class ParallelMixer(BaseLayer):
    """Two mixers that share one input: the mean of their outputs, each RMS-normed over the model
    width with a plain weight.  One product computes both mixers' projections.

    ``forward`` returns the two raw outputs as a ``NormedPair``; the norms and the mean are part of the
    residual update that follows (``hyper_ops.hyper_step`` / ``hyper_ops.combine_branch``)."""

    @config_class
    class Config(BaseLayer.Config):
        input_dim: Required[int] = REQUIRED
        left: Required[BaseSequenceMixer.Config] = REQUIRED
        right: Required[BaseSequenceMixer.Config] = REQUIRED
        norm_eps: float = 1e-6

    def __init__(self, cfg, *, parent=None):
        super().__init__(cfg, parent=parent)
        sections = []
        for side in ("left", "right"):
            mixer = self._add_child(side, getattr(cfg, side).clone(input_dim=cfg.input_dim, packed_input=True))
            sections += [((side, name), width) for name, width in mixer.sections()]
        columns, width = layout_sections(sections)
        self._columns = {side: {name: at for (s, name), at in columns.items() if s == side}
                         for side in ("left", "right")}
        self._add_child("i_proj", PaddedLinear.default_config().set(input_dim=cfg.input_dim, output_dim=width))

    def _create_layer_parameter_specs(self):
        d = self._config.input_dim
        return {"left_norm_scale": vector_spec((d,), 1.0), "right_norm_scale": vector_spec((d,), 1.0)}

    @nowrap
    def columns(self) -> dict:
        """``{side: {section: first column}}`` of the packed projection."""
        return self._columns

    @nowrap
    def init_states(self, **kwargs) -> dict:
        return {side: self._children[side].init_states(**kwargs) for side in ("left", "right")}

    def forward(self, x: Tensor, *, start=None, live=None, state=None):
        proj = self.i_proj(x)
        outs, states = {}, {}

        def mix(side):
            outs[side], states[side] = getattr(self, side).mix(
                proj, self._columns[side], start=start, live=live, state=None if state is None else state[side])

        if x.is_cuda and x.shape[1] == 1 and not torch.is_grad_enabled():
            # A decoding step's kernels are small: the two mixers run next to each other.  (The side stream's
            # tensors are read before the next fork, which orders their reuse.)
            main, side_stream = torch.cuda.current_stream(x.device), _side_stream(x.device)
            side_stream.wait_stream(main)
            with torch.cuda.stream(side_stream):
                mix("right")
            mix("left")
            main.wait_stream(side_stream)
        else:
            mix("left")
            mix("right")
        p = self.parameters
        pair = hyper_ops.NormedPair(outs["left"], outs["right"], p["left_norm_scale"], p["right_norm_scale"],
                                    self._config.norm_eps)
        return pair, states
