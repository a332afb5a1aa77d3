"""Typed configuration of the Sokalorn decoder (``"architecture": "Sokalorn"``).

config.json gives ``width``, ``vocab``, ``norm.eps``, optionally ``loop`` (``start``, ``stop``,
``times``: layers ``start .. stop - 1`` run ``times`` times in a row with the same tensors, each
pass with a cache and a state of its own; before each pass the residual x becomes ``W_in [x;
x0]``, x0 the embedding output), and the layers one by one: ``layers[i] = {"type": ..., "mixer":
{...}, "mlp": {"kind": "moe", ...} | null}``.

A layer has one norm and two sublayers side by side, ``x += mixer(n~) + ff(n)``, ``n =
norm1(x)``, the mixer reading the token-shifted ``n~ = n + (n' - n) * shift``.  Layer types:

* ``parallel``: the mean of two branches, each RMS-normed over the width.  ``left``: grouped-query
  attention in chunks of ``mask.size`` positions, rotate-half pairs over ``rot.dims`` features
  with base ``rot.base`` and frequencies divided by ``rot.scaling.factor``, scores scaled by
  ``scale`` and soft-capped at ``softcap``, sigmoid weights with a bias a head, a sigmoid gate a
  feature.  ``right``: RWKV-style time mixing (``heads`` of ``dim``; the rank of its decay's
  projection comes from the tensors' shapes);
* ``mamba2``: the state-space mixer (``heads`` of ``vdim``, ``state``, ``groups``, ``conv`` taps,
  ``norm_groups``).

The feed-forward is ``router.top`` of ``router.experts`` clamped gated experts
(``expert.{ff, limit}``) beside a shared one (``shared.{ff, limit}``) with a gate a token.
No size has a default; every size may differ from layer to layer.  A mechanism whose key is
absent or null (``mask``, ``softcap``, ``rot``, ``rot.scaling``, ``mlp``, ``mlp.shared``, ``loop``)
is left out.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from .base import ConfigError, ModelConfig
from .layout import (AttentionSpec, BlockSpec, LoopInputSpec, ModelLayout, NormSpec,
                     ParallelMixerSpec, PositionSpec, RopeScalingSpec, RoutedExpertsSpec, RunEntry,
                     StateSpaceSpec, TimeMixingSpec)
from .tifosun import _Reader

LAYER_TYPES = ("parallel", "mamba2")


@dataclass
class SokalornConfig(ModelConfig):
    width: int
    vocab: int
    norm_eps: float
    loop: Optional[tuple] = None                       # (start, stop, times)
    layers: list = field(default_factory=list)        # the raw layer objects of config.json
    stop_tokens: tuple = ()

    architecture = "Sokalorn"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "SokalornConfig":
        rd = _Reader()
        width = rd.get(raw, "config", "width", int)
        vocab = rd.get(raw, "config", "vocab", int)
        eps = rd.get(rd.get(raw, "config", "norm", dict), "config.norm", "eps", float)
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            rd.problems.append("config.layers must be a non-empty list")
            layers = []
        loop = None
        lp = rd.get(raw, "config", "loop", dict, default=None, required=False)
        if lp is not None:
            start, stop, times = (rd.get(lp, "config.loop", k, int) for k in
                                  ("start", "stop", "times"))
            if not (0 <= start < stop <= len(layers)) or times < 1:
                rd.problems.append(f"config.loop must name layers start < stop within the model "
                                   f"and times >= 1, got {dict(lp)!r}")
            else:
                loop = (start, stop, times)
        stops = raw.get("eos_token_id")
        if stops is None:
            stops = ()
        elif not isinstance(stops, (list, tuple)):
            stops = (stops,)
        cfg = cls(width=width, vocab=vocab, norm_eps=eps, loop=loop,
                  layers=copy.deepcopy(list(layers)), stop_tokens=tuple(int(t) for t in stops))
        rd.positive("config", width=width, vocab=vocab, **{"norm.eps": eps})
        if width > 0:
            cfg._blocks(rd)
        if rd.problems:
            raise ConfigError("unusable Sokalorn configuration: " + "; ".join(rd.problems))
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.stop_tokens:
            out["eos_token_id"] = list(self.stop_tokens)
        return out

    # -- what a checkpoint adds ---------------------------------------------
    def with_shapes(self, shape_of) -> "SokalornConfig":
        """The rank of the time mixing's decay projection is a size that only the tensors
        give (``shape_of(name)``: a checkpoint tensor's shape, or None); it is written into
        the layer's ``mixer.right`` as ``decay_rank``, the key under which a configuration may
        also state it itself."""
        for i, layer in enumerate(self.layers):
            if not isinstance(layer, Mapping) or layer.get("type") != "parallel":
                continue
            right = layer.get("mixer", {}).get("right")
            shape = shape_of(f"l{i}.mix.right.w1")
            if isinstance(right, dict) and shape is not None and len(shape) == 2:
                right["decay_rank"] = int(shape[0])
        return self

    # -- layers -------------------------------------------------------------
    def _left(self, rd: _Reader, path: str, m: Mapping) -> AttentionSpec:
        heads, kv_heads, dim, vdim = (rd.get(m, path, k, int)
                                      for k in ("heads", "kv_heads", "dim", "vdim"))
        scale = rd.get(m, path, "scale", float)
        rd.positive(path, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        if kv_heads > 0 and heads % kv_heads:
            rd.problems.append(f"{path}.heads ({heads}) is no multiple of kv_heads ({kv_heads})")
        position = PositionSpec(kind="none", head_dim=dim)
        rot = rd.get(m, path, "rot", dict, default=None, required=False)
        if rot is not None:
            base = rd.get(rot, path + ".rot", "base", float)
            dims = rd.get(rot, path + ".rot", "dims", int)
            rd.positive(path, **{"rot.base": base})
            scaling = rd.get(rot, path + ".rot", "scaling", dict, default=None, required=False)
            if scaling is not None:
                factor = rd.get(scaling, path + ".rot.scaling", "factor", float)
                rd.positive(path, **{"rot.scaling.factor": factor})
                scaling = RopeScalingSpec(rope_type="linear", factor=factor)
            if dims % 2 or not 0 <= dims <= dim:
                rd.problems.append(f"{path}.rot.dims must be even and at most dim, got {dims}")
            elif dims:
                position = PositionSpec(kind="rope", head_dim=dim, rotary_dim=dims, theta=base,
                                        scaling=scaling)
        cap = rd.get(m, path, "softcap", float, default=None, required=False)
        if cap is not None:
            rd.positive(path, softcap=cap)
        chunk = None
        mask = rd.get(m, path, "mask", dict, default=None, required=False)
        if mask is not None:
            chunk = rd.get(mask, path + ".mask", "size", int)
            rd.positive(path, **{"mask.size": chunk})
        return AttentionSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads,
                             head_dim=dim, position=position, scale=scale, v_head_dim=vdim,
                             feature_gate=True, softcap=cap, chunk=chunk, weights="sigmoid",
                             score_bias=True)

    def _right(self, rd: _Reader, path: str, m: Mapping) -> TimeMixingSpec:
        heads, dim = (rd.get(m, path, k, int) for k in ("heads", "dim"))
        rd.positive(path, heads=heads, dim=dim)
        rank = rd.get(m, path, "decay_rank", int, default=0, required=False)
        return TimeMixingSpec(hidden_size=self.width, num_heads=heads, dim=dim, decay_rank=rank,
                              norm_eps=self.norm_eps)

    def _mamba2(self, rd: _Reader, path: str, m: Mapping) -> StateSpaceSpec:
        heads, vdim, state, groups, taps, parts = (
            rd.get(m, path, k, int) for k in ("heads", "vdim", "state", "groups", "conv",
                                              "norm_groups"))
        rd.positive(path, heads=heads, vdim=vdim, state=state, groups=groups, conv=taps,
                    norm_groups=parts)
        if groups > 0 and heads % groups:
            rd.problems.append(f"{path}.heads ({heads}) is no multiple of groups ({groups})")
        if parts > 0 and (heads * vdim) % parts:
            rd.problems.append(f"{path}.norm_groups ({parts}) does not divide heads * vdim")
        return StateSpaceSpec(hidden_size=self.width, num_heads=heads, v_dim=vdim, state=state,
                              groups=groups, conv=taps, norm_groups=parts, norm_eps=self.norm_eps)

    def _mixer(self, rd: _Reader, i: int, layer: Mapping):
        kind = rd.get(layer, f"layers[{i}]", "type", str)
        if kind not in LAYER_TYPES:
            rd.problems.append(f"layers[{i}].type {kind!r} is not known (known: {LAYER_TYPES})")
            return None
        path = f"layers[{i}].mixer"
        m = rd.get(layer, f"layers[{i}]", "mixer", dict)
        if kind == "mamba2":
            return self._mamba2(rd, path, m)
        left = self._left(rd, path + ".left", rd.get(m, path, "left", dict))
        right = self._right(rd, path + ".right", rd.get(m, path, "right", dict))
        return ParallelMixerSpec(hidden_size=self.width, branches=(left, right),
                                 norm_eps=self.norm_eps, merge="mean_of_norms")

    def _ffn(self, rd: _Reader, i: int, layer: Mapping):
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        path = f"layers[{i}].mlp"
        kind = rd.get(mlp, path, "kind", str)
        if kind != "moe":
            rd.problems.append(f"{path}.kind {kind!r} is not known (known: moe)")
            return None
        router = rd.get(mlp, path, "router", dict)
        experts = rd.get(router, path + ".router", "experts", int)
        top = rd.get(router, path + ".router", "top", int)
        expert = rd.get(mlp, path, "expert", dict)
        ff = rd.get(expert, path + ".expert", "ff", int)
        limit = rd.get(expert, path + ".expert", "limit", float)
        rd.positive(path, **{"router.experts": experts, "router.top": top, "expert.ff": ff,
                             "expert.limit": limit})
        if experts > 0 and top > experts:
            rd.problems.append(f"{path}.router.top ({top}) is more than its experts ({experts})")
        shared_ff, shared_limit = 0, 0.0
        shared = rd.get(mlp, path, "shared", dict, default=None, required=False)
        if shared is not None:
            shared_ff = rd.get(shared, path + ".shared", "ff", int)
            shared_limit = rd.get(shared, path + ".shared", "limit", float)
            rd.positive(path, **{"shared.ff": shared_ff, "shared.limit": shared_limit})
        return RoutedExpertsSpec(hidden_size=self.width, num_experts=experts, top=top,
                                 expert_size=ff, shared_size=shared_ff, score="softmax",
                                 renormalize=True, scale_input=False, activation="clamped_swish",
                                 limit=limit, shared_limit=shared_limit,
                                 shared_gate=shared is not None)

    def _blocks(self, rd: Optional[_Reader] = None) -> list:
        rd = rd or _Reader()
        norm = NormSpec(kind="rmsnorm", size=self.width, eps=self.norm_eps)
        blocks = []
        for i, layer in enumerate(self.layers):
            if not isinstance(layer, Mapping):
                rd.problems.append(f"layers[{i}] must be an object")
                continue
            blocks.append(BlockSpec(kind="side_by_side", mixer=self._mixer(rd, i, layer),
                                    ffn=self._ffn(rd, i, layer), norm1=norm, norm2=None,
                                    token_shift=True))
        return blocks

    def run_order(self) -> list:
        """(layer index, whether a pass of the loop begins here) in the order of the runs."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        return ([(i, False) for i in range(start)]
                + [(i, i == start) for i in range(start, stop)] * times
                + [(i, False) for i in range(stop, n)])

    def layout(self) -> ModelLayout:
        norm = NormSpec(kind="rmsnorm", size=self.width, eps=self.norm_eps)
        order = [RunEntry(block=i, cache=run, loop_input=first)
                 for run, (i, first) in enumerate(self.run_order())]
        layout = ModelLayout(vocab_size=self.vocab, hidden_size=self.width,
                             blocks=self._blocks(), order=order, final_norm=norm,
                             tie_word_embeddings=False, max_positions=None,
                             loop_input=LoopInputSpec(hidden_size=self.width)
                             if self.loop is not None else None)
        layout.validate()
        return layout

    def stop_token_ids(self) -> tuple:
        return tuple(self.stop_tokens)

    def max_positions(self):
        return None
