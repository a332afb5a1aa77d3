"""Typed configuration of the Famarax decoder (``"architecture": "Famarax"``).

config.json gives ``width``, ``vocab``, ``norm.eps``, ``streams`` (hyper-connections: that many
copies of the residual), optionally ``logit_scale`` and ``logit_softcap``, and the layers one by
one: ``layers[i] = {"type": ..., "mixer": {...}, "mlp": {"kind": "moe", ...} | null}``.

Every norm of the model is a dynamic tanh (``tanh(alpha x) w + b``), the one on the embedding
rows included.  Layer types:

* ``attention``: grouped-query attention in a sliding window of ``mask.size`` keys; rotate-half
  pairs over ``rot.dims`` features with base ``rot.base``; q and k heads divided by their root mean
  square (no weight); scores scaled by ``scale`` and soft-capped at ``softcap``.  In layers with
  ``v_mix``, all but the first of them, the values are blended with that first one's values;
* ``delta``: the gated delta rule (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps) with
  one decay a head and a SiLU gate on the normed read-out.

The feed-forward is ``router.top`` of ``router.experts`` gated experts (``expert.ff``) beside a
shared one (``shared.ff``): softmax scores, a correction for the choice, ``router.groups.{count,
keep}``, weights renormalised and multiplied by ``router.scale``.

No size has a default; every size may differ from layer to layer.  A mechanism whose key is
absent or null (``mask``, ``softcap``, ``rot``, ``v_mix``, ``mlp``, ``mlp.shared``,
``router.groups``, ``router.scale``, the logits' scale and soft cap) is left out.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from .base import ConfigError, ModelConfig
from .layout import (AttentionSpec, BlockSpec, EmbeddingSpec, GatedDeltaSpec, HeadSpec, ModelLayout,
                     NormSpec, PositionSpec, RoutedExpertsSpec, RunEntry)
from .tifosun import _Reader

LAYER_TYPES = ("attention", "delta")
MAX_STREAMS = 8
RENORM_EPS = 1e-20      # added to the sum of the chosen scores


@dataclass
class FamaraxConfig(ModelConfig):
    width: int
    vocab: int
    norm_eps: float
    streams: int
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    layers: list = field(default_factory=list)        # the raw layer objects of config.json
    stop_tokens: tuple = ()

    architecture = "Famarax"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FamaraxConfig":
        rd = _Reader()
        width = rd.get(raw, "config", "width", int)
        vocab = rd.get(raw, "config", "vocab", int)
        eps = rd.get(rd.get(raw, "config", "norm", dict), "config.norm", "eps", float)
        streams = rd.get(raw, "config", "streams", int)
        if not 1 <= streams <= MAX_STREAMS:
            rd.problems.append(f"config.streams must lie in 1..{MAX_STREAMS}, got {streams}")
        scale = rd.get(raw, "config", "logit_scale", float, default=1.0, required=False)
        cap = rd.get(raw, "config", "logit_softcap", float, default=None, required=False)
        if cap is not None:
            rd.positive("config", logit_softcap=cap)
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            rd.problems.append("config.layers must be a non-empty list")
            layers = []
        stops = raw.get("eos_token_id")
        if stops is None:
            stops = ()
        elif not isinstance(stops, (list, tuple)):
            stops = (stops,)
        cfg = cls(width=width, vocab=vocab, norm_eps=eps, streams=streams, logit_scale=scale,
                  logit_softcap=cap, layers=copy.deepcopy(list(layers)),
                  stop_tokens=tuple(int(t) for t in stops))
        rd.positive("config", width=width, vocab=vocab, **{"norm.eps": eps})
        if width > 0:
            cfg._blocks(rd)
        if rd.problems:
            raise ConfigError("unusable Famarax configuration: " + "; ".join(rd.problems))
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
               "norm": {"eps": self.norm_eps}, "streams": self.streams,
               "logit_scale": self.logit_scale, "layers": copy.deepcopy(self.layers)}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.stop_tokens:
            out["eos_token_id"] = list(self.stop_tokens)
        return out

    # -- layers -------------------------------------------------------------
    @staticmethod
    def _heads(rd: _Reader, path: str, m: Mapping) -> tuple:
        heads, kv_heads, dim, vdim = (rd.get(m, path, k, int)
                                      for k in ("heads", "kv_heads", "dim", "vdim"))
        rd.positive(path, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        if kv_heads > 0 and heads % kv_heads:
            rd.problems.append(f"{path}.heads ({heads}) is no multiple of kv_heads ({kv_heads})")
        return heads, kv_heads, dim, vdim

    def _attention(self, rd: _Reader, path: str, m: Mapping, first_values) -> AttentionSpec:
        """``first_values``: (path, size) of the first layer with ``v_mix``, None before it."""
        heads, kv_heads, dim, vdim = self._heads(rd, path, m)
        scale = rd.get(m, path, "scale", float)
        position = PositionSpec(kind="none", head_dim=dim)
        rot = rd.get(m, path, "rot", dict, default=None, required=False)
        if rot is not None:
            base = rd.get(rot, path + ".rot", "base", float)
            dims = rd.get(rot, path + ".rot", "dims", int)
            rd.positive(path, **{"rot.base": base})
            if dims % 2 or not 0 <= dims <= dim:
                rd.problems.append(f"{path}.rot.dims must be even and at most dim, got {dims}")
            elif dims:
                position = PositionSpec(kind="rope", head_dim=dim, rotary_dim=dims, theta=base)
        cap = rd.get(m, path, "softcap", float, default=None, required=False)
        if cap is not None:
            rd.positive(path, softcap=cap)
        window = None
        mask = rd.get(m, path, "mask", dict, default=None, required=False)
        if mask is not None:
            window = rd.get(mask, path + ".mask", "size", int)
            rd.positive(path, **{"mask.size": window})
        mix = None
        if m.get("v_mix"):
            mix = "first" if first_values is None else "blend"
            if mix == "blend" and first_values[1] != kv_heads * vdim:
                rd.problems.append(f"{path} blends {kv_heads} x {vdim} values with the "
                                   f"{first_values[1]} of {first_values[0]}")
        return AttentionSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads,
                             head_dim=dim, position=position, window=window, scale=scale,
                             v_head_dim=vdim, qk_norm_eps=self.norm_eps, qk_norm_weight=False,
                             softcap=cap, value_mix=mix)

    def _delta(self, rd: _Reader, path: str, m: Mapping) -> GatedDeltaSpec:
        heads, kv_heads, dim, vdim = self._heads(rd, path, m)
        taps = rd.get(m, path, "conv", int)
        rd.positive(path, conv=taps)
        return GatedDeltaSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads,
                              qk_dim=dim, v_dim=vdim, conv=taps, norm_eps=self.norm_eps,
                              head_decay=True, full_gate=True, gate_activation="silu")

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
        scale = rd.get(router, path + ".router", "scale", float, default=1.0, required=False)
        ff = rd.get(rd.get(mlp, path, "expert", dict), path + ".expert", "ff", int)
        rd.positive(path, **{"router.experts": experts, "router.top": top, "expert.ff": ff})
        open_to = experts
        groups = rd.get(router, path + ".router", "groups", dict, default=None, required=False)
        if groups is not None:
            count = rd.get(groups, path + ".router.groups", "count", int)
            keep = rd.get(groups, path + ".router.groups", "keep", int)
            rd.positive(path, **{"router.groups.count": count, "router.groups.keep": keep})
            groups = (count, keep)
            if count > 0 and experts % count:
                rd.problems.append(f"{path}.router.experts ({experts}) do not form {count} equal "
                                   "groups")
            elif count > 0:
                if keep > count:
                    rd.problems.append(f"{path}.router.groups.keep ({keep}) is more than its groups "
                                       f"({count})")
                open_to = experts // count * min(keep, count)
        if top > open_to:
            rd.problems.append(f"{path}.router.top ({top}) is more than the {open_to} experts that "
                               "can be chosen")
        shared_ff = 0
        shared = rd.get(mlp, path, "shared", dict, default=None, required=False)
        if shared is not None:
            shared_ff = rd.get(shared, path + ".shared", "ff", int)
            rd.positive(path, **{"shared.ff": shared_ff})
        return RoutedExpertsSpec(hidden_size=self.width, num_experts=experts, top=top,
                                 expert_size=ff, shared_size=shared_ff, score="softmax",
                                 renormalize=True, renorm_eps=RENORM_EPS, weight_scale=scale,
                                 scale_input=False, choice_bias=True, groups=groups)

    def _norm(self) -> NormSpec:
        return NormSpec(kind="dynamic_tanh", size=self.width)

    def _blocks(self, rd: Optional[_Reader] = None) -> list:
        rd = rd or _Reader()
        norm = self._norm()
        blocks = []
        first_values = None
        for i, layer in enumerate(self.layers):
            if not isinstance(layer, Mapping):
                rd.problems.append(f"layers[{i}] must be an object")
                continue
            path = f"layers[{i}].mixer"
            kind = rd.get(layer, f"layers[{i}]", "type", str)
            m = rd.get(layer, f"layers[{i}]", "mixer", dict)
            mixer = None
            if kind == "attention":
                mixer = self._attention(rd, path, m, first_values)
                if mixer.value_mix == "first":
                    first_values = (path, mixer.num_kv_heads * mixer.value_dim)
            elif kind == "delta":
                mixer = self._delta(rd, path, m)
            else:
                rd.problems.append(f"layers[{i}].type {kind!r} is not known (known: {LAYER_TYPES})")
            ffn = self._ffn(rd, i, layer)
            blocks.append(BlockSpec(kind="hyper", mixer=mixer, ffn=ffn, norm1=norm,
                                    norm2=None if ffn is None else norm, streams=self.streams))
        return blocks

    def layout(self) -> ModelLayout:
        blocks = self._blocks()
        layout = ModelLayout(
            vocab_size=self.vocab, hidden_size=self.width, blocks=blocks,
            order=[RunEntry(block=i, cache=i) for i in range(len(blocks))],
            final_norm=self._norm(), tie_word_embeddings=False, max_positions=None,
            embedding=EmbeddingSpec(vocab_size=self.vocab, hidden_size=self.width,
                                    norm=self._norm()),
            head=HeadSpec(vocab_size=self.vocab, hidden_size=self.width,
                          logit_scale=self.logit_scale, softcap=self.logit_softcap))
        layout.validate()
        return layout

    def stop_token_ids(self) -> tuple:
        return tuple(self.stop_tokens)

    def max_positions(self):
        return None
