"""Checkpoint tensor names of the Famarax decoder and where each goes.

Layer i's tensors start with ``l<i>.``: ``norm1`` / ``norm2`` (a weight, with ``.b`` and the scalar
``.alpha`` beside it, like every norm of the model), the hyper-connection tables ``hc1.{in,out,
mix}`` / ``hc2.{in,out,mix}``, the mixer under ``mix.``, the experts under ``mlp.``; the model's ends
are ``embed``, ``embed.norm``, ``final.norm``, ``head``.  Stacked into one engine parameter: an
attention's ``[q; k; v]``, the delta rule's ``[q; k; v; b; a; g]`` and its three convolutions, every
expert's ``[gate; up]``.
"""
from __future__ import annotations

from ..config.layout import ModelLayout
from .names import CheckpointMap, TensorSource
from .tifosun import _stack


def _norm_sources(src: list, ck: str, me: str, size: int) -> None:
    src.append(TensorSource(ck, f"{me}.weight", 0, size))
    src.append(TensorSource(f"{ck}.b", f"{me}.bias", 0, size))
    src.append(TensorSource(f"{ck}.alpha", f"{me}.alpha", 0, 1, scalar=True))


def _attention_sources(src: list, ck: str, me: str, a, width: int) -> None:
    _stack(src, f"{me}.qkv.weight", [(f"{ck}.q", a.num_heads * a.head_dim),
                                     (f"{ck}.k", a.num_kv_heads * a.head_dim),
                                     (f"{ck}.v", a.num_kv_heads * a.value_dim)])
    if a.value_mix == "blend":
        src.append(TensorSource(f"{ck}.vmix", f"{me}.value_mix", 0, 1, scalar=True))
    src.append(TensorSource(f"{ck}.o", f"{me}.o.weight", 0, width))


def _delta_sources(src: list, ck: str, me: str, d, width: int) -> None:
    qk, vv = d.num_kv_heads * d.qk_dim, d.num_heads * d.v_dim
    _stack(src, f"{me}.in.weight", [(f"{ck}.q", qk), (f"{ck}.k", qk), (f"{ck}.v", vv),
                                    (f"{ck}.b", d.num_heads), (f"{ck}.a", d.num_heads),
                                    (f"{ck}.g", vv)])
    _stack(src, f"{me}.conv.weight", [(f"{ck}.q.conv", qk), (f"{ck}.k.conv", qk),
                                      (f"{ck}.v.conv", vv)])
    for name, param, rows in (("dt_bias", "dt_bias", d.num_heads), ("A_log", "A_log", d.num_heads),
                              ("norm", "norm.weight", d.v_dim), ("o", "o.weight", width)):
        src.append(TensorSource(f"{ck}.{name}", f"{me}.{param}", 0, rows))


def _expert_sources(src: list, ck: str, me: str, f, width: int) -> None:
    src.append(TensorSource(f"{ck}.router", f"{me}.router.weight", 0, f.num_experts))
    src.append(TensorSource(f"{ck}.correction", f"{me}.router.correction", 0, f.num_experts))
    gate_up, down = [], []
    for e in range(f.num_experts):
        gate_up += [(f"{ck}.e{e}.gate", f.expert_size), (f"{ck}.e{e}.up", f.expert_size)]
        down.append((f"{ck}.e{e}.down", width))
    _stack(src, f"{me}.experts.gate_up.weight", gate_up)
    _stack(src, f"{me}.experts.down.weight", down)
    if f.shared_size:
        _stack(src, f"{me}.shared.gate_up.weight", [(f"{ck}.shared.gate", f.shared_size),
                                                    (f"{ck}.shared.up", f.shared_size)])
        src.append(TensorSource(f"{ck}.shared.down", f"{me}.shared.down.weight", 0, width))


def famarax_checkpoint_map(config, layout: ModelLayout) -> CheckpointMap:
    src: list = []
    unused: set = set()     # present or not, never read
    width = layout.hidden_size
    src.append(TensorSource("embed", "embed.weight", 0, layout.vocab_size))
    _norm_sources(src, "embed.norm", "embed.norm", width)
    for i, block in enumerate(layout.blocks):
        ck, me = f"l{i}", f"blocks.{i}"
        for q in (1, 2):
            names = [f"{ck}.hc{q}.{t}" for t in ("in", "out", "mix")]
            if q == 2 and block.ffn is None:
                unused.update(names + [f"{ck}.norm2{t}" for t in ("", ".b", ".alpha")])
                continue
            _norm_sources(src, f"{ck}.norm{q}", f"{me}.norm{q}", width)
            for name, t in zip(names, ("in", "out", "mix")):
                src.append(TensorSource(name, f"{me}.hc{q}.{t}", 0, block.streams))
        m = block.mixer
        if m.kind == "attention":
            _attention_sources(src, f"{ck}.mix", f"{me}.mixer", m, width)
            if m.value_mix != "blend":          # the layer whose values the others blend in
                unused.add(f"{ck}.mix.vmix")
        elif m.kind == "gated_delta":
            _delta_sources(src, f"{ck}.mix", f"{me}.mixer", m, width)
        else:
            raise ValueError(f"no checkpoint names for a mixer of kind {m.kind!r}")
        if block.ffn is not None:
            _expert_sources(src, f"{ck}.mlp", f"{me}.ffn", block.ffn, width)
    _norm_sources(src, "final.norm", "final_norm", width)
    src.append(TensorSource("head", "head.weight", 0, layout.vocab_size))
    return CheckpointMap(sources=src, ignore=unused.__contains__)
