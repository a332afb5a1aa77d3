"""Checkpoint tensor names of the Sokalorn decoder and where each goes.

Layer i's tensors start with ``l<i>.``: ``norm1``, ``shift``, the mixer under ``mix.`` (the two
branches of a parallel mixer under ``mix.left.`` / ``mix.right.``, with their output norms
``left.out`` / ``right.out``), the experts under ``mlp.``; the model's ends are ``embed``,
``final.norm``, ``head``, and a looped stretch has ``loop.in``.  Stacked into one engine
parameter: the attention's ``[q; k; v; g]``, the time mixing's ``[r; k; v; g; w1]`` and its five
``mu``, the router's rows with the shared expert's gate, every expert's ``[gate; up]``.
"""
from __future__ import annotations

from ..config.layout import ModelLayout
from .names import CheckpointMap, TensorSource
from .tifosun import _stack


def _attention_sources(src: list, ck: str, me: str, a, width: int) -> None:
    _stack(src, f"{me}.qkv.weight", [(f"{ck}.q", a.num_heads * a.head_dim),
                                     (f"{ck}.k", a.num_kv_heads * a.head_dim),
                                     (f"{ck}.v", a.num_kv_heads * a.value_dim),
                                     (f"{ck}.g", a.num_heads * a.value_dim)])
    src.append(TensorSource(f"{ck}.pb", f"{me}.score_bias", 0, a.num_heads))
    src.append(TensorSource(f"{ck}.o", f"{me}.o.weight", 0, width))


def _time_mixing_sources(src: list, ck: str, me: str, m, width: int) -> None:
    rows = m.num_heads * m.dim
    _stack(src, f"{me}.in.weight", [(f"{ck}.{n}", rows) for n in "rkvg"]
           + [(f"{ck}.w1", m.decay_rank)])
    # the five mixing vectors are kept end to end
    _stack(src, f"{me}.mu", [(f"{ck}.mu.{n}", width) for n in "rkvgw"])
    src.append(TensorSource(f"{ck}.w2", f"{me}.w2.weight", 0, rows))
    src.append(TensorSource(f"{ck}.w0", f"{me}.w0", 0, rows))
    src.append(TensorSource(f"{ck}.u", f"{me}.u", 0, m.num_heads))
    src.append(TensorSource(f"{ck}.norm", f"{me}.norm.weight", 0, rows))
    src.append(TensorSource(f"{ck}.o", f"{me}.o.weight", 0, width))


def _state_space_sources(src: list, ck: str, me: str, m, width: int) -> None:
    for name, param, rows in (("in", "in.weight", m.inner + m.channels + m.num_heads),
                              ("conv", "conv.weight", m.channels), ("conv.b", "conv.bias", m.channels),
                              ("dt_bias", "dt_bias", m.num_heads), ("A_log", "A_log", m.num_heads),
                              ("D", "D", m.num_heads), ("norm", "norm.weight", m.inner),
                              ("o", "o.weight", width)):
        src.append(TensorSource(f"{ck}.{name}", f"{me}.{param}", 0, rows))


def _expert_sources(src: list, ck: str, me: str, f, width: int) -> None:
    router = [(f"{ck}.router", f.num_experts)]
    if f.shared_gate:
        router.append((f"{ck}.shared.sg", 1))
    _stack(src, f"{me}.router.weight", router)
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


def sokalorn_checkpoint_map(config, layout: ModelLayout) -> CheckpointMap:
    src: list = []
    width = layout.hidden_size
    src.append(TensorSource("embed", "embed.weight", 0, layout.vocab_size))
    if layout.loop_input is not None:
        src.append(TensorSource("loop.in", "loop_input.weight", 0, width))
    for i, block in enumerate(layout.blocks):
        ck, me = f"l{i}", f"blocks.{i}"
        src.append(TensorSource(f"{ck}.norm1", f"{me}.norm1.weight", 0, width))
        src.append(TensorSource(f"{ck}.shift", f"{me}.shift", 0, width))
        m = block.mixer
        if m.kind == "state_space":
            _state_space_sources(src, f"{ck}.mix", f"{me}.mixer", m, width)
        elif m.kind == "parallel" and len(m.branches) == 2:
            _attention_sources(src, f"{ck}.mix.left", f"{me}.mixer.branch0", m.branches[0], width)
            _time_mixing_sources(src, f"{ck}.mix.right", f"{me}.mixer.branch1", m.branches[1], width)
            for b, side in enumerate(("left", "right")):
                src.append(TensorSource(f"{ck}.mix.{side}.out", f"{me}.mixer.out{b}.weight", 0, width))
        else:
            raise ValueError(f"no checkpoint names for a mixer of kind {m.kind!r}")
        if block.ffn is not None:
            _expert_sources(src, f"{ck}.mlp", f"{me}.ffn", block.ffn, width)
    src.append(TensorSource("final.norm", "final_norm.weight", 0, layout.final_norm.size))
    src.append(TensorSource("head", "head.weight", 0, layout.vocab_size))
    return CheckpointMap(sources=src)
