"""Configuration, layout, checkpoint map and plain implementation of the Sokalorn decoder (no
GPU needed)."""
import copy

import numpy as np
import pytest

import plain_sokalorn as P
import sokalorn_util as U
from mstar_b200.cache.storage import plan_groups
from mstar_b200.config.base import ConfigError
from mstar_b200.config.registry import config_from_dict, get_architecture, known_architectures
from mstar_b200.engine.model import cache_needs, model_param_specs
from mstar_b200.parts.rope import rope_inverse_frequencies


def test_architecture_is_registered_and_round_trips():
    assert "Sokalorn" in known_architectures()
    cfg = config_from_dict(U.MIXED)
    assert cfg.architecture == "Sokalorn" and cfg.to_dict()["layers"] == U.MIXED["layers"]
    assert cfg.to_dict()["loop"] == U.MIXED["loop"]
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


def test_layout_reads_every_size_and_constant_per_layer():
    lay = U.shaped(U.MIXED).layout()
    # five sets of weights; the stretch 1..3 runs twice; a cache for every run; the residual
    # passes the loop's input before the first run of each pass
    assert len(lay.blocks) == 5
    assert [(e.block, e.cache, e.loop_input) for e in lay.order] == [
        (0, 0, False), (1, 1, True), (2, 2, False), (3, 3, False), (1, 4, True), (2, 5, False),
        (3, 6, False), (4, 7, False)]
    assert lay.loop_input.kind == "concat_linear" and lay.loop_input.hidden_size == 64
    assert all(b.kind == "side_by_side" and b.token_shift and b.norm2 is None for b in lay.blocks)
    s0, s2 = lay.blocks[0].mixer, lay.blocks[2].mixer
    assert (s0.kind, s0.num_heads, s0.v_dim, s0.state, s0.groups, s0.conv, s0.norm_groups) == (
        "state_space", 4, 20, 24, 2, 4, 2)
    assert s0.inner == 80 and s0.channels == 80 + 2 * 2 * 24
    assert (s2.num_heads, s2.groups, s2.conv, s2.norm_groups) == (6, 3, 2, 1)
    p1 = lay.blocks[1].mixer
    assert p1.merge == "mean_of_norms"
    l1, r1 = p1.branches
    assert (l1.num_heads, l1.num_kv_heads, l1.head_dim, l1.value_dim, l1.chunk) == (4, 2, 24, 40, 11)
    assert (l1.weights, l1.score_bias, l1.feature_gate, l1.softcap) == ("sigmoid", True, True, 6.0)
    assert l1.window is None and l1.sink is None and not l1.plain
    assert l1.position.rotary_dim == 8 and not l1.position.interleaved
    assert np.allclose(rope_inverse_frequencies(l1.position),
                       [300.0 ** (-2 * i / 8) / 2.5 for i in range(4)])
    assert (r1.kind, r1.num_heads, r1.dim, r1.decay_rank) == ("time_mixing", 3, 20, U.RANK)
    l4 = lay.blocks[4].mixer.branches[0]
    assert l4.softcap is None and l4.chunk == 7
    f0, f2, f4 = (lay.blocks[i].ffn for i in (0, 2, 4))
    assert (f0.num_experts, f0.top, f0.expert_size, f0.shared_size) == (6, 2, 40, 56)
    assert (f0.limit, f0.shared_limit, f0.activation, f0.shared_gate) == (1.2, 0.8, "clamped_swish", True)
    assert f0.score == "softmax" and f0.renormalize and not f0.scale_input
    assert (f2.shared_size, f2.shared_gate, f2.top) == (0, False, 3)
    assert (f4.num_experts, f4.top) == (9, 4) and lay.blocks[3].ffn is None
    needs = cache_needs(lay)
    # the token shift's row follows the mixer's own state, both padded to whole 16-byte pieces
    assert needs[0].kv is None and needs[0].state.shape == (3 * 176 + 4 * 24 * 20 + 64,)
    assert needs[1].kv.v_head_dim == 40 and needs[1].kv.window == 11
    assert needs[1].state.shape == (64 + 3 * 20 * 20 + 64,)
    assert needs[4] == needs[1] and needs[6] == needs[3]          # the passes of one block
    windows, group_of = plan_groups(needs)
    assert windows == [11, 16, 7] and group_of == [None, 0, None, 1, 0, None, 1, 2]


def test_loops_at_either_end_and_none():
    layers = U.MIXED["layers"]
    plain = U.shaped(U.config(layers)).layout()
    assert [e.block for e in plain.order] == [0, 1, 2, 3, 4] and plain.loop_input is None
    assert not any("loop" in k for k in model_param_specs(plain))
    for loop in ((0, 2, 3), (3, 5, 2), (0, 5, 1), (2, 3, 4)):
        raw = U.config(layers, loop=loop)
        order = [(e.block, e.loop_input) for e in U.shaped(raw).layout().order]
        assert order == P.plain_run_order(raw)
        assert sum(first for _, first in order) == loop[2]         # the first pass too


def test_checkpoint_names_cover_the_parameters():
    weights = U.random_weights(U.MIXED, 2)
    cfg = U.shaped(U.MIXED, weights)
    lay = cfg.layout()
    specs = model_param_specs(lay)
    cmap = get_architecture("Sokalorn").checkpoint_map(cfg, lay)
    assert {s.name for s in cmap.sources} == set(weights)
    filled = {}
    for s in cmap.sources:
        assert tuple(weights[s.name].shape) == (s.rows,) + tuple(specs[s.param].shape[1:]), s.name
        filled[s.param] = filled.get(s.param, 0) + s.rows
    assert {k: v.shape[0] for k, v in specs.items()} == filled
    assert specs["blocks.1.mixer.branch0.qkv.weight"].shape == (4 * 24 + 2 * 24 + 2 * 40 + 4 * 40, 64)
    assert specs["blocks.1.mixer.branch1.in.weight"].shape == (4 * 60 + U.RANK, 64)
    assert specs["blocks.0.ffn.router.weight"].shape == (7, 64)           # the shared gate's row
    assert specs["blocks.2.ffn.router.weight"].shape == (3, 64)
    assert specs["loop_input.weight"].shape == (64, 128) and "blocks.3.ffn.router.weight" not in specs


def test_rank_comes_from_the_tensors_or_the_configuration():
    raw = copy.deepcopy(U.MIXED)
    assert config_from_dict(raw).layout().blocks[1].mixer.branches[1].decay_rank == 0   # not known
    got = U.shaped(raw, U.random_weights(raw, 3, rank=9)).layout()
    assert got.blocks[3].mixer.branches[1].decay_rank == 9
    raw["layers"][1]["mixer"]["right"]["decay_rank"] = 11
    assert config_from_dict(raw).layout().blocks[1].mixer.branches[1].decay_rank == 11


def test_unusable_configurations_name_everything():
    raw = copy.deepcopy(U.MIXED)
    del raw["layers"][1]["mixer"]["left"]["scale"]
    raw["layers"][1]["mixer"]["left"]["heads"] = 5
    raw["layers"][0]["mixer"]["groups"] = 3
    raw["layers"][0]["mlp"]["router"]["top"] = 7
    raw["layers"][2]["mixer"]["norm_groups"] = 7
    raw["layers"][3]["type"] = "mamba3"
    raw["layers"][4]["mlp"] = {"kind": "dense"}
    raw["loop"] = {"start": 2, "stop": 2, "times": 2}
    del raw["vocab"]
    with pytest.raises(ConfigError) as err:
        config_from_dict(raw)
    text = str(err.value)
    for part in ("layers[1].mixer.left.scale", "layers[1].mixer.left.heads", "layers[0].mixer.heads",
                 "router.top", "layers[2].mixer.norm_groups", "mamba3", "layers[4].mlp.kind",
                 "config.loop", "vocab"):
        assert part in text, part


def test_pieces_of_a_scan():
    from mstar_b200.ops import linear_scan_pieces

    assert linear_scan_pieces(8, 16, 1, 148) == (0, 1)            # decoding
    assert linear_scan_pieces(64, 32, 4096, 148) == (0, 1)        # the heads alone fill the GPU
    piece, pieces = linear_scan_pieces(1, 16, 2048, 148)
    assert piece % 16 == 0 and piece >= 32 and (pieces - 1) * piece < 2048 <= pieces * piece


def test_plain_mechanisms_on_hand_computed_cases():
    # halves, angle p * base^(-2i/dims) / factor; features beyond dims pass
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]])
    y = P.plain_rotate_half(x, [3], 4, 100.0, 2.0)
    a0, a1 = 3.0 / 2.0, 3.0 * 100.0 ** -0.5 / 2.0
    assert np.allclose(y[0, 0], [np.cos(a0), -2 * np.sin(a1), np.sin(a0), 2 * np.cos(a1), 5])
    # chunks of two positions, weights that do not sum to one
    q = np.zeros((4, 1, 1))
    v = np.array([[[1.0]], [[10.0]], [[100.0]], [[1000.0]]])
    o = P.plain_sigmoid_attention(q, q, v, 0, 1.0, None, [0.0], 2)
    assert np.allclose(o[:, 0, 0], [0.5, 5.5, 50.0, 550.0])
    o = P.plain_sigmoid_attention(q, q, v, 0, 1.0, 4.0, [np.log(3.0)], None)
    assert np.allclose(o[:, 0, 0], 0.75 * np.array([1.0, 11.0, 111.0, 1111.0]))
    # time mixing: the bonus holds for the current token only, the decay for later reads
    r = k = np.ones((3, 1))
    S = np.zeros((1, 1))
    o = P.plain_rwkv_scan(r, k, np.array([[1.0], [2.0], [4.0]]), np.full((3, 1), 0.5), [3.0], S)
    assert np.allclose(o[:, 0], [3.0, 1.0 + 6.0, 2.5 + 12.0]) and np.allclose(S, [[0.5 * 2.5 + 4.0]])
    # state space: the read sees the token's own write
    S = np.zeros((1, 1))
    one = np.ones((2, 1))
    o = P.plain_ssd_scan(np.array([[1.0], [2.0]]), one, one, np.array([0.5, 1.0]), np.log(2.0), 10.0, S)
    s0 = 0.5
    s1 = 0.5 * s0 + 2.0
    assert np.allclose(o[:, 0], [s0 + 10.0, s1 + 20.0])
    # the clamps: gate from above only, up from both sides
    g = P.plain_clamped_expert(np.array([[1.0]]), np.array([[5.0], [-5.0]]), np.array([[-9.0], [0.5]]),
                               np.eye(2), 2.0)
    sig = lambda z: 1 / (1 + np.exp(-z))
    assert np.allclose(g[0], [2 * sig(1.702 * 2) * (-2 + 1), -5 * sig(1.702 * -5) * 1.5])
    chosen, weight = P.plain_route(np.array([[0.0, 2.0, 1.0]]), 2)
    assert chosen.tolist() == [[1, 2]] and np.allclose(weight[0], [np.e / (np.e + 1), 1 / (np.e + 1)])
    # the row before the first is zero, then the last row of the call before
    st = {}
    assert np.allclose(P.plain_previous(np.array([[1.0], [2.0]]), st, "p"), [[0.0], [1.0]])
    assert np.allclose(P.plain_previous(np.array([[5.0]]), st, "p"), [[2.0]])
    # the convolution's last column meets the token itself, zeros before the start
    st = {}
    c = P.plain_short_conv(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0]]), [0.5], st, "c")
    assert np.allclose(c[:, 0], [1.5, 12.5]) and np.allclose(st["c"], [[2.0]])


def test_plain_model_in_portions_equals_whole():
    w = U.as_numpy(U.random_weights(U.MIXED, 4))
    toks = U.tokens(U.MIXED, 29, 1)
    whole = P.plain_forward(toks, w, U.MIXED)
    states = [{} for _ in range(U.runs(U.MIXED))]
    parts = [P.plain_forward(toks[a:b], w, U.MIXED, states)
             for a, b in ((0, 7), (7, 9), (9, 10), (10, 29))]
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9
    # every mechanism matters: without it the logits differ
    other = P.plain_forward(toks, w, dict(U.MIXED, loop={"start": 1, "stop": 4, "times": 1}))
    assert np.abs(other - whole).max() > 1e-2
    for name, change in (("l0.shift", 0.0), ("l1.mix.left.pb", 3.0), ("l1.mix.right.u", 0.0),
                         ("l1.mix.right.mu.w", 0.0), ("l2.mix.D", 0.0), ("l0.mix.conv.b", 0.0),
                         ("l0.mlp.shared.sg", 0.0)):
        w2 = dict(w)
        w2[name] = np.full_like(w[name], change)
        assert np.abs(P.plain_forward(toks, w2, U.MIXED) - whole).max() > 1e-3, name
