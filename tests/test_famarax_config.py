"""Configuration, layout, checkpoint map and plain implementation of the Famarax decoder (no GPU
needed)."""
import copy

import numpy as np
import pytest
import torch

import famarax_util as U
import plain_famarax as P
from mstar_b200.cache.storage import plan_groups
from mstar_b200.config.base import ConfigError
from mstar_b200.config.registry import config_from_dict, get_architecture, known_architectures
from mstar_b200.engine.model import cache_needs, model_param_specs
from mstar_b200.weights.loader import WeightsError, load_parameters
from mstar_b200.weights.random_init import random_checkpoint


def test_architecture_is_registered_and_round_trips():
    assert "Famarax" in known_architectures()
    cfg = config_from_dict(U.MIXED)
    assert cfg.architecture == "Famarax" and cfg.to_dict()["layers"] == U.MIXED["layers"]
    assert cfg.to_dict()["streams"] == 3 and cfg.to_dict()["logit_softcap"] == 9.0
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


def test_layout_reads_every_size_and_constant_per_layer():
    lay = config_from_dict(U.MIXED).layout()
    assert [(e.block, e.cache) for e in lay.order] == [(i, i) for i in range(6)]
    assert all(b.kind == "hyper" and b.streams == 3 and b.residual_mult == 1.0 for b in lay.blocks)
    assert all(b.norm1.kind == "dynamic_tanh" and b.norm1.size == 64 for b in lay.blocks)
    assert lay.final_norm.kind == "dynamic_tanh" and lay.embedding.norm.kind == "dynamic_tanh"
    assert (lay.head.logit_scale, lay.head.softcap) == (0.7, 9.0)
    a0, a2, a3, a5 = (lay.blocks[i].mixer for i in (0, 2, 3, 5))
    assert (a0.num_heads, a0.num_kv_heads, a0.head_dim, a0.value_dim, a0.window) == (4, 2, 24, 40, 11)
    assert a0.qk_norm_eps == 1e-5 and not a0.qk_norm_weight and not a0.plain
    assert (a0.softcap, a0.position.rotary_dim, a0.position.theta) == (6.0, 8, 300.0)
    assert not a0.position.interleaved
    assert (a2.scale, a2.softcap, a2.window, a2.position.rotary_dim) == (0.5, 2.5, None, 16)
    assert (a3.softcap, a3.position.kind, a3.window) == (None, "none", 30)
    # the first layer with blended values only hands its own on
    assert [m.value_mix for m in (a0, a2, a3, a5)] == ["first", None, "blend", "blend"]
    d1, d4 = lay.blocks[1].mixer, lay.blocks[4].mixer
    assert (d1.kind, d1.num_heads, d1.num_kv_heads, d1.qk_dim, d1.v_dim, d1.conv) == (
        "gated_delta", 4, 2, 24, 20, 3)
    assert d1.head_decay and d1.full_gate and d1.gate_activation == "silu"
    assert (d4.num_heads, d4.num_kv_heads, d4.qk_dim, d4.v_dim, d4.conv) == (3, 3, 10, 36, 4)
    f = [b.ffn for b in lay.blocks]
    assert f[3] is None and lay.blocks[3].norm2 is None
    assert [x and (x.num_experts, x.top, x.expert_size, x.shared_size, x.groups, x.weight_scale)
            for x in f] == [(8, 3, 40, 56, (4, 2), 1.6), (6, 2, 24, 0, (2, 1), 0.8),
                            (9, 4, 16, 24, (3, 2), 1.0), None, (5, 5, 24, 8, None, 1.0),
                            (8, 2, 32, 40, (8, 3), 2.2)]
    assert all(x.choice_bias and x.renormalize and x.score == "softmax" and not x.scale_input
               and x.renorm_eps == 1e-20 for x in f if x)
    needs = cache_needs(lay)
    assert needs[0].kv.window == 11 and needs[0].kv.v_head_dim == 40 and needs[0].state is None
    assert needs[1].kv is None and needs[1].state.shape == (2 * (2 * 48 + 80) + 4 * 24 * 20,)
    windows, group_of = plan_groups(needs)
    assert windows == [11, None, 30, 7] and group_of == [0, None, 1, 2, None, 3]


def test_keys_that_may_be_absent():
    layers = [U.layer("attention", U.attention(2, 1, 16, 16, softcap=None, window=None, rot_dims=0,
                                               v_mix=None), U.moe(4, 2, 8, 0, None, None)),
              U.layer("delta", U.delta(2, 1, 8, 8, 1), None)]
    lay = config_from_dict(U.config(layers, logit_scale=None, logit_softcap=None)).layout()
    assert lay.blocks[0].mixer.value_mix is None and lay.blocks[0].ffn.groups is None
    assert (lay.head.logit_scale, lay.head.softcap, lay.blocks[0].ffn.weight_scale) == (1.0, None, 1.0)
    nulls = copy.deepcopy(layers)
    nulls[0]["mixer"].update(mask=None, softcap=None, rot=None)
    nulls[0]["mlp"].update(shared=None)
    nulls[0]["mlp"]["router"].update(groups=None)
    assert config_from_dict(U.config(nulls, logit_scale=None, logit_softcap=None)).layout() == lay


def test_checkpoint_names_cover_the_parameters():
    weights = U.random_weights(U.MIXED, 2)
    cfg = config_from_dict(U.MIXED)
    lay = cfg.layout()
    specs = model_param_specs(lay)
    cmap = get_architecture("Famarax").checkpoint_map(cfg, lay)
    # the first layer's blend is in the checkpoint and read by nobody
    assert set(weights) - {s.name for s in cmap.sources} == {"l0.mix.vmix"}
    assert {s.name for s in cmap.sources} < set(weights)
    filled = {}
    for s in cmap.sources:
        assert tuple(weights[s.name].shape) == s.checkpoint_shape(specs[s.param].shape), s.name
        filled[s.param] = filled.get(s.param, 0) + s.rows
    assert {k: v.shape[0] for k, v in specs.items()} == filled
    assert specs["blocks.1.mixer.in.weight"].shape == (2 * 48 + 80 + 4 + 4 + 80, 64)
    assert specs["blocks.0.mixer.qkv.weight"].shape == (4 * 24 + 2 * 24 + 2 * 40, 64)
    assert specs["embed.norm.alpha"].shape == specs["blocks.3.mixer.value_mix"].shape == (1,)
    assert "blocks.0.mixer.q_norm.weight" not in specs and "blocks.3.norm2.weight" not in specs
    params = load_parameters(weights, specs, cmap, torch.bfloat16, "cpu")
    assert float(params["blocks.5.norm1.alpha"]) == float(weights["l5.norm1.alpha"])
    assert torch.equal(params["blocks.1.mixer.in.weight"][176:180], weights["l1.mix.b"])
    assert torch.equal(params["blocks.1.mixer.in.weight"][184:], weights["l1.mix.g"])
    # a number where a vector of one is expected, and the other way round, is a wrong shape
    with pytest.raises(WeightsError, match="l5.norm1.alpha"):
        load_parameters(dict(weights, **{"l5.norm1.alpha": torch.ones(1)}), specs, cmap,
                        torch.bfloat16, "cpu")


def test_tensors_of_an_absent_sublayer_are_left_alone():
    weights = U.random_weights(U.MIXED, 2)
    cfg = config_from_dict(U.MIXED)
    lay = cfg.layout()
    cmap = get_architecture("Famarax").checkpoint_map(cfg, lay)
    extra = {"l3.norm2": torch.ones(64), "l3.norm2.b": torch.ones(64), "l3.norm2.alpha": torch.ones(()),
             "l3.hc2.in": torch.ones(3), "l3.hc2.out": torch.ones(3), "l3.hc2.mix": torch.eye(3)}
    load_parameters({**weights, **extra}, model_param_specs(lay), cmap, torch.bfloat16, "cpu")
    with pytest.raises(WeightsError, match="l3.mlp.router"):
        load_parameters({**weights, "l3.mlp.router": torch.ones(4, 64)}, model_param_specs(lay), cmap,
                        torch.bfloat16, "cpu")


def test_random_weights_mode_makes_a_loadable_checkpoint():
    cfg = config_from_dict(U.MIXED)
    lay = cfg.layout()
    tensors = random_checkpoint(cfg, seed=3)
    assert tensors["embed.norm.alpha"].shape == () and tensors["l3.mix.vmix"].shape == ()
    load_parameters(tensors, model_param_specs(lay),
                    get_architecture("Famarax").checkpoint_map(cfg, lay), torch.bfloat16, "cpu")


def test_unusable_configurations_name_everything():
    raw = copy.deepcopy(U.MIXED)
    del raw["layers"][0]["mixer"]["scale"]
    raw["layers"][1]["mixer"]["heads"] = 5
    raw["layers"][1]["mlp"]["router"]["groups"]["count"] = 4
    raw["layers"][2]["mixer"]["rot"]["dims"] = 7
    raw["layers"][3]["type"] = "attention_3"
    raw["layers"][4]["mlp"]["router"]["top"] = 6
    raw["layers"][5]["mixer"]["vdim"] = 24
    raw["layers"][5]["mlp"]["router"]["groups"]["keep"] = 9
    raw["streams"] = 9
    del raw["vocab"]
    with pytest.raises(ConfigError) as err:
        config_from_dict(raw)
    text = str(err.value)
    for part in ("layers[0].mixer.scale", "layers[1].mixer.heads", "4 equal groups", "rot.dims",
                 "attention_3", "layers[4].mlp.router.top", "blends 2 x 24", "groups.keep",
                 "config.streams", "vocab"):
        assert part in text, part


def test_plain_mechanisms_on_hand_computed_cases():
    # dynamic tanh: one alpha, a weight and a bias a feature
    y = P.plain_dynamic_tanh(np.array([[0.5, -2.0]]), 2.0, [3.0, 1.0], [0.0, 0.25])
    assert np.allclose(y, [[3 * np.tanh(1.0), 0.25 - np.tanh(4.0)]])
    # halves of the rotated part are paired, features beyond pass
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]])
    y = P.plain_rotate_half(x, [3], 4, 100.0)
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(y[0, 0], [np.cos(a0), -2 * np.sin(a1), np.sin(a0), 2 * np.cos(a1), 5])
    # a rotation keeps the root mean square, so the norm may stand on either side of it
    q = np.random.default_rng(0).normal(size=(5, 2, 8))
    rot = lambda z: P.plain_rotate_half(z, np.arange(5), 6, 30.0)
    assert np.allclose(P.plain_over_rms(rot(q), 1e-6), rot(P.plain_over_rms(q, 1e-6)))
    # a window of two sees itself and one before; equal scores share the weight
    v = np.arange(4.0).reshape(4, 1, 1)
    o = P.plain_window_attention(np.zeros((4, 1, 3)), np.ones((4, 1, 3)), v, 0, 1.0, None, 2)
    assert np.allclose(o[:, 0, 0], [0.0, 0.5, 1.5, 2.5])
    # one number fades the whole matrix; a second write along a key replaces what it finds
    k = np.array([[1.0, 0.0], [1.0, 0.0], [0.0, 1.0]])
    S = np.zeros((2, 1))
    o = P.plain_delta_rule(k, k, np.array([[3.0], [5.0], [7.0]]), np.full(3, 0.5),
                           np.array([1.0, 0.5, 0.25]), S)
    assert np.allclose(o[:, 0], [1.5, 0.75 + 0.5 * (5 - 0.75), 3.5])
    assert np.allclose(S[:, 0], [2.875 * 0.25, 3.5])
    assert np.allclose(P.plain_mix_values(np.array([2.0]), np.array([10.0]), 0.25), [4.0])


def test_plain_choice_of_experts():
    z = np.log(np.array([[0.4, 0.05, 0.2, 0.15, 0.12, 0.08]]))
    # no correction, no groups: the two largest, renormalised and scaled
    c, w = P.plain_route(z, np.zeros(6), 2, None, 3.0)
    assert list(c[0]) == [0, 2] and np.allclose(w[0], [3 * 0.4 / 0.6, 3 * 0.2 / 0.6])
    # the correction decides the choice and stays out of the weights; choice scores of both signs
    corr = np.array([-0.9, 0.0, -0.3, 0.0, 0.0, 0.3])
    c, w = P.plain_route(z, corr, 2, None, 1.0)
    assert list(c[0]) == [5, 3] and np.allclose(w[0], [0.08 / 0.23, 0.15 / 0.23])
    # groups {0,1}, {2,3}, {4,5}: their best are 0.05, 0.15, 0.38; one is kept, then two
    assert list(P.plain_route(z, corr, 2, {"count": 3, "keep": 1})[0][0]) == [5, 4]
    assert list(P.plain_route(z, corr, 3, {"count": 3, "keep": 2})[0][0]) == [5, 3, 4]
    # a closed expert is closed, not zero: with negative scores everywhere it still loses
    low = np.full(6, -2.0)
    low[:2] = -1.0
    assert sorted(P.plain_route(z, low, 2, {"count": 3, "keep": 1})[0][0]) == [0, 1]


def test_plain_model_in_portions_equals_whole_and_every_mechanism_matters():
    w = U.as_numpy(U.random_weights(U.MIXED, 4))
    toks = U.tokens(U.MIXED, 19, 1)
    whole = P.plain_forward(toks, w, U.MIXED)
    states = [{} for _ in U.MIXED["layers"]]
    parts = [P.plain_forward(toks[a:b], w, U.MIXED, states) for a, b in ((0, 7), (7, 9), (9, 10), (10, 19))]
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9

    def differs(w2=None, **cfg):
        return np.abs(P.plain_forward(toks, w2 or w, dict(U.MIXED, **cfg)) - whole).max() > 1e-2

    assert differs(logit_softcap=None) and differs(logit_scale=1.0)
    for name in ("embed.norm.alpha", "l3.mix.vmix", "l1.mix.dt_bias", "l0.mlp.correction", "l2.hc2.mix"):
        assert differs(dict(w, **{name: w[name] * 0.5})), name
    for i, path, value in ((0, ("mixer", "mask", "size"), 10), (5, ("mixer", "softcap"), 1.0),
                           (0, ("mlp", "router", "groups", "keep"), 4),
                           (5, ("mlp", "router", "scale"), 1.0)):
        layers = copy.deepcopy(U.MIXED["layers"])
        at = layers[i]
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        assert differs(layers=layers), path
    # the first layer's blend is not used
    assert not differs(dict(w, **{"l0.mix.vmix": w["l0.mix.vmix"] + 1.0}))
