"""Small Famarax configurations with random weights for the tests, and the plumbing to run them
through the plain implementation (the engine side is shared with the other decoders' tests:
``tifosun_util.run_schedule`` and its comparisons)."""
from __future__ import annotations

import copy

import torch

import plain_famarax as P
from tifosun_util import assert_close, relative_error, row_errors, run_schedule, tokens  # noqa: F401


def attention(heads=4, kv_heads=2, dim=24, vdim=40, scale=None, softcap=6.0, window=11, rot_dims=8,
              base=300.0, v_mix=True):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
           "scale": dim ** -0.5 if scale is None else scale}
    if rot_dims:
        out["rot"] = {"base": base, "dims": rot_dims}
    if softcap is not None:
        out["softcap"] = softcap
    if window is not None:
        out["mask"] = {"size": window}
    if v_mix is not None:
        out["v_mix"] = v_mix
    return out


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts=8, top=3, ff=40, shared_ff=56, groups=(4, 2), scale=1.6):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = dict(zip(("count", "keep"), groups))
    if scale is not None:
        router["scale"] = scale
    out = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff}
    return out


def layer(kind, mixer, mlp="moe"):
    return {"type": kind, "mixer": mixer, "mlp": moe() if mlp == "moe" else mlp}


def config(layers, width=64, vocab=157, eps=1e-5, streams=3, logit_scale=0.7, logit_softcap=9.0):
    out = {"architecture": "Famarax", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "streams": streams, "layers": copy.deepcopy(layers)}
    if logit_scale is not None:
        out["logit_scale"] = logit_scale
    if logit_softcap is not None:
        out["logit_softcap"] = logit_softcap
    return out


# Layers that differ in every size: query groups of 2, 1 and 4, value sizes above and below the
# key size, windows of 11, 30 and 7 and none, all, part and nothing of a head rotated, one to four
# taps, delta-rule heads that share keys and that do not, groups of one, two and three experts and
# no groups, no scale, no shared expert, a layer without a feed-forward, an attention between the
# layers with blended values that blends nothing, three copies of the residual.
MIXED = config([
    layer("attention", attention(4, 2, 24, 40, window=11)),
    layer("delta", delta(4, 2, 24, 20, 3), moe(6, 2, 24, 0, (2, 1), 0.8)),
    layer("attention", attention(3, 1, 16, 8, scale=0.5, softcap=2.5, window=None, rot_dims=16,
                                 base=50.0, v_mix=False), moe(9, 4, 16, 24, (3, 2), None)),
    layer("attention", attention(2, 2, 12, 40, softcap=None, window=30, rot_dims=0), mlp=None),
    layer("delta", delta(3, 3, 10, 36, 4), moe(5, 5, 24, 8, None, 1.0)),
    layer("attention", attention(8, 2, 40, 40, window=7, rot_dims=12), moe(8, 2, 32, 40, (8, 3), 2.2)),
])


def random_weights(cfg: dict, seed: int, sharp: float = 1.0) -> dict:
    """Checkpoint tensors (bfloat16 values).  Projections keep activations of order one (queries
    and keys have a root mean square of one whatever their projection: how sharp an attention is
    says its ``scale``); alphas lie where a good part of the inputs saturates the tanh and a good
    part does not; decays spread from nearly one to a half a token, write strengths over (0, 1),
    blends over (0.2, 0.8); corrections are as large as the scores, so that they decide choices,
    and choice scores of both signs occur."""
    g = torch.Generator().manual_seed(seed)
    w: dict = {}
    W, S = cfg["width"], cfg["streams"]

    def mat(name, rows, cols, gain=1.0):
        w[name] = (gain * torch.randn(rows, cols, generator=g) / cols ** 0.5).to(torch.bfloat16)

    def vec(name, n, mean=0.0, std=0.1):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def uniform(name, shape, lo, hi):
        w[name] = (lo + (hi - lo) * torch.rand(shape, generator=g)).to(torch.bfloat16)

    def norm(name, lo=0.3, hi=0.9):
        vec(name, W, 1.0, 0.2)
        vec(name + ".b", W, 0.0, 0.2)
        uniform(name + ".alpha", (), lo, hi)

    def expert(p, ff):
        mat(p + "gate", ff, W)
        mat(p + "up", ff, W)
        mat(p + "down", W, ff, 0.7)

    w["embed"] = torch.randn(cfg["vocab"], W, generator=g).to(torch.bfloat16)
    norm("embed.norm")
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        for q in (1, 2) if l["mlp"] is not None else (1,):
            norm(f"{p}norm{q}")
            vec(f"{p}hc{q}.in", S, 1.0 / S, 0.3)
            vec(f"{p}hc{q}.out", S, 1.0, 0.4)
            w[f"{p}hc{q}.mix"] = (torch.eye(S) * 0.8 + 0.25 * torch.randn(S, S, generator=g)).to(
                torch.bfloat16)
        m, q = l["mixer"], p + "mix."
        H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if l["type"] == "attention":
            mat(q + "q", H * D, W, sharp)
            mat(q + "k", G * D, W)
            mat(q + "v", G * VD, W)
            if m.get("v_mix"):
                uniform(q + "vmix", (), 0.2, 0.8)
        else:
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * VD)):
                mat(q + n, rows, W, 1.5)
                mat(q + n + ".conv", rows, m["conv"], 1.5)
            mat(q + "b", H, W, 2.0)
            mat(q + "a", H, W, 2.0)
            uniform(q + "dt_bias", (H,), -3.0, 0.0)
            w[q + "A_log"] = torch.log(0.3 + 2.0 * torch.rand(H, generator=g)).to(torch.bfloat16)
            mat(q + "g", H * VD, W, 2.0)
            vec(q + "norm", VD, 1.0, 0.3)
        mat(q + "o", W, H * VD)
        mlp = l["mlp"]
        if mlp is None:
            continue
        q, E = p + "mlp.", mlp["router"]["experts"]
        mat(q + "router", E, W, 2.0)
        vec(q + "correction", E, -0.5 / E, 1.0 / E)
        for e in range(E):
            expert(f"{q}e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            expert(q + "shared.", mlp["shared"]["ff"])
    norm("final.norm")
    mat("head", cfg["vocab"], W, 2.0)
    return w


def as_numpy(weights: dict) -> dict:
    return {k: v.double().numpy() for k, v in weights.items()}


def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v.double().numpy() for k, v in weights.items() if k.startswith(prefix)}


def plain_logits(cfg: dict, weights: dict, toks: list) -> torch.Tensor:
    """float64 logits [len(toks), vocab] of one sequence."""
    return torch.from_numpy(P.plain_forward(list(toks), as_numpy(weights), cfg))


def load(cfg: dict, weights: dict, dtype: str):
    from mstar_b200.config.registry import config_from_dict
    from mstar_b200.engine.model import load_model

    return load_model(None, dtype=dtype, device="cuda:0", config=config_from_dict(cfg),
                      tensors=weights)
