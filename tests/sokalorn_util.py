"""Small Sokalorn configurations with random weights for the tests, and the plumbing to run
them through the plain implementation (the engine side is shared with the other decoders'
tests: ``tifosun_util.run_schedule`` and its comparisons)."""
from __future__ import annotations

import copy

import torch

import plain_sokalorn as P
from tifosun_util import assert_close, relative_error, row_errors, run_schedule, tokens  # noqa: F401

RANK = 5      # of the time mixing's decay projection, where nothing else is said


def left(heads=4, kv_heads=2, dim=24, vdim=40, scale=None, softcap=6.0, chunk=11, rot_dims=8,
         base=300.0, factor=2.5):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
           "scale": dim ** -0.5 if scale is None else scale,
           "rot": {"base": base, "dims": rot_dims, "scaling": {"factor": factor}}}
    if softcap is not None:
        out["softcap"] = softcap
    if chunk is not None:
        out["mask"] = {"size": chunk}
    return out


def right(heads=3, dim=20):
    return {"heads": heads, "dim": dim}


def mamba2(heads=4, vdim=20, state=24, groups=2, conv=4, norm_groups=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
            "norm_groups": norm_groups}


def moe(experts=6, top=2, ff=40, limit=1.2, shared_ff=56, shared_limit=0.8):
    out = {"kind": "moe", "router": {"experts": experts, "top": top},
           "expert": {"ff": ff, "limit": limit}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def parallel(l=None, r=None, mlp="moe"):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right()},
            "mlp": moe() if mlp == "moe" else mlp}


def ssd(m=None, mlp="moe"):
    return {"type": "mamba2", "mixer": m or mamba2(), "mlp": moe() if mlp == "moe" else mlp}


def config(layers, width=64, vocab=157, eps=1e-5, loop=None):
    out = {"architecture": "Sokalorn", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "layers": copy.deepcopy(layers)}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# Layers that differ in every size: query groups of 2, 3 and 1, value sizes above and below the
# key size, chunks of 11, 16 and 7 positions, one to four taps, groups and norm groups of one and
# more, more experts than a token uses and as many, a layer without a feed-forward, one without a
# shared expert, a stretch of three layers that runs twice.
MIXED = config([
    ssd(mamba2(4, 20, 24, 2, 4, 2)),
    parallel(left(4, 2, 24, 40, chunk=11), right(3, 20)),
    ssd(mamba2(6, 8, 40, 3, 2, 1), moe(3, 3, 24, 0.7, 0)),
    parallel(left(3, 1, 16, 8, scale=0.5, softcap=2.0, chunk=16, rot_dims=16, base=50.0, factor=4.0),
             right(2, 36), mlp=None),
    parallel(left(2, 2, 12, 20, softcap=None, chunk=7, rot_dims=4), right(1, 8), moe(9, 4, 16)),
], loop=(1, 4, 2))


def random_weights(cfg: dict, seed: int, sharp: float = 1.0, rank: int = RANK) -> dict:
    """Checkpoint tensors (bfloat16 values).  Projections keep activations of order one;
    ``sharp`` multiplies the query projection (the tests of the attention alone use 3: weights
    near zero and one); the score bias keeps most sigmoid weights small, or the sums over the
    keys would drown everything else; decays of both recurrences spread from nearly one to a
    half a token; clamps and gates of the experts are reached by a good part of the units."""
    g = torch.Generator().manual_seed(seed)
    w: dict = {}
    W = cfg["width"]

    def mat(name, rows, cols, gain=1.0):
        w[name] = (gain * torch.randn(rows, cols, generator=g) / cols ** 0.5).to(torch.bfloat16)

    def vec(name, n, mean=0.0, std=0.1):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def uniform(name, n, lo, hi):
        w[name] = (lo + (hi - lo) * torch.rand(n, generator=g)).to(torch.bfloat16)

    def expert(p, ff):
        mat(p + "gate", ff, W, 1.5)
        mat(p + "up", ff, W, 1.5)
        mat(p + "down", W, ff)

    w["embed"] = torch.randn(cfg["vocab"], W, generator=g).to(torch.bfloat16)
    if cfg.get("loop"):
        mat("loop.in", W, 2 * W, 1.4)
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        vec(p + "norm1", W, 1.0, 0.2)
        uniform(p + "shift", W, 0.0, 1.0)
        if l["type"] == "parallel":
            a, q = l["mixer"]["left"], p + "mix.left."
            H, G, D, VD = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            mat(q + "q", H * D, W, sharp)
            mat(q + "k", G * D, W)
            mat(q + "v", G * VD, W)
            mat(q + "g", H * VD, W, 2.0)
            vec(q + "pb", H, -1.5, 0.7)
            mat(q + "o", W, H * VD)
            vec(q + "out", W, 1.0, 0.2)
            m, r = l["mixer"]["right"], p + "mix.right."
            HD = m["heads"] * m["dim"]
            rk = m.get("decay_rank", rank)
            for s in "rkvgw":
                uniform(r + "mu." + s, W, 0.0, 1.0)
            for s in "rkvg":
                mat(r + s, HD, W)
            mat(r + "w1", rk, W)
            mat(r + "w2", HD, rk, 2.0)
            uniform(r + "w0", HD, -6.0, -0.5)
            vec(r + "u", HD, 0.0, 1.0)
            w[r + "u"] = w[r + "u"].view(m["heads"], m["dim"])
            vec(r + "norm", HD, 1.0, 0.2)
            mat(r + "o", W, HD)
            vec(r + "out", W, 1.0, 0.2)
        else:
            m, q = l["mixer"], p + "mix."
            inner = m["heads"] * m["vdim"]
            chan = inner + 2 * m["groups"] * m["state"]
            mat(q + "in", inner + chan + m["heads"], W, 1.5)
            mat(q + "conv", chan, m["conv"], 1.5)
            vec(q + "conv.b", chan, 0.0, 0.3)
            uniform(q + "dt_bias", m["heads"], -4.0, 0.5)
            w[q + "A_log"] = torch.log(0.1 + 2.0 * torch.rand(m["heads"], generator=g)).to(torch.bfloat16)
            vec(q + "D", m["heads"], 1.0, 0.3)
            vec(q + "norm", inner, 1.0, 0.2)
            mat(q + "o", W, inner)
        mlp = l["mlp"]
        if mlp is None:
            continue
        q = p + "mlp."
        mat(q + "router", mlp["router"]["experts"], W, 3.0)
        for e in range(mlp["router"]["experts"]):
            expert(f"{q}e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            expert(q + "shared.", mlp["shared"]["ff"])
            mat(q + "shared.sg", 1, W, 2.0)
    vec("final.norm", W, 1.0, 0.2)
    mat("head", cfg["vocab"], W)
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


def runs(cfg: dict) -> int:
    return len(P.plain_run_order(cfg))


def shaped(raw, weights=None):
    """The typed configuration with the rank that only the tensors give."""
    from mstar_b200.config.registry import config_from_dict
    from mstar_b200.weights.loader import checkpoint_shapes

    cfg = config_from_dict(raw)
    return cfg.with_shapes(checkpoint_shapes(weights if weights is not None
                                             else random_weights(raw, 1)))


assert [i for i, _ in P.plain_run_order(MIXED)] == [0, 1, 2, 3, 1, 2, 3, 4]
