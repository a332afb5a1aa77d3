"""The Famarax decoder in the engine against the plain implementation (tests/plain_famarax.py):
each mechanism alone, then whole models through the step function, the cache and state manager,
the scheduler and the entry point, under every kind of schedule."""
import numpy as np
import pytest
import torch

import famarax_util as U
import plain_famarax as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
EPS = 1e-5


def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (scale * torch.randn(*shape, generator=g)).to(torch.bfloat16)


def runtime(dtype):
    from mstar_b200.parts import Runtime
    return Runtime(dtype=TORCH[dtype], device=torch.device(DEV))


def dev(t, dtype):
    return t.to(TORCH[dtype]).to(DEV)


def f64(t):
    return t.double().numpy()


def step_ctx(q_lens, starts, slots=None):
    from test_gpu_parts import simple_ctx
    ctx = simple_ctx(q_lens, starts)
    if slots is not None:
        ctx.slots = torch.tensor(slots, dtype=torch.int32, device=DEV)
        ctx.host_slots = list(slots)
    return ctx


def close(got, want, dtype, what, f32=2e-5, bf16=4e-2):
    """Worst difference relative to the largest wanted value."""
    want = torch.as_tensor(np.asarray(want))
    err = (got.double().cpu() - want.double()).abs().max().item() / want.abs().max().item()
    assert err < (f32 if dtype == "float32" else bf16), (what, dtype, err)


# ------------------------------------------------------------------ norms and residual
def tanh_norm(width, seed, alpha=0.7):
    w, b = rnd(width, seed=seed) + 1.0, rnd(width, seed=seed + 1, scale=0.3)
    return w, b, alpha


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 50, 1000, 2048, 4104])
def test_dynamic_tanh_alone(dtype, width):
    """The norm as a part: a pending output folded into the residual, rows without one, the
    embedding rows (tokens from the host and from the device); inputs far into saturation and
    near zero."""
    from mstar_b200 import ops
    from mstar_b200.config.layout import EmbeddingSpec, NormSpec
    from mstar_b200.parts import build_part
    from mstar_b200.parts.base import ResidualStream

    w, b, alpha = tanh_norm(width, 1)
    part = build_part("norm", NormSpec(kind="dynamic_tanh", size=width),
                      {"weight": dev(w, dtype), "bias": dev(b, dtype),
                       "alpha": torch.tensor([alpha], device=DEV)}, runtime(dtype))
    x, d = rnd(9, width, seed=3, scale=4.0).float(), rnd(9, width, seed=4)
    x[0] *= 100.0
    x[1] *= 1e-3
    stream = ResidualStream(x.to(DEV).contiguous())
    stream.push(dev(d, dtype))
    got = part.add_norm(stream)
    want = P.plain_dynamic_tanh(f64(x) + f64(d), alpha, f64(w), f64(b))
    close(got, want, dtype, "add and norm", bf16=8e-3)
    close(stream.h, f64(x) + f64(d), "float32", "residual")
    close(part.norm_rows(x.to(DEV)), P.plain_dynamic_tanh(f64(x), alpha, f64(w), f64(b)), dtype,
          "rows", bf16=8e-3)
    # after a sublayer: resid += scale * norm(output)
    resid = x.to(DEV).clone()
    part.add_normed(resid, dev(d, dtype), 0.5)
    close(resid, f64(x) + 0.5 * P.plain_dynamic_tanh(f64(d), alpha, f64(w), f64(b)), "float32", "post")
    # the embedding's norm; the second and third token are on the device only
    table = rnd(31, width, seed=5)
    emb = build_part("embedding", EmbeddingSpec(vocab_size=31, hidden_size=width, multiplier=1.5,
                                                norm=NormSpec(kind="dynamic_tanh", size=width)),
                     {"weight": dev(table, dtype), "norm.weight": dev(w, dtype),
                      "norm.bias": dev(b, dtype), "norm.alpha": torch.tensor([alpha], device=DEV)},
                     runtime(dtype))
    ctx = step_ctx([4], [0])
    ids = torch.tensor([7, 0, 0, 30], dtype=torch.int32, device=DEV)
    ctx.token_source = (torch.tensor([-1, 1, 0, -1], dtype=torch.int32, device=DEV),
                        torch.tensor([12, 29], dtype=torch.int32, device=DEV))
    got = emb.forward(ids, ctx)
    assert got.dtype == torch.float32
    close(got, P.plain_dynamic_tanh(1.5 * f64(table)[[7, 29, 12, 30]], alpha, f64(w), f64(b)),
          "float32", "embedding")


def test_embedding_with_another_norm():
    """The embedding takes any norm part; a kind without a fused kernel runs after the lookup."""
    from mstar_b200.config.layout import EmbeddingSpec, NormSpec
    from mstar_b200.parts import build_part

    table, w = rnd(20, 48, seed=1), rnd(48, seed=2) + 1.0
    emb = build_part("embedding", EmbeddingSpec(vocab_size=20, hidden_size=48,
                                                norm=NormSpec(kind="rmsnorm", size=48, eps=EPS)),
                     {"weight": dev(table, "bfloat16"), "norm.weight": dev(w, "bfloat16")},
                     runtime("bfloat16"))
    got = emb.forward(torch.tensor([3, 19], dtype=torch.int32, device=DEV), step_ctx([2], [0]))
    close(got, P.plain_over_rms(f64(table)[[3, 19]], EPS) * f64(w), "float32", "normed embedding")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,width", [(1, 64), (2, 200), (3, 1001), (4, 2048), (8, 72), (5, 4100)])
def test_hyper_connections_through_a_dynamic_tanh(dtype, streams, width):
    """First read from the embedding output, a write with one output, a write with two weighted
    outputs and a bias, and the sum of chosen rows through a norm with a write still pending."""
    from mstar_b200 import ops

    T = 7
    g = torch.Generator().manual_seed(streams)
    emb = rnd(T, width, seed=1).float()
    tabs = [(torch.randn(streams, generator=g), torch.randn(streams, generator=g),
             torch.randn(streams, streams, generator=g)) for _ in range(3)]
    norms = [tanh_norm(width, 10 + 2 * i, 0.3 + 0.4 * i) for i in range(3)]
    y1, y2 = rnd(T, width, seed=3, scale=2.0), rnd(T, width, seed=4, scale=2.0)
    bias = rnd(width, seed=5)
    x = torch.empty(T, streams, width, device=DEV)
    f = lambda t: t.contiguous().to(DEV)
    n = lambda i: (dev(norms[i][0], dtype), dev(norms[i][1], dtype), norms[i][2])
    plain = lambda i, u: P.plain_dynamic_tanh(u, norms[i][2], f64(norms[i][0]), f64(norms[i][1]))
    xs = np.stack([f64(emb)] * streams)
    got = ops.hyper_step(x, init=f(emb), mix=f(torch.eye(streams)), out=f(torch.zeros(streams)),
                         read=f(tabs[0][0]), tanh_norm=n(0), out_dtype=TORCH[dtype])
    close(got, plain(0, P.plain_hyper_read(xs, f64(tabs[0][0]))), dtype, "first read", bf16=8e-3)
    close(x.transpose(0, 1), xs, "float32", "copies written")
    xs = P.plain_hyper_write(xs, f64(y1), f64(tabs[0][2]), f64(tabs[0][1]))
    got = ops.hyper_step(x, y=dev(y1, dtype), mix=f(tabs[0][2]), out=f(tabs[0][1]), read=f(tabs[1][0]),
                         tanh_norm=n(1), out_dtype=TORCH[dtype], x_static=True)
    close(x.transpose(0, 1), xs, "float32", "write")
    close(got, plain(1, P.plain_hyper_read(xs, f64(tabs[1][0]))), dtype, "read after write", bf16=8e-3)
    y = 1.2 * f64(y1) + 0.9 * f64(y2) + f64(bias)
    after = P.plain_hyper_write(xs, y, f64(tabs[1][2]), f64(tabs[1][1]))
    rows = torch.tensor([T - 1, 0, 3, 3], dtype=torch.int32, device=DEV)
    before = x.clone()
    got = ops.hyper_step(x, y=dev(y1, dtype), y2=dev(y2, dtype), y_scales=(1.2, 0.9),
                         y_bias=dev(bias, dtype), mix=f(tabs[1][2]), out=f(tabs[1][1]), rows=rows,
                         tanh_norm=n(2), out_dtype=TORCH[dtype])
    close(got, plain(2, after.sum(0)[[T - 1, 0, 3, 3]]), dtype, "normed sum of copies", bf16=8e-3)
    assert torch.equal(x, before)                      # a sum leaves the copies alone


# ------------------------------------------------------------------ attention
def attention_part(m, width, dtype, seed, sharp=1.0, mix=None):
    """(part, spec, plain tensors) of an attention; ``mix``: None, "first" or "blend"."""
    from dataclasses import replace

    from mstar_b200.config.registry import config_from_dict
    from mstar_b200.parts import build_part

    cfg = U.config([U.layer("attention", m)], width=width)
    w = U.random_weights(cfg, seed, sharp=sharp)
    p = "l0.mix."
    spec = replace(config_from_dict(cfg).layout().blocks[0].mixer, value_mix=mix)
    params = {"qkv.weight": torch.cat([w[p + n] for n in ("q", "k", "v")]), "o.weight": w[p + "o"]}
    if mix == "blend":
        params["value_mix"] = w[p + "vmix"].reshape(1)
    part = build_part("mixer", spec, {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    return part, spec, U.sub(w, p)


def paged_cache(part_spec, tokens, page, dtype, seed=1):
    """Pages scattered over a pool that holds leftovers of other requests."""
    from mstar_b200 import ops
    from mstar_b200.parts import LayerCache

    pages = -(-tokens // page)
    elems = ops.sink_page_elements(part_spec.num_kv_heads, page, part_spec.head_dim,
                                   part_spec.value_dim)
    kv = torch.full((pages + 3, elems), 7.0, dtype=TORCH[dtype], device=DEV)
    table = (torch.randperm(pages + 3, generator=torch.Generator().manual_seed(seed))[:pages]
             .to(torch.int32).to(DEV)[None])
    return LayerCache(kv=kv, page_size=page, block_table=table)


def plain_attention(x, p, m):
    return P.plain_attention(x, np.arange(x.shape[0]), p, "", dict(m, v_mix=False), EPS, {}, {})


ATTENTIONS = [
    (U.attention(4, 2, 24, 40, window=11), 4),
    (U.attention(3, 3, 16, 8, scale=0.9, softcap=2.0, window=1, rot_dims=16), 8),
    (U.attention(34, 1, 16, 24, scale=1.2, softcap=20.0, window=29, rot_dims=4), 16),
    (U.attention(2, 1, 160, 256, scale=0.2, softcap=8.0, window=16, rot_dims=32, base=1e6), 8),
    (U.attention(2, 2, 12, 10, scale=0.8, softcap=None, window=64), 4),
    (U.attention(4, 2, 128, 128, scale=0.19, softcap=9.0, window=None, rot_dims=128, base=7e4), 16),
    (U.attention(1, 1, 20, 20, scale=1.0, softcap=4.0, window=50, rot_dims=2, base=10.0), 8),
    (U.attention(5, 5, 96, 72, scale=0.25, window=17, rot_dims=0), 16),
    (U.attention(8, 2, 64, 64, scale=0.21, softcap=18.0, window=33, rot_dims=64), 16),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", ATTENTIONS)
def test_attention_alone(dtype, m, page):
    """Scores so sharp that a query's weight lies on a few keys; a prompt portion, portions of
    two, single tokens, pages scattered over the pool.  The norm, the rotation, the cap and the
    window each change the output."""
    part, spec, p = attention_part(m, 96, dtype, seed=7, sharp=3.0)
    T = 70
    x = rnd(T, 96, seed=8)
    want = plain_attention(f64(x), p, m)
    for key in ("softcap", "mask", "rot"):
        if m.get(key) and not (key == "mask" and m[key]["size"] >= T) and not (
                key in ("softcap", "rot") and m.get("mask", {}).get("size") == 1):
            assert np.abs(plain_attention(f64(x), p, dict(m, **{key: None})) - want).max() > (
                0.01 * np.abs(want).max()), key
    cache = paged_cache(spec, T, page, dtype)
    outs, at = [], 0
    for n in (23, 2, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 29, 3, 2):
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
        at += n
    assert at == T
    close(torch.cat(outs), want, dtype, "attention", bf16=6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,window", [(8, 2, 64, 300), (4, 4, 32, 1000), (8, 1, 128, 37)])
def test_long_prompts(dtype, heads, kv_heads, dim, window):
    """Prompts of more tokens than a few row tiles in one step, then a portion, then single
    tokens, against float64 (windows shorter and longer than a key tile)."""
    m = U.attention(heads, kv_heads, dim, dim, scale=2.0 * dim ** -0.5, softcap=15.0, window=window,
                    rot_dims=dim // 2, base=1e4)
    part, spec, p = attention_part(m, 64, dtype, seed=5)
    T = 1300
    x = rnd(T, 64, seed=6)
    want = plain_attention(f64(x), p, m)
    cache = paged_cache(spec, T, 16, dtype)
    outs, at = [], 0
    for n in [1100, 187] + [1] * 13:
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
        at += n
    assert at == T
    close(torch.cat(outs), want, dtype, ("long prompt", window), bf16=6e-2)


def marked_inputs(p, m, width, T, marked, queries, gain=6.0):
    """Inputs in which the key at ``marked`` stands out for the ``queries``: the query tokens lie
    along a direction d, the marked token along the direction whose key equals the query of d (a
    solution of W_k d' = W_q d; no rotation), so that of the normed keys it alone points along the
    query."""
    x = rnd(T, width, seed=4, scale=0.3)
    d = f64(rnd(width, seed=5))
    d /= np.linalg.norm(d)
    target = p["q"][:m["dim"]] @ d                             # the first query head
    d_key = np.linalg.lstsq(p["k"][:m["dim"]], target, rcond=None)[0]
    d_key /= np.linalg.norm(d_key)
    x[marked] = torch.from_numpy(gain * d_key).to(torch.bfloat16)
    for q in queries:
        x[q] += torch.from_numpy(gain * d).to(torch.bfloat16)
    return x


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,page", [(80, 16), (81, 16), (64, 4), (130, 8), (16, 16)])
def test_edges_of_a_window(dtype, window, page):
    """A key that stands out is the oldest of one query's window and just outside the next
    query's: in one prompt, in portions cut at and around both, and decoded.  Inside, the output
    hangs on that key; outside, not at all."""
    m = U.attention(2, 1, 32, 32, scale=1.0, softcap=40.0, window=window, rot_dims=0)
    part, spec, p = attention_part(m, 64, dtype, seed=3)
    T = 2 * window + 9
    for marked in (0, 5, page, window):
        inside, outside = marked + window - 1, marked + window
        x = marked_inputs(p, m, 64, T, marked, [q for q in (inside, outside) if q < T])
        want = plain_attention(f64(x), p, m)
        hidden = f64(x).copy()
        hidden[marked] = 0.0
        blind = plain_attention(hidden, p, m)
        assert np.abs(blind[inside] - want[inside]).max() > 0.3 * np.abs(want[inside]).max()
        assert np.abs(blind[outside] - want[outside]).max() < 1e-9
        for cuts in ([T], [outside, T - outside], [inside, 2, T - inside - 2], [inside - 1]):
            cache = paged_cache(spec, T, page, dtype, seed=len(cuts))
            outs, at = [], 0
            for n in cuts + [1] * min(7, T - sum(cuts)):
                outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
                at += n
            got = torch.cat(outs)
            ref = torch.from_numpy(want)[:at]
            # row by row: a stray key would drown in the largest rows
            err = (got.double().cpu() - ref).abs().amax(1) / ref.abs().amax(1)
            assert float(err.max()) < (1e-4 if dtype == "float32" else 8e-2), (marked, cuts, int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("marked,page", [(0, 16), (15, 16), (16, 16), (3, 4), (257, 8)])
def test_one_far_key_stands_out(dtype, marked, page):
    """One key hundreds of tokens back (the first token, the last of a page, the first of the
    next) carries a query's weight, under a window that still holds it and without one."""
    T, queries = 330, [300, 329]
    for window in (None, 330):
        m = U.attention(2, 1, 32, 32, scale=1.0, softcap=40.0, window=window, rot_dims=0)
        part, spec, p = attention_part(m, 64, dtype, seed=3)
        x = marked_inputs(p, m, 64, T, marked, queries)
        want = plain_attention(f64(x), p, m)
        hidden = f64(x).copy()
        hidden[marked] = 0.0
        blind = plain_attention(hidden, p, m)
        for q in queries:             # how much hangs on the one key
            assert np.abs(blind[q] - want[q]).max() > 0.3 * np.abs(want[q]).max(), (marked, q)
        for first in (T, 290):                    # one prompt; a prompt and decoded tokens
            cache = paged_cache(spec, T, page, dtype, seed=first)
            outs = [part.forward(dev(x[:first], dtype), step_ctx([first], [0]), cache)]
            outs += [part.forward(dev(x[t:t + 1], dtype), step_ctx([1], [t]), cache)
                     for t in range(first, T)]
            close(torch.cat(outs), want, dtype, ("far key", marked, first), bf16=6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_heads,vdim,page", [(2, 40, 4), (1, 16, 16), (3, 7, 8)])
def test_blended_values(dtype, kv_heads, vdim, page):
    """A first layer hands its values on, a second of other sizes blends them in before it caches
    its own; a batch of two requests at different places, then single tokens.  The first layer
    itself blends nothing, and a step uses the values of its own tokens."""
    from mstar_b200.parts import LayerCache

    first_m = U.attention(kv_heads * 2, kv_heads, 24, vdim, window=9)
    second_m = U.attention(kv_heads, kv_heads, 16, vdim, window=20, rot_dims=16)
    first, fspec, fp = attention_part(first_m, 64, dtype, seed=1, mix="first")
    second, sspec, sp = attention_part(second_m, 64, dtype, seed=2, mix="blend")
    lens = {"a": 30, "b": 21}
    xs = {r: (rnd(n, 64, seed=n), rnd(n, 64, seed=n + 1)) for r, n in lens.items()}
    want = {}
    for r, (x1, x2) in xs.items():
        shared, pos = {}, np.arange(len(x1))
        want[r] = [P.plain_attention(f64(x1), pos, fp, "", dict(first_m, v_mix=True), EPS, {}, shared),
                   P.plain_attention(f64(x2), pos, sp, "", dict(second_m, v_mix=True), EPS, {}, shared)]
        alone = plain_attention(f64(x2), sp, second_m)
        assert np.abs(alone - want[r][1]).max() > 0.1 * np.abs(want[r][1]).max()

    def pool(spec, seed):
        a, b = (paged_cache(spec, 30, page, dtype, seed=seed) for _ in range(2))
        kv = torch.cat([a.kv, b.kv])
        return LayerCache(kv=kv, page_size=page,
                          block_table=torch.cat([a.block_table, b.block_table + a.kv.shape[0]]))

    c1, c2 = pool(fspec, 1), pool(sspec, 2)
    at = {"a": 0, "b": 0}
    got = {r: ([], []) for r in lens}
    for step in ((("a", 17), ("b", 2)), (("a", 1), ("b", 18)), (("a", 1), ("b", 1)), (("a", 11), ("b", 0))):
        parts = [(r, n) for r, n in step if n]
        ctx = step_ctx([n for _, n in parts], [at[r] for r, _ in parts])
        rows = ["ab".index(r) for r, _ in parts]
        for k, (part, c) in enumerate(((first, c1), (second, c2))):
            x = torch.cat([xs[r][k][at[r]:at[r] + n] for r, n in parts])
            y = part.forward(dev(x, dtype), ctx, LayerCache(kv=c.kv, page_size=page,
                                                            block_table=c.block_table[rows].contiguous()))
            row = 0
            for r, n in parts:
                got[r][k].append(y[row:row + n])
                row += n
        for r, n in parts:
            at[r] += n
    for r in lens:
        for k in range(2):
            close(torch.cat(got[r][k]), want[r][k], dtype, ("blended", r, k), bf16=6e-2)


# ------------------------------------------------------------------ delta rule
def delta_part(m, width, dtype, seed):
    from mstar_b200.config.registry import config_from_dict
    from mstar_b200.parts import build_part

    cfg = U.config([U.layer("delta", m)], width=width)
    w = U.random_weights(cfg, seed)
    p = "l0.mix."
    spec = config_from_dict(cfg).layout().blocks[0].mixer
    params = {"in.weight": torch.cat([w[p + n] for n in ("q", "k", "v", "b", "a", "g")]),
              "conv.weight": torch.cat([w[p + n + ".conv"] for n in ("q", "k", "v")]),
              "dt_bias": w[p + "dt_bias"], "A_log": w[p + "A_log"], "norm.weight": w[p + "norm"],
              "o.weight": w[p + "o"]}
    part = build_part("mixer", spec, {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    return part, spec, U.sub(w, p)


DELTAS = [(4, 2, 24, 20, 3), (3, 3, 10, 36, 4), (1, 1, 64, 32, 1), (4, 4, 64, 48, 3), (6, 2, 72, 130, 2),
          (2, 1, 130, 8, 5), (8, 2, 300, 16, 2), (4, 2, 128, 256, 4), (1, 1, 1, 4, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", DELTAS)
def test_delta_rule_with_one_decay_a_head(dtype, heads, kv_heads, dim, vdim, taps):
    """A sequence cut into a portion, a two-token portion, single tokens (fewer than the
    convolution has taps) and more portions, in a slot that held another request's state; then
    two sequences in one batch in other slots."""
    from mstar_b200 import ops
    from mstar_b200.parts import LayerCache

    m = U.delta(heads, kv_heads, dim, vdim, taps)
    part, spec, p = delta_part(m, 96, dtype, seed=dim)
    T = 45
    x = rnd(T, 96, seed=5)
    want = P.plain_gated_delta(f64(x), p, "", m, EPS, {})
    size = ops.gated_delta_state_size(heads, kv_heads, dim, vdim, taps)
    slots = torch.randn(4, size, device=DEV)               # leftovers of earlier requests
    slots[2].zero_()
    cache = LayerCache(state=slots)
    outs, at = [], 0
    for n in (19, 2, 1, 1, 1, 17, 4):
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at], [2]), cache))
        at += n
    assert at == T
    close(torch.cat(outs), want, dtype, "delta rule", bf16=5e-2)
    slots2 = torch.zeros(4, size, device=DEV)
    both = part.forward(dev(torch.cat([x[:9], x[:30]]), dtype), step_ctx([9, 30], [0, 0], [3, 0]),
                        LayerCache(state=slots2))
    close(both[:9], want[:9], dtype, "first of two", bf16=5e-2)
    close(both[9:], want[:30], dtype, "second of two", bf16=5e-2)
    assert float(slots2[1].abs().max()) == 0.0 and float(slots2[3].abs().max()) > 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps",
                         [(4, 2, 24, 20, 3), (2, 1, 128, 40, 2), (2, 2, 200, 9, 1), (5, 1, 64, 64, 3),
                          (2, 2, 32, 12, 3), (2, 1, 256, 20, 2), (3, 1, 64, 7, 4), (24, 2, 32, 36, 4),
                          (16, 4, 128, 128, 4), (3, 3, 96, 10, 4)])
def test_delta_rule_long_portions_in_pieces(dtype, heads, kv_heads, dim, vdim, taps):
    """A portion long enough to be scanned in pieces of 16 tokens (key sizes of 32, 64, 96, 128
    and 256; the others and a state that does not start on a 16-byte boundary token by token), beside a short portion of another request in the same batch; then more
    tokens of both, a portion that is no multiple of 16 and a last one of a single token."""
    from mstar_b200 import ops
    from mstar_b200.parts import LayerCache

    m = U.delta(heads, kv_heads, dim, vdim, taps)
    part, spec, p = delta_part(m, 96, dtype, seed=dim + 1)
    T = ops.DELTA_PIECES_FROM + 3 * ops.DELTA_PIECE + 5
    x = rnd(T + 80, 96, seed=6)
    want = P.plain_gated_delta(f64(x), p, "", m, EPS, {})
    short = P.plain_gated_delta(f64(x[:9]), p, "", m, EPS, {})
    size = ops.gated_delta_state_size(heads, kv_heads, dim, vdim, taps)
    slots = torch.randn(3, size, device=DEV)
    slots[:2].zero_()
    cache = LayerCache(state=slots)
    got = part.forward(dev(torch.cat([x[:5], x[:T]]), dtype), step_ctx([5, T], [0, 0], [1, 0]), cache)
    close(got[5:], want[:T], dtype, "pieces", bf16=5e-2)
    close(got[:5], short[:5], dtype, "short beside pieces", bf16=5e-2)
    more = part.forward(dev(torch.cat([x[5:9], x[T:T + 79]]), dtype), step_ctx([4, 79], [5, T], [1, 0]),
                        cache)
    close(more[4:], want[T:T + 79], dtype, "after pieces", bf16=5e-2)
    close(more[:4], short[5:], dtype, "short after pieces", bf16=5e-2)
    last = part.forward(dev(x[T + 79:], dtype), step_ctx([1], [T + 79], [0]), cache)
    close(last, want[T + 79:], dtype, "one more token", bf16=5e-2)


@pytest.mark.parametrize("forced", ["0", "1"])
def test_delta_rule_forms_agree(forced, monkeypatch):
    """Token by token and in pieces, whatever the portion's length: strong writes along nearly
    equal keys (the triangular system is then far from the identity), decays near one and near
    zero."""
    from mstar_b200 import ops

    monkeypatch.setenv("MSTAR_DELTA_PIECES", forced)
    g = torch.Generator().manual_seed(3)
    H, G, D, VD, T = 4, 2, 64, 24, 83
    base = torch.randn(G, D, generator=g)
    k = torch.nn.functional.normalize(base + 0.2 * torch.randn(T, G, D, generator=g), dim=-1)
    k = k * torch.where(torch.rand(T, G, 1, generator=g) < 0.3, -1.0, 1.0)
    q = torch.nn.functional.normalize(base + 0.5 * torch.randn(T, G, D, generator=g), dim=-1) * D ** -0.5
    v = torch.randn(T, H, VD, generator=g)
    beta = 0.9 + 0.1 * torch.rand(T, H, generator=g)
    decay = torch.where(torch.rand(T, H, generator=g) < 0.1, 1e-6, 0.999)
    state = torch.randn(2, H * VD * D, generator=g)
    want = np.zeros((T, H, VD))
    S1 = state[1].double().numpy().reshape(H, VD, D).transpose(0, 2, 1).copy()
    for h in range(H):
        want[:, h] = P.plain_delta_rule(f64(q[:, h // 2]), f64(k[:, h // 2]), f64(v[:, h]),
                                        f64(beta[:, h]), f64(decay[:, h]), S1[h])
    ctx = step_ctx([T], [0], [1])
    st = state.to(DEV)
    f = lambda t: t.reshape(T, -1).contiguous().to(DEV)
    got = ops.delta_scan(f(q), f(k), f(v), f(beta), f(decay), ctx.qo_indptr, ctx.slots, st, 1, H, G, D,
                         VD, 1, max_q_len=T)
    close(got, want.reshape(T, -1), "float32", "outputs")
    close(st[1], S1.transpose(0, 2, 1).reshape(-1), "float32", "state")
    assert torch.equal(st[0].cpu(), state[0])


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_state_is_carried_a_long_way(dtype):
    """Decays close to one: what the first tokens wrote is still read hundreds of tokens on, so
    a state lost or reset at a portion's edge shows."""
    from mstar_b200 import ops
    from mstar_b200.parts import LayerCache

    m = U.delta(2, 1, 64, 12, 2)
    part, spec, p = delta_part(m, 64, dtype, seed=21)
    part.dt_bias.fill_(-12.0)                               # decays of about 0.99999 a token
    p["dt_bias"] = np.full_like(p["dt_bias"], -12.0)
    part.w_in[-2 * 12 - 4:-2 * 12].zero_()                  # the rows of b and a: beta is a half
    p["b"], p["a"] = np.zeros_like(p["b"]), np.zeros_like(p["a"])
    T = 300
    x = rnd(T, 64, seed=6)
    want = P.plain_gated_delta(f64(x), p, "", m, EPS, {})
    late = P.plain_gated_delta(f64(x)[200:], p, "", m, EPS, {})
    assert np.abs(late[-1] - want[-1]).max() > 0.02 * np.abs(want[-1]).max()
    size = ops.gated_delta_state_size(2, 1, 64, 12, 2)
    cache = LayerCache(state=torch.zeros(1, size, device=DEV))
    outs, at = [], 0
    for n in [130, 2, 101] + [1] * 67:
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at], [0]), cache))
        at += n
    close(torch.cat(outs), want, dtype, "long carry", bf16=5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vdim", [4, 7, 64, 130, 256, 600])
def test_head_norm_and_silu_gate(dtype, vdim):
    """Both activations, a gate in the activations' type and one in float that is a column view."""
    from mstar_b200 import ops

    T, H = 6, 3
    o, w = rnd(T, H * vdim, seed=1).float(), rnd(vdim, seed=2).float()
    wide = rnd(T, H * vdim + 9, seed=3, scale=3.0)
    for act, gate in (("silu", wide.float().to(DEV)[:, 5:5 + H * vdim]),
                      ("sigmoid", dev(wide[:, :H * vdim], dtype))):
        got = ops.delta_finish(o.to(DEV), gate, w.to(DEV), H, vdim, EPS, TORCH[dtype], 1.0, act)
        g = gate.double().cpu().numpy()
        n = P.plain_over_rms(f64(o).reshape(T, H, vdim), EPS) * f64(w)
        want = n.reshape(T, -1) * (P.plain_silu(g) if act == "silu" else P.plain_sigmoid(g))
        close(got, want, dtype, (act, vdim), bf16=8e-3)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("experts,top,groups,scale", [
    (8, 3, (4, 2), 1.6), (6, 2, (2, 1), 0.8), (9, 4, (3, 2), 1.0), (5, 5, None, 2.0), (20, 4, (5, 3), 2.2),
    (64, 8, (32, 5), 1.5), (256, 8, (8, 4), 2.5), (1024, 16, (512, 9), 1.0), (40, 4, (1, 1), 0.5),
    (12, 3, (4, 1), 1.0), (1, 1, (1, 1), 3.0)])
def test_choice_of_experts(experts, top, groups, scale):
    """Groups of one and more experts, all groups kept and one, choice scores of both signs; the
    logits a column view of a wider product."""
    from mstar_b200 import ops

    T = 37
    g = torch.Generator().manual_seed(experts)
    z = 2.0 * torch.randn(T, experts + 3, generator=g)
    corr = (torch.randn(experts, generator=g) - 0.5) / experts
    named = dict(zip(("count", "keep"), groups)) if groups else None
    want_c, want_w = P.plain_route(f64(z)[:, :experts], f64(corr), top, named, scale)
    got_c, got_w = ops.route_topk(z.to(DEV)[:, :experts], top, softmax=True, renormalize=True,
                                  choice_bias=corr.to(DEV), groups=groups, renorm_eps=1e-20,
                                  weight_scale=scale)
    assert np.array_equal(got_c.cpu().numpy(), want_c)
    close(got_w, want_w, "float32", "weights")
    if groups and groups[1] < groups[0]:        # the groups decide
        free, _ = P.plain_route(f64(z)[:, :experts], f64(corr), top, None, scale)
        assert not np.array_equal(free, want_c)


def test_choice_of_experts_refuses_impossible_groups():
    from mstar_b200 import ops

    z = torch.randn(2, 8, device=DEV)
    for groups, top in (((3, 2), 2), ((4, 5), 2), ((4, 1), 3), ((4, 0), 1)):
        with pytest.raises(ops.KernelError):
            ops.route_topk(z, top, softmax=True, groups=groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 9, 100])
@pytest.mark.parametrize("width,mlp", [(96, U.moe(6, 2, 40, 56, (3, 2), 1.7)), (64, U.moe(5, 5, 24, 0, None, None)),
                                       (128, U.moe(40, 4, 64, 8, (8, 3), 2.5)), (52, U.moe(4, 1, 10, 14, (4, 1), 0.6))])
def test_experts_alone(dtype, rows, width, mlp):
    """The whole feed-forward, few rows and many (sorted by expert), sizes that are multiples of
    nothing.  Without the correction, the groups or the scale the output differs."""
    from mstar_b200.config.registry import config_from_dict
    from mstar_b200.parts import build_part

    cfg = U.config([U.layer("delta", U.delta(), mlp)], width=width)
    w = U.random_weights(cfg, 3)
    p, E = "l0.mlp.", mlp["router"]["experts"]
    params = {"router.weight": w[p + "router"], "router.correction": w[p + "correction"],
              "experts.gate_up.weight": torch.cat([w[f"{p}e{e}.{n}"] for e in range(E) for n in ("gate", "up")]),
              "experts.down.weight": torch.cat([w[f"{p}e{e}.down"] for e in range(E)])}
    if mlp.get("shared"):
        params["shared.gate_up.weight"] = torch.cat([w[p + "shared.gate"], w[p + "shared.up"]])
        params["shared.down.weight"] = w[p + "shared.down"]
    part = build_part("ffn", config_from_dict(cfg).layout().blocks[0].ffn,
                      {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    x = rnd(rows, width, seed=9)
    wn = U.as_numpy(w)
    want = P.plain_experts(f64(x), wn, p, mlp)
    top = np.abs(want).max()
    if rows > 9:
        others = [(dict(wn, **{p + "correction": 0 * wn[p + "correction"]}), mlp)]
        r = mlp["router"]
        if "scale" in r:
            others.append((wn, dict(mlp, router=dict(r, scale=1.0))))
        if r.get("groups"):
            others.append((wn, dict(mlp, router=dict(r, groups=None))))
        for w2, m2 in others:
            if not (m2["router"]["top"] == E and m2 is mlp):      # every expert is chosen anyway
                assert np.abs(P.plain_experts(f64(x), w2, p, m2) - want).max() > 0.01 * top or (
                    m2["router"].get("groups") is None and r["groups"]["keep"] >= r["top"])
    got = part.forward(dev(x, dtype), None)
    if dtype == "float32":
        close(got, want, dtype, ("experts", rows))
        return
    # a close call between two experts may turn the other way: that row and nothing else
    err = (got.double().cpu() - torch.from_numpy(want)).abs().amax(1) / top
    assert int((err > 3e-2).sum()) <= max(1, rows // 20), err


# ------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def mixed_model():
    weights = U.random_weights(U.MIXED, seed=3)
    reqs = {"a": U.tokens(U.MIXED, 61, 1), "b": U.tokens(U.MIXED, 24, 2),
            "c": [52], "d": U.tokens(U.MIXED, 37, 4),
            "e": U.tokens(U.MIXED, 90, 5)}
    want = {r: U.plain_logits(U.MIXED, weights, t) for r, t in reqs.items()}
    models = {}

    def get(dtype):
        if dtype not in models:
            models[dtype] = U.load(U.MIXED, weights, dtype)
        return models[dtype]

    return weights, reqs, want, get


def check_all(got, want, dtype, what):
    for r in want:
        U.assert_close(got[r], want[r], dtype, (what, r))


def stepper_for(model, **kw):
    from mstar_b200.engine.step import make_stepper
    kw.setdefault("page_size", 4)
    kw.setdefault("num_pages", 64)
    kw.setdefault("num_slots", 3)
    return make_stepper(model, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(mixed_model, dtype):
    """The sum of the residual's copies after each layer against the plain model's: a fault
    shows in the layer it enters."""
    from mstar_b200.engine.step import StepEntry
    from mstar_b200.parts import block as B

    weights, reqs, _, get = mixed_model
    want = []
    P.plain_forward(reqs["b"], U.as_numpy(weights), U.MIXED, layer_outputs=want)
    seen = []
    orig = B.HyperBlock.forward

    def recording(self, stream, ctx, cache):
        orig(self, stream, ctx, cache)
        rows = torch.arange(stream.copies.x.shape[0], dtype=torch.int32, device=DEV)
        seen.append(stream.copies.gather(rows).cpu())

    B.HyperBlock.forward = recording
    try:
        st = stepper_for(get(dtype))
        st.add_request("b")
        st.step([StepEntry("b", reqs["b"], [0])])
    finally:
        B.HyperBlock.forward = orig
    assert len(seen) == len(want) == len(U.MIXED["layers"])
    for i, (g, w) in enumerate(zip(seen, want)):
        close(g, w, dtype, ("layer", i), f32=2e-5, bf16=5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_and_token_by_token(mixed_model, dtype):
    """Each request alone: its prompt in one step, and every token as a step of its own (with
    and without captured graphs); the three agree with the plain model."""
    _, reqs, want, get = mixed_model
    model = get(dtype)
    whole = U.run_schedule(stepper_for(model), reqs, [[(r, len(t))] for r, t in reqs.items()])
    check_all(whole, want, dtype, "whole")
    for graphs in (False, True):
        st = stepper_for(model, cuda_graphs=graphs)
        single = U.run_schedule(st, reqs, [[(r, 1)] for r, t in reqs.items() for _ in t])
        check_all(single, want, dtype, f"token by token, graphs={graphs}")
        assert (st.graph_replays > 0) == graphs


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(mixed_model, dtype):
    """Prompts cut into portions of changing size, down to two tokens, ends decoded one by one:
    cuts fall inside pages, inside windows, inside the convolutions' taps and inside the scan's
    pieces."""
    _, reqs, want, get = mixed_model
    schedule = []
    for r, t in reqs.items():
        left, sizes, k = len(t), (2, 17, 3, 2, 16, 5, 33, 2), 0
        while left > 6:
            n = min(sizes[k % len(sizes)], left - 6)
            schedule.append([(r, n)])
            left -= n
            k += 1
        schedule += [[(r, 1)]] * left
    got = U.run_schedule(stepper_for(get(dtype)), reqs, schedule)
    check_all(got, want, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_reuse_pages_and_slots(mixed_model, dtype):
    """Up to three live requests in a batch, portions beside single tokens, a request sitting
    out a step; five requests go through three slots and a pool of pages that holds less than
    all of them, so that slots and pages are used again; each agrees with itself alone."""
    _, reqs, want, get = mixed_model
    schedule = [
        [("a", 2), ("b", 3), ("c", 1)],               # c ends here: its slot goes to d
        [("a", 29), ("b", 1), ("d", 16)],
        [("a", 1), ("d", 2)],
        [("a", 1), ("b", 18), ("d", 1)],
        [("b", 1), ("a", 20), ("d", 17)],
        [("b", 1), ("a", 1), ("d", 1)],               # b and d end
        [("a", 1), ("e", 2)],
        [("a", 6), ("e", 64)],                        # a ends
        [("e", 1)], [("e", 21)], [("e", 1)], [("e", 1)],
    ]
    st = stepper_for(get(dtype), num_pages=40, num_slots=3)
    got = U.run_schedule(st, reqs, schedule)
    check_all(got, want, dtype, "mixed")
    assert st.manager.num_requests() == 0 and st.manager.check() == 0
    assert st.manager.free_slots() == 3


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_behind_a_window_are_given_back(dtype):
    """A sequence far longer than the pool: only the pages a window can reach are held, so the
    pool is gone through several times; and a model of delta-rule layers alone, which holds no
    page at all."""
    for layers in ([U.layer("attention", U.attention(2, 1, 16, 16, window=24), None),
                    U.layer("delta", U.delta(2, 1, 16, 16, 4), U.moe(4, 2, 16, 0, (2, 1)))],
                   [U.layer("delta", U.delta(2, 2, 32, 16, 2), U.moe(4, 2, 16, 8, (2, 2)))] * 2):
        cfg = U.config(layers, width=48, vocab=61)
        w = U.random_weights(cfg, 8)
        toks = U.tokens(cfg, 200, 3)
        want = U.plain_logits(cfg, w, toks)
        st = stepper_for(U.load(cfg, w, dtype), page_size=4, num_pages=16, num_slots=1)
        sizes, schedule = (9, 2, 31, 1, 1, 17), []
        left = len(toks)
        while left:
            n = min(sizes[len(schedule) % 6], left)
            schedule.append([("r", n)])
            left -= n
        got = U.run_schedule(st, {"r": toks}, schedule)
        U.assert_close(got["r"], want, dtype, "pages of old windows")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """A short prompt and 400 decoded tokens through captured graphs: windows that pass over
    decoded tokens, the delta rule's matrix and the convolutions' rows carried 400 steps, values
    blended in a captured step."""
    cfg = U.config([U.layer("attention", U.attention(2, 1, 16, 24, window=90), U.moe(8, 2, 24, 16, (4, 2))),
                    U.layer("delta", U.delta(2, 1, 24, 8, 4), U.moe(4, 2, 32, 0, None)),
                    U.layer("attention", U.attention(4, 1, 24, 24, window=None, rot_dims=24), None)],
                   width=64, vocab=97, streams=2)
    weights = U.random_weights(cfg, 11)
    toks = U.tokens(cfg, 410, 12)
    want = U.plain_logits(cfg, weights, toks)
    st = stepper_for(U.load(cfg, weights, dtype), page_size=4, num_pages=104, num_slots=1)
    got = U.run_schedule(st, {"r": toks}, [[("r", 10)]] + [[("r", 1)]] * 400)
    U.assert_close(got["r"], want, dtype, "long decoding")
    assert st.graph_replays == 400


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_that_are_one_or_equal(dtype):
    """One head, one tap, one expert, one group, one copy of the residual, a window of one
    position, keys as wide as values, every expert chosen, no scale, no caps; and sizes that are
    multiples of nothing (a width of 100, heads of 12 and 10, a vocabulary of 53)."""
    for layers, kw in (
            ([U.layer("attention", U.attention(1, 1, 16, 16, scale=1.0, softcap=1.0, window=1, rot_dims=16),
                      U.moe(1, 1, 16, 8, (1, 1), 1.0)),
              U.layer("delta", U.delta(1, 1, 8, 8, 1), None)],
             dict(width=32, vocab=50, streams=1, logit_scale=1.0, logit_softcap=1.0)),
            ([U.layer("delta", U.delta(2, 2, 8, 8, 2), U.moe(2, 2, 8, 8, (2, 2), None)),
              U.layer("attention", U.attention(2, 2, 8, 8, softcap=None, window=None, rot_dims=8),
                      U.moe(4, 2, 8, 0, (2, 1))),
              U.layer("attention", U.attention(2, 2, 8, 8, window=4, rot_dims=0, v_mix=None), None)],
             dict(width=32, vocab=50, streams=4, logit_scale=None, logit_softcap=None)),
            ([U.layer("attention", U.attention(3, 1, 12, 10, rot_dims=6, window=19), U.moe(6, 3, 18, 10, (3, 2))),
              U.layer("delta", U.delta(5, 1, 12, 10, 3), U.moe(3, 2, 20, 12, None)),
              U.layer("attention", U.attention(2, 1, 10, 10, rot_dims=10, window=5), U.moe(5, 1, 18, 0, (5, 2)))],
             dict(width=100, vocab=53, streams=2))):
        cfg = U.config(layers, **kw)
        weights = U.random_weights(cfg, 21)
        reqs = {"x": U.tokens(cfg, 33, 1), "y": U.tokens(cfg, 12, 2)}
        want = {r: U.plain_logits(cfg, weights, t) for r, t in reqs.items()}
        st = stepper_for(U.load(cfg, weights, dtype))
        got = U.run_schedule(st, reqs, [[("x", 7), ("y", 2)], [("x", 1), ("y", 10)],
                                        [("x", 25)]])
        check_all(got, want, dtype, "small sizes")


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(mixed_model, dtype, tmp_path):
    """LLM.generate with its scheduler (portions under a small token budget, several requests
    at once) picks the tokens the plain model picks; in bfloat16 a pick may differ only where
    the plain model's own margin is small, but for one token in twenty."""
    import json

    from safetensors.torch import save_file

    from mstar_b200 import LLM, SamplingParams

    weights, reqs, _, _ = mixed_model
    (tmp_path / "config.json").write_text(json.dumps(U.MIXED))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(tmp_path / "model.safetensors"))
    llm = LLM(str(tmp_path), dtype=dtype, page_size=8, max_num_pages=48,
              max_num_batched_tokens=16, max_concurrent_requests=3)
    prompts = [reqs["a"][:40], reqs["b"][:5], reqs["d"][:19], reqs["e"][:2]]
    n_new = 12
    results = llm.generate(prompts, SamplingParams(temperature=0.0, ignore_eos=True,
                                                   max_output_tokens=n_new))
    w = U.as_numpy(weights)
    far_off = 0
    for prompt, res in zip(prompts, results):
        assert len(res.token_ids) == n_new
        states = [{} for _ in U.MIXED["layers"]]
        logits = P.plain_forward(list(prompt), w, U.MIXED, states)[-1]
        for tok in res.token_ids:
            best = int(np.argmax(logits))
            margin = float(logits[best] - logits[tok])
            assert tok == best or dtype == "bfloat16", (tok, best, margin)
            far_off += tok != best and margin >= 0.25
            logits = P.plain_forward([tok], w, U.MIXED, states)[-1]
    assert far_off <= len(prompts) * n_new // 20, far_off


def test_trace_replay_of_a_model_folder(mixed_model, tmp_path):
    """bin/trace_run on a folder of this design: the registry picks the model by config.json."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    from safetensors.torch import save_file

    weights, reqs, want, _ = mixed_model
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(U.MIXED))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:50], "want": [3, 49]},
                                     {"id": "b", "tokens": reqs["b"][:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": reqs["b"][2:], "want": [0]},
                                     {"id": "a", "tokens": reqs["a"][50:51], "want": [0]}],
              "end": ["b"]}]
    exe = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, str(exe), "--model", str(folder), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "128"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                          capture_output=True, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1))
    got1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1))
    U.assert_close(got0, want["a"][[3, 49]], "float32", "trace step 0")
    U.assert_close(got1, torch.stack([want["b"][2], want["a"][50]]), "float32", "trace step 1")
