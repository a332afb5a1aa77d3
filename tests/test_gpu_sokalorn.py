"""The Sokalorn decoder in the engine against the plain implementation
(tests/plain_sokalorn.py): each mechanism alone, then whole models through the step function, the
cache and state manager, the scheduler and the entry point, under every kind of schedule."""
import numpy as np
import pytest
import torch

import plain_sokalorn as P
import sokalorn_util as U

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


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 100, 1000, 4104, 5000, 9000])
def test_side_step(dtype, width):
    """Sum, norm and token shift as one kernel: nothing pending, one output, two normed branches
    with a feed-forward's output; portions of several entries beside single tokens, entries
    longer than a block's run of tokens; the slot's row is read and moved on."""
    from mstar_b200 import ops

    shift, nw = rnd(width, seed=2), (rnd(width, seed=3, scale=0.2).float() + 1.0).to(torch.bfloat16)
    w0, w1 = rnd(width, seed=4), rnd(width, seed=5)
    slots = torch.randn(4, width + 8, device=DEV)
    prev0 = slots.clone()
    view = slots[:, 8:]
    # enough tokens that a block takes a run of them
    q_lens, order = [1, 2600 if width <= 1000 else 700, 3, 1], [2, 0, 3, 1]
    T = sum(q_lens)
    ctx = step_ctx(q_lens, [5, 9, 0, 2], order)
    resid = rnd(T, width, seed=6).float()
    y0, y1, f = (rnd(T, width, seed=s, scale=2.0) for s in (7, 8, 9))
    x0 = resid.double().numpy()
    bound = 8e-3
    for case in ("none", "one", "float", "branches"):
        slots.copy_(prev0)
        pending, x = None, x0
        if case == "one":
            pending, x = ops.SideBySideOutput(dev(y0, dtype)), x0 + y0.double().numpy()
        elif case == "float":
            pending, x = y0.float().to(DEV), x0 + y0.double().numpy()
        elif case == "branches":
            mean = ops.MeanOfNorms([dev(y0, dtype), dev(y1, dtype)],
                                   [w0.float().to(DEV), w1.float().to(DEV)], EPS)
            pending = ops.SideBySideOutput(mean, dev(f, dtype))
            x = x0 + f.double().numpy() + 0.5 * (
                P.plain_rms_norm(y0.double().numpy(), w0.double().numpy(), EPS)
                + P.plain_rms_norm(y1.double().numpy(), w1.double().numpy(), EPS))
        h = resid.to(DEV)
        got_x, got_n, got_s = ops.side_step(
            h, pending, act_dtype=TORCH[dtype], norm_weight=dev(nw, dtype), eps=EPS, normed=True,
            shift=dev(shift, dtype), prev=view, ctx=ctx)
        assert torch.equal(h.cpu(), resid), "the residual read is left as it is"
        n = P.plain_rms_norm(x, nw.double().numpy(), EPS)
        want, at = [], 0
        for e, (q, s) in enumerate(zip(q_lens, order)):
            st = {"p": prev0[s, 8:].double().cpu().numpy()}
            want.append(P.plain_mix(n[at:at + q], P.plain_previous(n[at:at + q], st, "p"),
                                    shift.double().numpy()))
            close(view[s], st["p"], "float32", (case, "slot", e))
            at += q
        close(got_x, x, "float32", (case, "residual"))
        close(got_n, n, dtype, (case, "normed"), bf16=bound)
        close(got_s, np.concatenate(want), dtype, (case, "shifted"), bf16=bound)
        assert torch.equal(slots[:, :8], prev0[:, :8])            # the mixer's part of the slot
        rows = torch.tensor([T - 1, 0, 3, 3], dtype=torch.int32, device=DEV)
        close(ops.side_step(h, pending, rows=rows), x[[T - 1, 0, 3, 3]], "float32", (case, "rows"))
        close(ops.side_step(h, pending, act_dtype=TORCH[dtype], raw=True), x, dtype, (case, "raw"),
              bf16=bound)


def left_part(m, width, dtype, seed, sharp=3.0):
    from mstar_b200.parts import build_part

    cfg = U.config([U.parallel(l=m)], width=width)
    w = U.random_weights(cfg, seed, sharp=sharp)
    p = "l0.mix.left."
    spec = U.shaped(cfg, w).layout().blocks[0].mixer.branches[0]
    params = {"qkv.weight": torch.cat([w[p + n] for n in "qkvg"]), "score_bias": w[p + "pb"],
              "o.weight": w[p + "o"]}
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


def plain_left(x, p, m):
    return P.plain_left(x, np.arange(x.shape[0]), p, "", m, {})


ATTENTIONS = [
    (U.left(4, 2, 24, 40, scale=0.3, softcap=5.0, chunk=11), 4),
    (U.left(3, 3, 16, 8, scale=0.4, softcap=50.0, chunk=64, rot_dims=16, factor=1.0), 8),
    (U.left(34, 1, 16, 24, scale=0.4, softcap=1.0, chunk=33, rot_dims=2), 16),
    (U.left(2, 1, 160, 256, scale=0.06, softcap=30.0, chunk=1, rot_dims=160), 8),
    (U.left(2, 2, 12, 10, scale=0.5, softcap=4.0, chunk=5, rot_dims=4, base=10.0), 4),
    (U.left(4, 1, 64, 64, scale=0.125, softcap=None, chunk=None, rot_dims=32, factor=8.0), 16),
    (U.left(6, 2, 128, 128, scale=0.09, softcap=20.0, chunk=48, rot_dims=128, base=70000.0), 16),
    (U.left(5, 5, 96, 72, scale=0.1, softcap=9.0, chunk=200, rot_dims=24), 16),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", ATTENTIONS)
def test_attention_alone(dtype, m, page):
    """The chunked attention with sigmoid weights alone, scores spread over the whole sigmoid; a
    prompt portion, portions of two, single tokens, pages scattered over the pool; with the
    chunk, the bias or the soft cap left out the output differs."""
    part, spec, p = left_part(m, 96, dtype, seed=7)
    T = 70
    x = rnd(T, 96, seed=8)
    xn = x.double().numpy()
    want = plain_left(xn, p, m)
    top = np.abs(want).max()
    assert np.abs(plain_left(xn, dict(p, pb=p["pb"] + 1.0), m) - want).max() > 0.05 * top
    if m.get("mask") and m["mask"]["size"] < T:
        assert np.abs(plain_left(xn, p, dict(m, mask=None)) - want).max() > 0.05 * top
    if m.get("softcap", 99.0) < 6.0:
        assert np.abs(plain_left(xn, p, dict(m, softcap=None)) - want).max() > 0.02 * top
    cache = paged_cache(spec, T, page, dtype)
    outs, at = [], 0
    for n in (23, 2, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 29, 3, 2):
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
        at += n
    assert at == T
    close(torch.cat(outs), want, dtype, ("attention", m), bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,heads,kv_heads", [(1100, 8, 2), (300, 8, 2), (37, 8, 2), (2000, 16, 4), (None, 8, 2)])
def test_long_prompts(dtype, chunk, heads, kv_heads):
    """A prompt of two thousand tokens in one portion and as a short portion before a long one:
    the order in which row tiles are taken, and the two shares of a long chunk's keys."""
    m = U.left(heads, kv_heads, 16, 16, scale=0.25, softcap=5.0, chunk=chunk, rot_dims=8, base=5000.0)
    part, spec, p = left_part(m, 64, dtype, seed=7)
    T = 2100
    x = rnd(T, 64, seed=8)
    want = plain_left(x.double().numpy(), p, m)
    for cuts in ([T], [37, T - 37]):
        cache = paged_cache(spec, T, 16, dtype)
        outs, at = [], 0
        for n in cuts:
            outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
            at += n
        err = (torch.cat(outs).double().cpu() - torch.from_numpy(want)).abs().amax(1)
        err /= torch.from_numpy(want).abs().amax(1)
        assert float(err.max()) < (1e-4 if dtype == "float32" else 5e-2), (cuts, int(err.argmax()), float(err.max()))


def marked_inputs(p, m, width, T, marked, queries, gain=6.0):
    """Inputs in which the key at ``marked`` stands out for the ``queries``: the query tokens lie
    along a direction d, the marked token along the direction whose key equals the query of d (a
    solution of W_k d' = W_q d; no rotation), so that its weight is near one while the others',
    under a bias far below zero, are small."""
    x = rnd(T, width, seed=4, scale=0.3)
    d = rnd(width, seed=5).double().numpy()
    d /= np.linalg.norm(d)
    target = p["q"][:m["dim"]] @ d                             # the first query head
    d_key = np.linalg.lstsq(p["k"][:m["dim"]], target, rcond=None)[0]
    d_key *= np.linalg.norm(target) / np.linalg.norm(p["k"][:m["dim"]] @ d_key)
    for t in np.atleast_1d(marked):
        x[t] = torch.from_numpy(gain * d_key).to(torch.bfloat16)
    for q in queries:
        x[q] += torch.from_numpy(gain * d).to(torch.bfloat16)
    return x


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,page", [(96, 16), (97, 16), (64, 4), (130, 8)])
def test_edges_of_a_chunk(dtype, chunk, page):
    """A key that stands out, just inside a chunk (its first position) and just outside (the last
    of the chunk before): the queries are the chunk's last position, far from it, and the next
    chunk's first, in one prompt, in portions cut right at and around the edge, and decoded.
    Inside, the output hangs on that key; outside, not at all."""
    m = U.left(2, 1, 32, 32, scale=1.0, softcap=30.0, chunk=chunk, rot_dims=0)
    T = 2 * chunk + 3
    part, spec, p = left_part(m, 64, dtype, seed=3, sharp=1.0)
    part.score_bias.fill_(-9.0)
    p["pb"] = np.full_like(p["pb"], -9.0)
    for marked, near, far in ((chunk, 2 * chunk - 1, 2 * chunk), (chunk - 1, chunk - 1, chunk + 1)):
        x = marked_inputs(p, m, 64, T, marked, [q for q in (2 * chunk - 1, 2 * chunk, chunk + 1) if q != marked])
        xn = x.double().numpy()
        want = plain_left(xn, p, m)
        hidden = xn.copy()
        hidden[marked] = 0.0
        blind = plain_left(hidden, p, m)
        if marked == chunk:
            assert np.abs(blind[near] - want[near]).max() > 0.3 * np.abs(want[near]).max()
        assert np.abs(blind[far] - want[far]).max() < 1e-9
        for cuts in ([T], [chunk, chunk, 3], [chunk - 1, 2, chunk - 1, 3], [chunk + 1, chunk - 3]):
            cache = paged_cache(spec, T, page, dtype, seed=len(cuts))
            outs, at = [], 0
            for n in cuts + [1] * (T - sum(cuts)):
                outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at]), cache))
                at += n
            got = torch.cat(outs)
            # row by row: a stray key would drown in the largest rows
            err = ((got.double().cpu() - torch.from_numpy(want)).abs().amax(1)
                   / torch.from_numpy(want).abs().amax(1))
            assert float(err.max()) < (1e-4 if dtype == "float32" else 8e-2), (marked, cuts, int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("marked,page", [(0, 16), (15, 16), (16, 16), (3, 4), (257, 8)])
def test_one_far_key_stands_out(dtype, marked, page):
    """One key hundreds of tokens back (the first token, the last of a page, the first of the
    next) in a long chunk: a wrong page or a lost key changes the output by that key's whole
    value.  The query in a prompt portion and decoded alone."""
    m = U.left(2, 1, 32, 32, scale=1.0, softcap=40.0, chunk=400, rot_dims=0)
    T, queries = 330, [300, 329]
    part, spec, p = left_part(m, 64, dtype, seed=3, sharp=1.0)
    part.score_bias.fill_(-10.0)
    p["pb"] = np.full_like(p["pb"], -10.0)
    x = marked_inputs(p, m, 64, T, marked, queries)
    xn = x.double().numpy()
    want = plain_left(xn, p, m)
    hidden = xn.copy()
    hidden[marked] = 0.0
    blind = plain_left(hidden, p, m)
    for q in queries:             # how much hangs on the one key
        assert np.abs(blind[q] - want[q]).max() > 0.3 * np.abs(want[q]).max(), (marked, q)
    for first in (T, 290):                    # one prompt; a prompt and decoded tokens
        cache = paged_cache(spec, T, page, dtype, seed=first)
        outs = [part.forward(dev(x[:first], dtype), step_ctx([first], [0]), cache)]
        outs += [part.forward(dev(x[t:t + 1], dtype), step_ctx([1], [t]), cache)
                 for t in range(first, T)]
        close(torch.cat(outs), want, dtype, ("far key", marked, first), bf16=4e-2)


def right_part(m, width, dtype, seed, rank=U.RANK):
    from mstar_b200.parts import build_part

    cfg = U.config([U.parallel(r=m)], width=width)
    w = U.random_weights(cfg, seed, rank=rank)
    p = "l0.mix.right."
    spec = U.shaped(cfg, w).layout().blocks[0].mixer.branches[1]
    params = {"in.weight": torch.cat([w[p + n] for n in ("r", "k", "v", "g", "w1")]),
              "mu": torch.cat([w[p + "mu." + n] for n in "rkvgw"]), "w2.weight": w[p + "w2"],
              "w0": w[p + "w0"], "u": w[p + "u"], "norm.weight": w[p + "norm"], "o.weight": w[p + "o"]}
    part = build_part("mixer", spec, {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    return part, U.sub(w, p)


def ssd_part(m, width, dtype, seed):
    from mstar_b200.parts import build_part

    cfg = U.config([U.ssd(m)], width=width)
    w = U.random_weights(cfg, seed)
    p = "l0.mix."
    spec = U.shaped(cfg, w).layout().blocks[0].mixer
    params = {"in.weight": w[p + "in"], "conv.weight": w[p + "conv"], "conv.bias": w[p + "conv.b"],
              "dt_bias": w[p + "dt_bias"], "A_log": w[p + "A_log"], "D": w[p + "D"],
              "norm.weight": w[p + "norm"], "o.weight": w[p + "o"]}
    part = build_part("mixer", spec, {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    return part, U.sub(w, p)


def recurrent_alone(part, plain, width, dtype, what, T=45):
    """A sequence cut into a portion, a two-token portion, single tokens and more portions, in a
    slot among others that hold other requests' states; then two sequences in one batch; then a
    portion long enough to be walked in pieces beside a short one, and what follows it."""
    from mstar_b200.parts import LayerCache

    size = part.cache_need(part.spec).state.shape[0]
    long = 420
    x = rnd(long + 9, width, seed=5)
    want = plain(x.double().numpy())
    slots = torch.randn(4, size, device=DEV)               # leftovers of earlier requests
    slots[2].zero_()
    cache = LayerCache(state=slots)
    outs, at = [], 0
    for n in (19, 2, 1, 1, 1, 17, 4):
        outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at], [2]), cache))
        at += n
    assert at == T
    close(torch.cat(outs), want[:T], dtype, (what, "portions"), bf16=4e-2)
    slots2 = torch.zeros(4, size, device=DEV)
    cache2 = LayerCache(state=slots2)
    both = part.forward(dev(torch.cat([x[:9], x[:30]]), dtype), step_ctx([9, 30], [0, 0], [3, 0]), cache2)
    close(both[:9], want[:9], dtype, (what, "first of two"), bf16=4e-2)
    close(both[9:], want[:30], dtype, (what, "second of two"), bf16=4e-2)
    assert float(slots2[1].abs().max()) == 0.0 and float(slots2[3].abs().max()) > 0.0
    slots2[:2].zero_()
    got = part.forward(dev(torch.cat([x[:5], x[:long]]), dtype), step_ctx([5, long], [0, 0], [1, 0]), cache2)
    close(got[5:], want[:long], dtype, (what, "long portion"), bf16=4e-2)
    close(got[:5], want[:5], dtype, (what, "short beside long"), bf16=4e-2)
    more = part.forward(dev(torch.cat([x[5:6], x[long:long + 8]]), dtype),
                        step_ctx([1, 8], [5, long], [1, 0]), cache2)
    close(more[1:], want[long:long + 8], dtype, (what, "after long"), bf16=4e-2)
    close(more[:1], want[5:6], dtype, (what, "short after"), bf16=4e-2)
    last = part.forward(dev(x[long + 8:], dtype), step_ctx([1], [long + 8], [0]), cache2)
    close(last, want[long + 8:], dtype, (what, "one more token"), bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,width,rank", [(3, 20, 96, 5), (1, 64, 64, 16), (2, 48, 128, 8),
                                                  (9, 8, 100, 1), (2, 130, 64, 3), (1, 300, 96, 40)])
def test_time_mixing_alone(dtype, heads, dim, width, rank):
    part, p = right_part(U.right(heads, dim), width, dtype, seed=dim, rank=rank)
    m = {"heads": heads, "dim": dim}
    recurrent_alone(part, lambda x: P.plain_right(x, p, "", m, EPS, {}), width, dtype, "time mixing")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,width", [(U.mamba2(4, 20, 24, 2, 4, 2), 96), (U.mamba2(1, 8, 8, 1, 1, 1), 64),
                                     (U.mamba2(6, 64, 128, 3, 3, 4), 128), (U.mamba2(5, 10, 7, 5, 2, 5), 72),
                                     (U.mamba2(2, 130, 200, 1, 5, 1), 64), (U.mamba2(4, 32, 512, 4, 4, 8), 64),
                                     (U.mamba2(16, 64, 32, 2, 4, 1), 96)])
def test_state_space_alone(dtype, m, width):
    part, p = ssd_part(m, width, dtype, seed=m["state"])
    recurrent_alone(part, lambda x: P.plain_mamba2(x, p, "", m, EPS, {}), width, dtype, "state space")


@pytest.mark.parametrize("piece", ["0", "16", "48", "1024"])
def test_scan_in_pieces_of_any_size(piece, monkeypatch):
    """The scan walked whole, in pieces of one chunk, in pieces that leave a short last one, and
    in pieces longer than the entry: the same outputs and the same state."""
    from mstar_b200.parts import LayerCache

    monkeypatch.setenv("MSTAR_LINEAR_PIECE", piece)
    for part, plain, width in (
            (lambda q: (q[0], lambda x: P.plain_right(x, q[1], "", U.right(2, 40), EPS, {}), 64))(
                right_part(U.right(2, 40), 64, "float32", 1)),
            (lambda q: (q[0], lambda x: P.plain_mamba2(x, q[1], "", U.mamba2(2, 24, 40, 1, 3, 1), EPS, {}), 64))(
                ssd_part(U.mamba2(2, 24, 40, 1, 3, 1), 64, "float32", 2))):
        x = rnd(140, width, seed=3)
        want = plain(x.double().numpy())
        cache = LayerCache(state=torch.zeros(2, part.cache_need(part.spec).state.shape[0], device=DEV))
        outs, at = [], 0
        for n in (100, 2, 33, 5):
            outs.append(part.forward(dev(x[at:at + n], "float32"), step_ctx([n], [at], [1]), cache))
            at += n
        close(torch.cat(outs), want, "float32", ("pieces", piece))


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_are_carried_a_long_way(dtype):
    """Decays close to one: what the first tokens wrote is still read hundreds of tokens on, so a
    state lost or reset at a portion's edge shows.  The plain model without its first tokens
    gives another output at the end."""
    from mstar_b200.parts import LayerCache

    rp, p = right_part(U.right(2, 32), 64, dtype, seed=21)
    rp.w0.fill_(-9.0)
    p["w0"] = np.full_like(p["w0"], -9.0)
    rp.w2.zero_()
    p["w2"] = np.zeros_like(p["w2"])
    m = U.mamba2(2, 16, 32, 1, 4, 1)
    sp, q = ssd_part(m, 64, dtype, seed=22)
    sp.a_exp.fill_(1e-3)
    q["A_log"] = np.full_like(q["A_log"], np.log(1e-3))
    T = 300
    x = rnd(T, 64, seed=6)
    xn = x.double().numpy()
    for part, plain in ((rp, lambda v: P.plain_right(v, p, "", U.right(2, 32), EPS, {})),
                        (sp, lambda v: P.plain_mamba2(v, q, "", m, EPS, {}))):
        want, late = plain(xn), plain(xn[200:])
        assert np.abs(late[-1] - want[-1]).max() > 0.05 * np.abs(want[-1]).max()
        cache = LayerCache(state=torch.zeros(1, part.cache_need(part.spec).state.shape[0], device=DEV))
        outs, at = [], 0
        for n in [130, 2, 101] + [1] * 67:
            outs.append(part.forward(dev(x[at:at + n], dtype), step_ctx([n], [at], [0]), cache))
            at += n
        close(torch.cat(outs), want, dtype, "long carry", bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 9, 100])
@pytest.mark.parametrize("width,mlp", [(96, U.moe(6, 2, 40, 1.2, 56, 0.8)), (64, U.moe(5, 5, 24, 0.3, 0)),
                                       (128, U.moe(40, 4, 64, 3.0, 8, 0.2)), (52, U.moe(4, 1, 10, 1.0, 14, 2.0))])
def test_clamped_experts(dtype, rows, width, mlp):
    """Experts whose gate and up values are clamped, a shared expert with clamps of its own and a
    gate a token; few rows and many (sorted by expert).  Without the clamps, with the shared
    expert's clamp for the others, or without its gate the output differs."""
    from mstar_b200.parts import build_part

    cfg = U.config([U.ssd(mlp=mlp)], width=width)
    w = U.random_weights(cfg, 3)
    lay = U.shaped(cfg, w).layout()
    p, E = "l0.mlp.", mlp["router"]["experts"]
    params = {"router.weight": torch.cat([w[p + "router"]] + ([w[p + "shared.sg"]] if mlp.get("shared") else [])),
              "experts.gate_up.weight": torch.cat([w[f"{p}e{e}.{n}"] for e in range(E) for n in ("gate", "up")]),
              "experts.down.weight": torch.cat([w[f"{p}e{e}.down"] for e in range(E)])}
    if mlp.get("shared"):
        params["shared.gate_up.weight"] = torch.cat([w[p + "shared.gate"], w[p + "shared.up"]])
        params["shared.down.weight"] = w[p + "shared.down"]
    part = build_part("ffn", lay.blocks[0].ffn, {k: dev(v, dtype) for k, v in params.items()}, runtime(dtype))
    x = rnd(rows, width, seed=9)
    xn, wn = x.double().numpy(), U.as_numpy(w)
    want = P.plain_moe(xn, wn, p, mlp)
    top = np.abs(want).max()
    if rows > 1:
        loose = dict(mlp, expert=dict(mlp["expert"], limit=1e9))
        assert np.abs(P.plain_moe(xn, wn, p, loose) - want).max() > 0.01 * top
        if mlp.get("shared"):
            other = dict(mlp, shared=dict(mlp["shared"], limit=mlp["expert"]["limit"]))
            assert np.abs(P.plain_moe(xn, wn, p, other) - want).max() > 0.01 * top
            open_gate = dict(wn, **{p + "shared.sg": np.zeros_like(wn[p + "shared.sg"])})
            assert np.abs(P.plain_moe(xn, open_gate, p, mlp) - want).max() > 0.01 * top
    got = part.forward(dev(x, dtype), None)
    if dtype == "float32":
        close(got, want, dtype, ("experts", rows))
        return
    # a close call between two experts may turn the other way: that row and nothing else
    err = (got.double().cpu() - torch.from_numpy(want)).abs().amax(1) / top
    assert int((err > 3e-2).sum()) <= max(1, rows // 20), err


@pytest.mark.parametrize("rows", [3, 16, 200, 1000])
def test_clamped_gate_of_every_product_kernel(rows):
    """The clamped activation in the epilogues of the weight-streaming and the tcgen05 kernels and
    as a kernel of its own after the library's product."""
    from mstar_b200 import ops

    width, ff = 256, 20480 if rows == 1000 else 192          # wide enough for the tcgen05 tiles
    x, w = rnd(rows, width, seed=1), rnd(2 * ff, width, seed=2, scale=0.12)
    got = ops.gated_up(x.to(DEV), w.to(DEV), kind="clamped_swish", limit=0.9, alpha=1.3)
    gu = x.to(DEV).float() @ w.to(DEV).float().t()
    g, u = gu[:, :ff].clamp(max=0.9), gu[:, ff:].clamp(-0.9, 0.9)
    want = g * torch.sigmoid(1.3 * g) * (u + 1)
    assert float((got.float() - want).abs().max() / want.abs().max()) < 2e-2
    if rows == 1000:
        assert ops.tcgen05_tile(rows, 2 * ff) is not None


@pytest.mark.parametrize("tokens", [1, 7, 16, 40])
@pytest.mark.parametrize("rows,rank,width", [(64, 16, 128), (96, 5, 256), (1024, 64, 1024), (60, 3, 96), (20, 9, 52)])
def test_products_with_planes(tokens, rows, rank, width):
    """Row groups of one matrix against inputs of their own: one launch for few rows."""
    from mstar_b200 import ops

    x, w = rnd(5, tokens, width, seed=1), rnd(4 * rows + rank, width, seed=2, scale=width ** -0.5)
    head, tail = ops.linear_planes(x.to(DEV), w.to(DEV), rows)
    assert tuple(head.shape) == (tokens, 4 * rows) and tuple(tail.shape) == (tokens, rank)
    for s in range(4):
        want = x[s].double() @ w[s * rows:(s + 1) * rows].double().t()
        close(head[:, s * rows:(s + 1) * rows], want, "bfloat16", ("plane", s), bf16=1e-4)
    close(tail, x[4].double() @ w[4 * rows:].double().t(), "bfloat16", "last plane", bf16=1e-4)


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
def test_residual_after_every_layer_run(mixed_model, dtype):
    """The residual after each of the eight layer runs (a looped stretch counts every pass)
    against the plain model's: a fault shows in the run it enters."""
    from mstar_b200.engine.step import StepEntry
    from mstar_b200.parts import block as B

    weights, reqs, _, get = mixed_model
    want = []
    P.plain_forward(reqs["b"], U.as_numpy(weights), U.MIXED, layer_outputs=want)
    seen = []
    orig = B.SideBySideBlock.forward

    def recording(self, stream, ctx, cache):
        orig(self, stream, ctx, cache)
        seen.append((stream.h + stream.delta.materialize().float()).cpu())

    B.SideBySideBlock.forward = recording
    try:
        st = stepper_for(get(dtype))
        st.add_request("b")
        st.step([StepEntry("b", reqs["b"], [0])])
    finally:
        B.SideBySideBlock.forward = orig
    assert len(seen) == len(want) == U.runs(U.MIXED)
    for run, (g, w) in enumerate(zip(seen, want)):
        # (the float residual's distance grows by rounding alone from run to run)
        close(g, w, dtype, ("layer run", run), f32=5e-5, bf16=6e-2)


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
    cuts fall inside pages and chunks, inside the convolutions' taps and inside the scans'
    token chunks."""
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
@pytest.mark.parametrize("streams", ["1", "0"])
def test_mixed_batches_reuse_pages_and_slots(mixed_model, dtype, streams, monkeypatch):
    """Up to three live requests in a batch, portions beside single tokens, a request sitting
    out a step; five requests go through three slots and a pool of pages that holds less than
    all of them, so that slots and pages are used again; each agrees with itself alone.  With
    the sublayers on streams of their own and one after the other."""
    monkeypatch.setenv("MSTAR_PARALLEL_STREAMS", streams)
    weights, reqs, want, get = mixed_model
    model = U.load(U.MIXED, weights, dtype)
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
    st = stepper_for(model, num_pages=40, num_slots=3)
    got = U.run_schedule(st, reqs, schedule)
    check_all(got, want, dtype, "mixed")
    assert st.manager.num_requests() == 0 and st.manager.check() == 0
    assert st.manager.free_slots() == 3


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_behind_a_chunk_are_given_back(dtype):
    """A sequence far longer than the pool: only the pages a chunk can reach are held, so the
    pool is gone through several times."""
    cfg = U.config([U.parallel(U.left(2, 1, 16, 16, chunk=24), U.right(2, 16), mlp=None)], width=48, vocab=61)
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
    U.assert_close(got["r"], want, dtype, "pages of old chunks")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """A short prompt and 400 decoded tokens through captured graphs: several chunks of keys,
    both recurrent states, the convolution's rows and the shifted rows carried 400 steps."""
    cfg = U.config([U.parallel(U.left(2, 1, 16, 24, scale=0.4, chunk=90), U.right(2, 24), U.moe(4, 2, 32, 1.0, 24)),
                    U.ssd(U.mamba2(2, 16, 24, 1, 4, 1), U.moe(4, 1, 32, 0.6, 0)),
                    U.parallel(U.left(2, 2, 32, 16, scale=0.3, rot_dims=32, chunk=150), U.right(1, 40), mlp=None)],
                   width=64, vocab=97, loop=(1, 3, 2))
    weights = U.random_weights(cfg, 11)
    toks = U.tokens(cfg, 410, 12)
    want = U.plain_logits(cfg, weights, toks)
    st = stepper_for(U.load(cfg, weights, dtype), page_size=4, num_pages=104, num_slots=1)
    got = U.run_schedule(st, {"r": toks}, [[("r", 10)]] + [[("r", 1)]] * 400)
    U.assert_close(got["r"], want, dtype, "long decoding")
    assert st.graph_replays == 400


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_that_are_one_or_equal(dtype):
    """One head, one group, one tap, one expert, one norm group, chunks of one position, a loop
    of one layer run three times, a loop that is the whole model run once, no loop; keys as
    wide as values, everything equal; and sizes that are multiples of nothing (a width of 100,
    heads of 12 and 10, a vocabulary of 53)."""
    for layers, kw, rank in (
            ([U.ssd(U.mamba2(1, 8, 8, 1, 1, 1), U.moe(1, 1, 16, 1.0, 8, 1.0)),
              U.parallel(U.left(1, 1, 16, 16, scale=0.25, softcap=1.0, chunk=1, rot_dims=16, factor=1.0),
                         U.right(1, 16), mlp=None)],
             dict(width=32, vocab=50, loop=(1, 2, 3)), 1),
            ([U.parallel(U.left(2, 2, 8, 8, scale=0.5, chunk=4, rot_dims=8), U.right(2, 8), U.moe(2, 2, 8, 2.0, 8)),
              U.ssd(U.mamba2(8, 8, 8, 8, 2, 8), U.moe(2, 1, 8, 1.0, 0))],
             dict(width=32, vocab=50, loop=(0, 2, 1)), 8),
            ([U.parallel(U.left(3, 1, 12, 10, rot_dims=6, chunk=19), U.right(5, 10), U.moe(5, 3, 18, 1.0, 10)),
              U.ssd(U.mamba2(3, 10, 6, 3, 3, 3), U.moe(3, 2, 20, 0.5, 12)),
              U.ssd(U.mamba2(5, 6, 9, 1, 4, 2), None)],
             dict(width=100, vocab=53, loop=None), 3)):
        cfg = U.config(layers, **kw)
        weights = U.random_weights(cfg, 21, rank=rank)
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
        states = [{} for _ in range(U.runs(U.MIXED))]
        logits = P.plain_forward(list(prompt), w, U.MIXED, states)[-1]
        for tok in res.token_ids:
            best = int(np.argmax(logits))
            margin = float(logits[best] - logits[tok])
            assert tok == best or dtype == "bfloat16", (tok, best, margin)
            far_off += tok != best and margin >= 0.25
            logits = P.plain_forward([tok], w, U.MIXED, states)[-1]
    assert far_off <= len(prompts) * n_new // 20, far_off


def test_trace_replay_of_a_model_folder(mixed_model, tmp_path):
    """bin/trace_run on a folder of this design: the registry picks the model by config.json,
    the rank of the decay's projection comes from the tensors."""
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
