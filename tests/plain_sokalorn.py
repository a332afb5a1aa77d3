"""A plain, slow implementation of the Sokalorn decoder in numpy float64: one function per
mechanism, written from the design's equations and sharing nothing with the engine.

A layer has one RMS norm ``h = norm1(x)`` and two sublayers side by side that read it:
``x += mixer(h~) + ff(h)``, where ``h~`` is the *token-shifted* h: ``h + (h' - h) * shift``
with h' the previous token's h (zeros before the first).  A mixer is one of

* ``parallel``: the mean of two branch outputs, each RMS-normed over the width with a weight
  of its own.  Left: grouped-query attention inside chunks of positions, rotate-half pairs
  with linearly scaled frequencies, soft-capped scores, *sigmoid* weights with a bias a head
  (nothing is normalised over the keys), a sigmoid gate a feature.  Right: RWKV-style time
  mixing with a decay per head and key channel and a bonus for the current token;
* ``mamba2``: the state-space recurrence with a scalar decay a head.

The feed-forward is routed experts (softmax scores over all, the chosen ones renormalised)
beside a shared expert with a sigmoid gate a token; every expert is a clamped gated
feed-forward.  Layers ``loop.start .. loop.stop - 1`` run ``loop.times`` times; before each
pass the residual becomes ``W_in [x; x0]``, x0 the embedding output.

Everything works on one sequence; ``states`` (a dict per layer run) carries what a layer
keeps from call to call, so that a sequence can be fed whole, in portions, or token by token.
"""
from __future__ import annotations

import numpy as np

F = np.float64


def plain_rms_norm(x, weight, eps):
    x = np.asarray(x, F)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * np.asarray(weight, F)


def plain_sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, F)))


def plain_silu(z):
    z = np.asarray(z, F)
    return z * plain_sigmoid(z)


def plain_softplus(z):
    z = np.asarray(z, F)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def plain_previous(x, state, name):
    """The row before each row of x [tokens, width]; the row before the first is the last one
    of the call before (zeros at the start of the sequence).  The last row is carried on."""
    before = state.get(name)
    if before is None:
        before = np.zeros(x.shape[1], F)
    state[name] = x[-1].copy()
    return np.concatenate([before[None], x[:-1]], axis=0)


def plain_mix(x, prev, amount):
    return x + (prev - x) * np.asarray(amount, F)


# ------------------------------------------------------------------ attention
def plain_rotate_half(x, positions, dims, base, factor):
    """x: [tokens, heads, dim]; feature i is rotated with feature i + dims/2 by the angle
    position * base^(-2i/dims) / factor, for i < dims / 2; the features past dims pass."""
    x = np.array(x, F)
    half = dims // 2
    for i in range(half):
        ang = np.asarray(positions, F) * (float(base) ** (-2.0 * i / dims) / float(factor))
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        u, v = x[..., i].copy(), x[..., i + half].copy()
        x[..., i] = u * c - v * s
        x[..., i + half] = v * c + u * s
    return x


def plain_sigmoid_attention(q, keys, values, first_position, scale, softcap, bias, chunk):
    """q: [tokens, heads, dim] at positions first_position ..; keys [n, kv_heads, dim] and values
    [n, kv_heads, vdim] of positions 0 .. n - 1.  The weight of a visible key is sigmoid(score +
    bias[h]), the score soft-capped; a key is visible from the same chunk of ``chunk``
    positions, at or before the token."""
    T, H, _ = q.shape
    G = keys.shape[1]
    out = np.zeros((T, H, values.shape[2]), F)
    for t in range(T):
        p = first_position + t
        lo = 0 if chunk is None else (p // chunk) * chunk
        for h in range(H):
            g = h // (H // G)
            s = keys[lo:p + 1, g] @ q[t, h] * scale
            if softcap is not None:
                s = softcap * np.tanh(s / softcap)
            out[t, h] = plain_sigmoid(s + bias[h]) @ values[lo:p + 1, g]
    return out


def _grow(state, name, rows):
    state[name] = rows if name not in state else np.concatenate([state[name], rows], axis=0)
    return state[name]


def plain_left(h, positions, w, p, m, state):
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    k = (h @ w[p + "k"].T).reshape(T, G, D)
    v = (h @ w[p + "v"].T).reshape(T, G, VD)
    rot = m["rot"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    q = plain_rotate_half(q, positions, rot["dims"], rot["base"], factor)
    k = plain_rotate_half(k, positions, rot["dims"], rot["base"], factor)
    keys, values = _grow(state, "k", k), _grow(state, "v", v)
    o = plain_sigmoid_attention(q, keys, values, int(positions[0]), m["scale"], m.get("softcap"),
                                w[p + "pb"], (m.get("mask") or {}).get("size"))
    o = o.reshape(T, H * VD) * plain_sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ------------------------------------------------------------------ recurrences
def plain_rwkv_scan(r, k, v, decay, bonus, S):
    """One head, token after token: o = (S + diag(bonus) k v^T)^T r from the old state S [dim,
    dim], then S = diag(decay) S + k v^T (in place).  Returns [tokens, dim]."""
    out = np.zeros_like(v)
    for t in range(r.shape[0]):
        out[t] = S.T @ r[t] + (np.asarray(bonus, F) * k[t] @ r[t]) * v[t]
        S *= decay[t][:, None]
        S += np.outer(k[t], v[t])
    return out


def plain_right(h, w, p, m, eps, state):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    prev = plain_previous(h, state, "right_prev")
    mixed = {s: plain_mix(h, prev, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).reshape(T, H, D) for s in "rkv")
    gate = plain_silu(mixed["g"] @ w[p + "g"].T)
    decay = np.exp(-np.exp(np.tanh(mixed["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))
    decay = decay.reshape(T, H, D)
    if "S" not in state:
        state["S"] = np.zeros((H, D, D), F)
    o = np.zeros((T, H, D), F)
    for hd in range(H):
        o[:, hd] = plain_rwkv_scan(r[:, hd], k[:, hd], v[:, hd], decay[:, hd], w[p + "u"][hd],
                                   state["S"][hd])
    o = plain_rms_norm(o, None, eps).reshape(T, H * D) * w[p + "norm"] * gate
    return o @ w[p + "o"].T


def plain_short_conv(x, weight, bias, state, name):
    """Causal convolution over time per channel with a bias: x [tokens, channels], weight
    [channels, taps] whose last column meets the token itself; zeros before the sequence's
    start.  The last taps - 1 inputs are carried in ``state[name]``."""
    taps = weight.shape[1]
    before = state.get(name)
    if before is None:
        before = np.zeros((taps - 1, x.shape[1]), F)
    padded = np.concatenate([before, x], axis=0)
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        out[t] = np.sum(padded[t:t + taps].T * weight, axis=1) + bias
    state[name] = padded[padded.shape[0] - (taps - 1):]
    return out


def plain_ssd_scan(x, B, C, dt, rate, skip, S):
    """One head, token after token: S [N, vdim] = exp(-rate dt) S + dt B x^T (in place), then y =
    S^T C + skip x.  Returns [tokens, vdim]."""
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        S *= np.exp(-rate * dt[t])
        S += dt[t] * np.outer(B[t], x[t])
        out[t] = S.T @ C[t] + skip * x[t]
    return out


def plain_mamba2(h, w, p, m, eps, state):
    T = h.shape[0]
    H, VD, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * VD
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = plain_silu(plain_short_conv(xbc, w[p + "conv"], w[p + "conv.b"], state, "conv"))
    x = xbc[:, :inner].reshape(T, H, VD)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = plain_softplus(dt + w[p + "dt_bias"])
    if "S" not in state:
        state["S"] = np.zeros((H, N, VD), F)
    y = np.zeros((T, H, VD), F)
    for hd in range(H):
        g = hd // (H // G)
        y[:, hd] = plain_ssd_scan(x[:, hd], B[:, g], C[:, g], dt[:, hd],
                                  float(np.exp(w[p + "A_log"][hd])), w[p + "D"][hd], state["S"][hd])
    y = y.reshape(T, inner) * plain_silu(z)
    parts = y.reshape(T, m["norm_groups"], inner // m["norm_groups"])
    y = plain_rms_norm(parts, None, eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def plain_mixer(kind, h, positions, w, p, m, eps, state):
    if kind == "mamba2":
        return plain_mamba2(h, w, p, m, eps, state)
    if kind == "parallel":
        left = plain_left(h, positions, w, p + "left.", m["left"], state)
        right = plain_right(h, w, p + "right.", m["right"], eps, state)
        return 0.5 * (plain_rms_norm(left, w[p + "left.out"], eps)
                      + plain_rms_norm(right, w[p + "right.out"], eps))
    raise ValueError(kind)


# ------------------------------------------------------------------ feed-forward
def plain_clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * plain_sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def plain_route(z, top):
    """Indices and weights of the ``top`` largest softmax scores per row, renormalised."""
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    weight = np.take_along_axis(s, chosen, axis=-1)
    return chosen, weight / (weight.sum(axis=-1, keepdims=True) + 1e-20)


def plain_moe(h, w, p, mlp):
    chosen, weight = plain_route(h @ w[p + "router"].T, mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], weight[t]):
            q = f"{p}e{e}."
            out[t] += s * plain_clamped_expert(h[t], w[q + "gate"], w[q + "up"], w[q + "down"],
                                               mlp["expert"]["limit"])
    if mlp.get("shared"):
        q = p + "shared."
        shared = plain_clamped_expert(h, w[q + "gate"], w[q + "up"], w[q + "down"],
                                      mlp["shared"]["limit"])
        out = out + shared * plain_sigmoid(h @ w[q + "sg"].T)
    return out


# ------------------------------------------------------------------ the model
def plain_loop_input(x, x0, w_in):
    return np.concatenate([x, x0], axis=-1) @ np.asarray(w_in, F).T


def plain_run_order(cfg):
    """(layer index, whether a pass of the loop begins with this run) in the order of runs."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * times
            + [(i, False) for i in range(b, n)])


def plain_forward(tokens, w, cfg, states=None, layer_outputs=None):
    """float64 logits [len(tokens), vocab].  ``states``: a list with one dict per layer run;
    given, the tokens continue the sequence it holds.  ``layer_outputs``: a list that takes
    the residual after every layer run."""
    order = plain_run_order(cfg)
    if states is None:
        states = [{} for _ in order]
    eps = cfg["norm"]["eps"]
    start = states[0].get("len", 0) if states else 0
    positions = np.arange(start, start + len(tokens))
    x0 = np.asarray(w["embed"], F)[np.asarray(tokens)]
    x = x0
    for run, (i, begins_pass) in enumerate(order):
        layer, state, p = cfg["layers"][i], states[run], f"l{i}."
        state["len"] = start + len(tokens)
        if begins_pass:
            x = plain_loop_input(x, x0, w["loop.in"])
        h = plain_rms_norm(x, w[p + "norm1"], eps)
        shifted = plain_mix(h, plain_previous(h, state, "prev"), w[p + "shift"])
        y = plain_mixer(layer["type"], shifted, positions, w, p + "mix.", layer["mixer"], eps, state)
        if layer.get("mlp") is not None:
            y = y + plain_moe(h, w, p + "mlp.", layer["mlp"])
        x = x + y
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return plain_rms_norm(x, w["final.norm"], eps) @ np.asarray(w["head"], F).T
