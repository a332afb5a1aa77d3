"""A plain, slow implementation of the Famarax decoder in numpy float64: one function per
mechanism, written from the design's equations and sharing nothing with the engine.

Every norm of the model is a *dynamic tanh*, ``tanh(alpha x) w + b`` with one alpha a norm: no
mean or variance.  The embedding row passes such a norm, and the residual is ``streams`` copies
of the result (hyper-connections): a sublayer reads ``norm(sum_s in[s] x_s)``, and every copy
becomes a mix of the old copies plus its own share of the sublayer's output.  A mixer is one of

* ``attention``: grouped queries; rotate-half pairs over the first features of q and k, *then*
  each q and k head divided by its root mean square (no weight); scores scaled and soft-capped;
  a sliding window; ordinary softmax.  With ``v_mix`` the values are blended with the first such
  layer's values of the same token before they are kept;
* ``delta``: the gated delta rule with one decay a head (short causal convolutions with SiLU on
  q, k and v, unit q and k, a write strength a head), each head's read-out RMS-normed and gated
  by a SiLU.

The feed-forward is routed experts: softmax scores over all experts, a correction added for the
choice only, experts in groups of which the best few stay eligible (a group counts as its best
choice score), the chosen scores renormalised and scaled, a shared expert beside them.  The
logits are scaled and soft-capped.

Everything works on one sequence; ``states`` (a dict per layer) carries what a layer keeps from
call to call, so that a sequence can be fed whole, in portions, or token by token.
"""
from __future__ import annotations

import numpy as np

F = np.float64


def plain_dynamic_tanh(x, alpha, weight, bias):
    return np.tanh(np.asarray(x, F) * float(alpha)) * np.asarray(weight, F) + np.asarray(bias, F)


def plain_norm(x, w, name):
    return plain_dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])


def plain_over_rms(x, eps):
    x = np.asarray(x, F)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def plain_sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, F)))


def plain_silu(z):
    z = np.asarray(z, F)
    return z * plain_sigmoid(z)


def plain_softplus(z):
    z = np.asarray(z, F)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def plain_soft_cap(z, cap):
    return z if cap is None else cap * np.tanh(np.asarray(z, F) / cap)


# ------------------------------------------------------------------ attention
def plain_rotate_half(x, positions, dims, base):
    """x: [tokens, heads, dim]; feature i is rotated with feature i + dims/2 by the angle
    position * base^(-2i/dims), for i < dims / 2; the features past dims pass."""
    x = np.array(x, F)
    half = dims // 2
    for i in range(half):
        ang = np.asarray(positions, F) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        u, v = x[..., i].copy(), x[..., i + half].copy()
        x[..., i] = u * c - v * s
        x[..., i + half] = v * c + u * s
    return x


def plain_window_attention(q, keys, values, first_position, scale, softcap=None, window=None):
    """q: [tokens, heads, dim], the tokens at positions first_position ..; keys [n, kv_heads,
    dim] and values [n, kv_heads, vdim] of positions 0 .. n - 1.  Position i sees the keys j with
    0 <= i - j < window.  Query head h reads key head h // (heads / kv_heads)."""
    T, H, _ = q.shape
    per = H // keys.shape[1]
    out = np.zeros((T, H, values.shape[2]), F)
    for t in range(T):
        i = first_position + t
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = plain_soft_cap(keys[lo:i + 1, h // per] @ q[t, h] * scale, softcap)
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ values[lo:i + 1, h // per]
    return out


def plain_mix_values(v, first, lam):
    """(1 - lam) v + lam first."""
    return (1.0 - float(lam)) * v + float(lam) * first


def _grow(state, name, rows):
    state[name] = rows if name not in state else np.concatenate([state[name], rows], axis=0)
    return state[name]


def plain_attention(h, positions, w, p, m, eps, state, shared):
    """``shared``: a dict that lives for one call of the model; the first layer with ``v_mix``
    leaves its values there."""
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    k = (h @ w[p + "k"].T).reshape(T, G, D)
    v = (h @ w[p + "v"].T).reshape(T, G, VD)
    rot = m.get("rot")
    if rot:
        q = plain_rotate_half(q, positions, rot["dims"], rot["base"])
        k = plain_rotate_half(k, positions, rot["dims"], rot["base"])
    q, k = plain_over_rms(q, eps), plain_over_rms(k, eps)
    if m.get("v_mix"):
        if "v_first" in shared:
            v = plain_mix_values(v, shared["v_first"], w[p + "vmix"])
        else:
            shared["v_first"] = v
    mask = m.get("mask")
    o = plain_window_attention(q, _grow(state, "k", k), _grow(state, "v", v), int(positions[0]),
                               m["scale"], m.get("softcap"), mask["size"] if mask else None)
    return o.reshape(T, H * VD) @ w[p + "o"].T


# ------------------------------------------------------------------ delta rule
def plain_short_conv(x, weight, state, name):
    """Causal convolution over time per channel: x [tokens, channels], weight [channels, taps]
    whose last column meets the token itself; zeros before the sequence's start.  The last
    taps - 1 inputs are carried in ``state[name]``."""
    taps = weight.shape[1]
    before = state.get(name)
    if before is None:
        before = np.zeros((taps - 1, x.shape[1]), F)
    padded = np.concatenate([before, x], axis=0)
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        out[t] = np.sum(padded[t:t + taps].T * weight, axis=1)
    state[name] = padded[padded.shape[0] - (taps - 1):]
    return out


def plain_delta_rule(q, k, v, beta, g, S):
    """One head, token after token: S [dim, vdim] first fades by the number g, the write is
    beta (v - S^T k), and the read-out S^T q sees it.  Returns the outputs [tokens, vdim];
    S is changed in place."""
    out = np.zeros((q.shape[0], v.shape[1]), F)
    for t in range(q.shape[0]):
        S *= g[t]
        u = beta[t] * (v[t] - S.T @ k[t])
        S += np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def plain_unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def plain_gated_delta(h, w, p, m, eps, state):
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (plain_silu(plain_short_conv(h @ w[p + n].T, w[p + n + ".conv"], state, "c" + n))
               for n in ("q", "k", "v"))
    q = plain_unit(q.reshape(T, G, D)) * D ** -0.5
    k = plain_unit(k.reshape(T, G, D))
    v = v.reshape(T, H, VD)
    beta = plain_sigmoid(h @ w[p + "b"].T)                                      # [T, H]
    decay = np.exp(-np.exp(np.asarray(w[p + "A_log"], F))
                   * plain_softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))        # [T, H]
    if "S" not in state:
        state["S"] = np.zeros((H, D, VD), F)
    o = np.zeros((T, H, VD), F)
    for hd in range(H):
        g = hd // (H // G)
        o[:, hd] = plain_delta_rule(q[:, g], k[:, g], v[:, hd], beta[:, hd], decay[:, hd],
                                    state["S"][hd])
    o = plain_over_rms(o, eps) * w[p + "norm"]
    return (o.reshape(T, H * VD) * plain_silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ experts
def plain_expert(h, w, p):
    return (plain_silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def plain_route(z, correction, top, groups=None, scale=1.0):
    """z: [tokens, experts] router logits.  Returns (chosen [tokens, top], weights)."""
    z = np.asarray(z, F)
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    choice = s + np.asarray(correction, F)
    if groups:
        T, E = z.shape
        per = E // groups["count"]
        best = choice.reshape(T, groups["count"], per).max(axis=-1)
        keep = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
        open_ = np.zeros((T, groups["count"]), bool)
        np.put_along_axis(open_, keep, True, axis=1)
        choice = np.where(np.repeat(open_, per, axis=1), choice, -np.inf)
    chosen = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    weights = np.take_along_axis(s, chosen, axis=1)
    return chosen, weights / (weights.sum(axis=-1, keepdims=True) + 1e-20) * scale


def plain_experts(h, w, p, mlp):
    r = mlp["router"]
    chosen, weights = plain_route(h @ w[p + "router"].T, w[p + "correction"], r["top"],
                                  r.get("groups"), r.get("scale", 1.0))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t], weights[t]):
            out[t] += c * plain_expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared") is not None:
        out = out + plain_expert(h, w, p + "shared.")
    return out


# ------------------------------------------------------------------ the model
def plain_hyper_read(xs, w_in):
    """xs: [streams, tokens, width] -> sum_s in[s] xs[s]."""
    return np.tensordot(np.asarray(w_in, F), xs, axes=(0, 0))


def plain_hyper_write(xs, y, w_mix, w_out):
    """new[t] = sum_s mix[s, t] xs[s] + out[t] * y, every t from the old copies."""
    new = np.tensordot(np.asarray(w_mix, F).T, xs, axes=(1, 0))
    return new + np.asarray(w_out, F)[:, None, None] * y[None]


def plain_head(x, w, cfg):
    z = plain_norm(x, w, "final.norm") @ np.asarray(w["head"], F).T * cfg.get("logit_scale", 1.0)
    return plain_soft_cap(z, cfg.get("logit_softcap"))


def plain_forward(tokens, w, cfg, states=None, layer_outputs=None):
    """float64 logits [len(tokens), vocab].  ``states``: a list with one dict per layer; given,
    the tokens continue the sequence it holds.  ``layer_outputs``: a list that takes the
    residual (the sum of the copies) after every layer."""
    if states is None:
        states = [{} for _ in cfg["layers"]]
    eps = cfg["norm"]["eps"]
    start = states[0].get("len", 0)
    positions = np.arange(start, start + len(tokens))
    x = plain_norm(np.asarray(w["embed"], F)[np.asarray(tokens)], w, "embed.norm")
    xs = np.stack([x] * cfg["streams"])
    shared: dict = {}
    for i, (layer, state) in enumerate(zip(cfg["layers"], states)):
        p = f"l{i}."
        state["len"] = start + len(tokens)
        for q in (1, 2):
            if q == 2 and layer.get("mlp") is None:
                continue
            h = plain_norm(plain_hyper_read(xs, w[f"{p}hc{q}.in"]), w, f"{p}norm{q}")
            if q == 2:
                y = plain_experts(h, w, p + "mlp.", layer["mlp"])
            elif layer["type"] == "attention":
                y = plain_attention(h, positions, w, p + "mix.", layer["mixer"], eps, state, shared)
            elif layer["type"] == "delta":
                y = plain_gated_delta(h, w, p + "mix.", layer["mixer"], eps, state)
            else:
                raise ValueError(layer["type"])
            xs = plain_hyper_write(xs, y, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"])
        if layer_outputs is not None:
            layer_outputs.append(xs.sum(axis=0))
    return plain_head(xs.sum(axis=0), w, cfg)
