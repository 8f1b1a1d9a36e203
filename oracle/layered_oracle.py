"""Plain, slow statement of the layered decoders in numpy float64: Fitodra (latent attention, Mamba-2, norm after the sum)
and Molopel (lightning attention, windowed attention beside retention, layer norm before each part).

One function per mechanism, token loops written out, no cache and no batching: the whole sequence is given and every
position is computed from it.  Nothing here is shared with the product code.
"""
from __future__ import annotations

import math

import numpy as np

F8 = np.float64


def sigmoid(z):
    out = np.empty_like(z, dtype=F8)
    pos = z >= 0
    out[pos] = 1.0 / (1.0 + np.exp(-z[pos]))
    e = np.exp(z[~pos])
    out[~pos] = e / (1.0 + e)
    return out


def silu(z):
    z = np.asarray(z, F8)
    return z * sigmoid(z)


def softplus(z):
    z = np.asarray(z, F8)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit_rms(x, eps):
    """Rows of unit mean square: x (mean(x^2) + eps)^(-1/2)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_plain(x, w, eps):
    return unit_rms(x, eps) * w


def norm_about_zero(x, w, eps):
    """RMS norm whose stored weight is an offset from one."""
    return unit_rms(x, eps) * (1.0 + w)


def norm_in_parts(x, w, parts, eps):
    t, n = x.shape
    return unit_rms(x.reshape(t, parts, n // parts), eps).reshape(t, n) * w


# ---- rotation
def rotary_frequencies(dims, base, scaling=None):
    """(frequencies [dims/2], factor on cosine and sine).  `scaling`: YaRN's factor, original, fast, slow or None."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], F8)
    if not scaling:
        return f, 1.0
    fac, orig = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = np.empty_like(f)
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / fac * r + f[i] * (1.0 - r)
    return out, 0.1 * math.log(fac) + 1.0


def rotate_halves(x, positions, freqs, factor):
    """x [T, ..., dims]: element i turns with element i + dims/2 by positions * freqs[i]."""
    h = x.shape[-1] // 2
    a = np.asarray(positions, F8)[:, None] * freqs[None, :]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (h,)
    c, s = (np.cos(a) * factor).reshape(shape), (np.sin(a) * factor).reshape(shape)
    u, v = x[..., :h], x[..., h:]
    return np.concatenate([u * c - v * s, v * c + u * s], axis=-1)


# ---- attention
def attend_window_sink(scores, values, sink, window):
    """scores [T, T] of one head (already scaled), values [T, dv]: softmax over the last `window` positions up to and
    including the query's, with exp(sink) added to the denominator (sink None: not)."""
    T = scores.shape[0]
    out = np.zeros((T, values.shape[1]), F8)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        s = scores[i, lo:i + 1]
        top = s.max() if sink is None else max(s.max(), sink)
        e = np.exp(s - top)
        den = e.sum() + (0.0 if sink is None else math.exp(sink - top))
        out[i] = (e / den) @ values[lo:i + 1]
    return out


def latent_attention(h, w, p, m, eps):
    """h [T, width]; w: tensor lookup with prefix p; m: the mixer's sizes.  Keys and values are written out per head."""
    T = h.shape[0]
    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    cq = norm_plain(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(T, H, dn + dr)
    low = h @ w[p + "dkv"].T
    c = norm_plain(low[:, :rk], w[p + "dkv.norm"], eps)
    freqs, fac = rotary_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    kr = rotate_halves(low[:, rk:], pos, freqs, fac)
    qr = rotate_halves(q[:, :, dn:], pos, freqs, fac)
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    heads = []
    for i in range(H):
        s = (q[:, i, :dn] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        heads.append(attend_window_sink(s, v[:, i], float(w[p + "sink"][i]), m["mask"]["size"]))
    return np.concatenate(heads, axis=1) @ w[p + "o"].T


# ---- Mamba-2
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K]: out[t] = bias + sum_j taps[:, j] x[t - K + 1 + j], nothing before t = 0."""
    T, K = x.shape[0], taps.shape[1]
    out = np.tile(np.asarray(bias, F8), (T, 1))
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return out


def state_space(x, b, c, dt, a_log, d, groups):
    """x [T, heads, vdim], b and c [T, groups, N], dt [T, heads] (after softplus) -> y [T, heads, vdim]."""
    T, H, P = x.shape
    N = b.shape[2]
    y = np.zeros((T, H, P), F8)
    for h in range(H):
        g = h // (H // groups)
        S = np.zeros((N, P), F8)
        for t in range(T):
            S = math.exp(-math.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(b[t, g], x[t, h])
            y[t, h] = S.T @ c[t, g] + d[h] * x[t, h]
    return y


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, bc = H * P, G * N
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * bc], u[:, 2 * inner + 2 * bc:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    b, c = xbc[:, inner:inner + bc].reshape(T, G, N), xbc[:, inner + bc:].reshape(T, G, N)
    y = state_space(x, b, c, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"], G).reshape(T, inner)
    return norm_in_parts(y * silu(z), w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def gated_ffn(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- layer norm, gated feed-forward with the tanh form of GELU
def layer_norm(x, w, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    z = np.asarray(z, F8)
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_ffn(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- linear attention with one fixed decay per head
def decayed_sum(q, k, v, decay):
    """q and k [T, heads, n], v [T, heads, m]: o_t = S_t^T q_t with S_t = decay S_(t-1) + k_t v_t^T, S = 0 before the first."""
    T, H, n = q.shape
    out = np.zeros((T, H, v.shape[2]), F8)
    for h in range(H):
        S = np.zeros((n, v.shape[2]), F8)
        for t in range(T):
            S = decay[h] * S + np.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def lightning(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k = (silu(h @ w[p + n].T).reshape(T, H, m["dim"]) for n in "qk")
    v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o = decayed_sum(q, k, v, m["decay"]).reshape(T, -1)
    return (norm_plain(o, w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def retention(h, w, p, m, eps):
    T, H, n = h.shape[0], m["heads"], m["dim"]
    rd, pos = m["rot"]["dims"], np.arange(T)
    freqs, fac = rotary_frequencies(rd, m["rot"]["base"])

    def turn(x):
        return np.concatenate([rotate_halves(x[..., :rd], pos, freqs, fac), x[..., rd:]], axis=-1)

    q = turn((h @ w[p + "q"].T).reshape(T, H, n))
    k = turn((h @ w[p + "k"].T).reshape(T, H, n)) * n ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o = unit_rms(decayed_sum(q, k, v, m["decay"]), eps).reshape(T, -1)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- attention over a window with a learned bias per distance
def distance_bucket(n, rows, reach):
    """Half of the table's rows stand for one distance each, the rest for logarithmically growing ranges up to `reach`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def biased_window_attention(h, w, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = norm_plain((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, m["dim"]), w[p + "q.norm"], eps)
    k = norm_plain((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, m["dim"]), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, m["vdim"])
    rel = w[p + "rel"]
    rows = [distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)]
    dist = np.maximum(np.arange(T)[:, None] - np.arange(T)[None, :], 0)
    heads = []
    for i in range(H):
        g = i // (H // G)
        bias = np.array([rel[b, i] for b in rows], F8)[dist]
        heads.append(attend_window_sink((q[:, i] @ k[:, g].T) * m["scale"] + bias, v[:, g], None, m["mask"]["size"]))
    return np.concatenate(heads, axis=1) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return (m["left_scale"] * biased_window_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * retention(h, w, p + "right.", m["right"], eps))


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2, "lightning": lightning, "parallel": side_by_side}


def forward(cfg, weights, tokens, collect=None):
    """Logits [T, vocab] of one sequence.  `collect`: a list that receives the residual stream after every layer."""
    return {"Fitodra": forward_norm_after, "Molopel": forward_norm_before}[cfg["architecture"]](cfg, weights, tokens, collect)


def forward_norm_before(cfg, w, tokens, collect=None):
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + gelu_ffn(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if collect is not None:
            collect.append(x.copy())
    cap = cfg["logit_softcap"]
    return cap * np.tanh(layer_norm(x, w["final.norm"], eps) @ w["embed"].T / cap)


def forward_norm_after(cfg, weights, tokens, collect=None):
    w = weights
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        owner = i
        while cfg["layers"][owner].get("weights_of", owner) != owner:
            owner = cfg["layers"][owner]["weights_of"]
        p = f"l{owner}."
        x = norm_about_zero(alpha * x + MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = norm_about_zero(alpha * x + gated_ffn(x, w, p + "mlp."), w[p + "norm2"], eps)
        if collect is not None:
            collect.append(x.copy())
    return norm_about_zero(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, n):
    """`n` greedy tokens after `prompt`, every one from a full pass over everything before it."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]
