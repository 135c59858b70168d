"""Plain numpy restatement of the hybrid decoder family (design "Zutalix"): one function per
mechanism, float64 throughout, recurrences as literal loops over tokens, attention as an explicit
sum over the visible keys of each query. Test infrastructure only: slow on purpose, no state other
than what a function is handed, nothing shared with emberlm_b200/.

A model is (cfg, w): cfg the parsed config.json, w a dict of float arrays by tensor name. All
functions take whole sequences from position 0; a prefix property (row t depends on rows <= t only)
is what the framework's portions and decode steps are held to.
"""
from __future__ import annotations

import numpy as np

F = np.float64


# ---- elementwise ------------------------------------------------------------------------------
def sigmoid(z):
    z = np.asarray(z, F)
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, times weight (None: no weight)."""
    y = x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def clamped_glu(h, w_gate, w_up, w_down, limit):
    """g = min(gate, limit); u = clip(up, +-limit); W_down (g sigmoid(1.702 g) (u + 1))."""
    g = np.minimum(h @ w_gate.T, limit)
    u = np.clip(h @ w_up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w_down.T


# ---- rotary positions ---------------------------------------------------------------------------
def rope_frequencies(dims, base, scaling=None):
    """Inverse frequencies of the dims/2 pairs; wavelength-dependent scaling with a smooth middle band."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], F)
    if scaling is None:
        return f
    fac, lo, hi, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for fi in f:
        wl = 2.0 * np.pi / fi
        if wl < orig / hi:
            out.append(fi)
        elif wl > orig / lo:
            out.append(fi / fac)
        else:
            s = (orig / wl - lo) / (hi - lo)
            out.append((1.0 - s) * fi / fac + s * fi)
    return np.array(out, F)


def rope_interleaved(x, positions, freqs):
    """x [T, heads, dim]: pair (2i, 2i+1) of the first 2*len(freqs) dimensions turned by position * freqs[i]."""
    y = np.array(x, F)
    for i, f in enumerate(freqs):
        a = positions.astype(F) * f
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * c - v * s
        y[:, :, 2 * i + 1] = v * c + u * s
    return y


# ---- attention ------------------------------------------------------------------------------------
def chunked_attention(q, k, v, scale, size):
    """Softmax attention of q [T, H, d] over k [T, G, d], v [T, G, dv]: query i sees keys j <= i of its own
    `size`-long chunk (chunks counted from position 0)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), F)
    for i in range(T):
        j0 = (i // size) * size
        for h in range(H):
            g = h // (H // G)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[j0:i + 1, g]
    return out


# ---- recurrences ------------------------------------------------------------------------------------
def lightning(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q, k [T, H, d], v [T, H, dv]."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((d, v.shape[2]), F)
        for t in range(T):
            S = decay[h] * S + np.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def short_conv(x, taps):
    """Causal depthwise convolution over time: x [T, C], taps [C, n], the last column meets the current row."""
    T, C = x.shape
    n = taps.shape[1]
    y = np.zeros((T, C), F)
    for t in range(T):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                y[t] += taps[:, j] * x[src]
    return y


def unit(x):
    return x / np.sqrt(np.sum(np.square(x), axis=-1, keepdims=True) + 1e-6)


def channel_delta_rule(q, k, v, g, beta):
    """Delta rule with one decay per key channel: q, k, g [T, H, d], v [T, H, dv], beta [T, H].
    S <- diag(g) S; S <- S + k (beta (v - S^T k))^T; o = S^T q."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((d, v.shape[2]), F)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + np.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


# ---- mixers -----------------------------------------------------------------------------------------
def mixer_parallel(h, w, p, m, eps):
    """Chunked attention with tied keys / values beside lightning attention, both reading h [T, W]."""
    T = h.shape[0]
    a, r = m["left"], m["right"]
    H, G, d = a["heads"], a["kv_heads"], a["dim"]
    L = p + "left."
    q = (h @ w[L + "q"].T + w[L + "q.b"]).reshape(T, H, d)
    k = (h @ w[L + "k"].T + w[L + "k.b"]).reshape(T, G, d)
    v = k
    f = rope_frequencies(a["rot"]["dims"], a["rot"]["base"], a["rot"].get("scaling"))
    pos = np.arange(T)
    o = chunked_attention(rope_interleaved(q, pos, f), rope_interleaved(k, pos, f), v, a["scale"], a["mask"]["size"])
    o = o * sigmoid(h @ w[L + "g"].T)[:, :, None]
    left = o.reshape(T, H * d) @ w[L + "o"].T

    R = p + "right."
    H, d, dv = r["heads"], r["dim"], r["vdim"]
    q = silu(h @ w[R + "q"].T).reshape(T, H, d)
    k = silu(h @ w[R + "k"].T).reshape(T, H, d)
    v = silu(h @ w[R + "v"].T).reshape(T, H, dv)
    o = lightning(q, k, v, r["decay"]).reshape(T, H * dv)
    o = rms_norm(o, w[R + "norm"], eps) * sigmoid(h @ w[R + "g"].T)
    right = o @ w[R + "o"].T
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


def mixer_channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, d)
    k = silu(short_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, d)
    v = silu(short_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(T, H, d))
    o = rms_norm(channel_delta_rule(q, k, v, g, beta), w[p + "norm"], eps)
    o = o * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"parallel": mixer_parallel, "channel_delta": mixer_channel_delta}


# ---- model ------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, F) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[lay["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", lay["mixer"], eps)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if lay["mlp"] is not None:
            y = clamped_glu(rms_norm(x, w[p + "norm2"], eps), w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"],
                            lay["mlp"]["limit"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n):
    """n greedy tokens after the prompt (first index of the maximum), recomputing the whole sequence each time."""
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
