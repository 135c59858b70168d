"""Plain numpy restatement of the design "Detatar" of the layer-list family: one function per mechanism,
float64 throughout, the recurrence as a literal loop over tokens, attention as an explicit sum over the
visible keys of each query, every expert run token by token. Test infrastructure only, like
oracle/hybrid.py (whose elementwise helpers it uses): nothing shared with emberlm_b200/.

A model is (cfg, w): cfg the parsed config.json, w a dict of float arrays by tensor name. All functions
take whole sequences from position 0.
"""
from __future__ import annotations

import numpy as np

from oracle.hybrid import F, rms_norm, sigmoid, silu


# ---- elementwise --------------------------------------------------------------------------------
def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def grouped_rms_norm(x, weight, eps, groups):
    """Equal consecutive parts of the last axis, each divided by its own root mean square."""
    parts = x.reshape(x.shape[:-1] + (groups, -1))
    return (parts / np.sqrt(np.mean(np.square(parts), axis=-1, keepdims=True) + eps)).reshape(x.shape) * weight


def previous(h):
    """Row t holds row t - 1, zeros in front of the first."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def token_mix(h, mu):
    """h + (previous h - h) mu."""
    return h + (previous(h) - h) * mu


def rotate_half(x, positions, base):
    """x [..., T, dims]: the pair (i, i + dims/2) turned by position * base^(-2i/dims)."""
    n = x.shape[-1] // 2
    a = positions[:, None].astype(F) * np.array([base ** (-2.0 * i / (2 * n)) for i in range(n)], F)[None]
    u, v = x[..., :n], x[..., n:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], axis=-1)


# ---- latent attention -----------------------------------------------------------------------------
def causal_attention(q, k, v, scale):
    """Softmax attention of q [T, H, d] over k [T, H, d], v [T, H, dv], query i over the keys j <= i."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for i in range(T):
        s = np.einsum("jhd,hd->hj", k[:i + 1], q[i]) * scale
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = np.einsum("hj,jhd->hd", p / p.sum(axis=1, keepdims=True), v[:i + 1])
    return out


def mixer_latent_attention(h, w, p, m, eps):
    """Keys and values of every head are read out of one normed latent per position; a rotated key part is
    shared by the heads; one sigmoid gate per head."""
    T = h.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, d + dr)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    pos = np.arange(T)
    k_rot = rotate_half(down[:, R:], pos, m["rot"]["base"])
    q_rot = rotate_half(q[:, :, d:].transpose(1, 0, 2), pos, m["rot"]["base"]).transpose(1, 0, 2)
    q = np.concatenate([q[:, :, :d], q_rot], axis=2)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot[:, None], H, axis=1)], axis=2)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = causal_attention(q, k, v, m["scale"]) * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- time mixing with a bonus ---------------------------------------------------------------------
def wkv_recurrence(r, k, v, decay, u):
    """o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(decay_t) S + k_t v_t^T; r, k, v, decay [T, H, d], u [H, d]."""
    T, H, d = r.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((d, v.shape[2]), F)
        for t in range(T):
            kv = np.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = decay[t, h][:, None] * S + kv
    return out


def mixer_wkv(h, w, p, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    mix = {s: token_mix(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).reshape(T, H, d) for s in "rkv")
    z = np.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    o = wkv_recurrence(r, k, v, np.exp(-np.exp(z)).reshape(T, H, d), w[p + "u"].reshape(H, d))
    o = rms_norm(o, None, eps).reshape(T, H * d) * w[p + "norm"] * silu(mix["g"] @ w[p + "g"].T)
    return o @ w[p + "o"].T


MIXERS = {"latent_attention": mixer_latent_attention, "wkv": mixer_wkv}


# ---- feed-forward ---------------------------------------------------------------------------------
def glu(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, top, groups=None):
    """Chosen outputs and their weights for router logits z of one token: softmax scores, the correction in
    the choice only, the best groups (by their best choice score) kept, weights normalised over the chosen."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    choice = s + correction
    if groups:
        per = len(z) // groups["count"]
        best = np.array([choice[g * per:(g + 1) * per].max() for g in range(groups["count"])])
        kept = np.argsort(-best, kind="stable")[:groups["keep"]]
        choice = np.array([c if i // per in kept else -np.inf for i, c in enumerate(choice)])
    chosen = np.argsort(-choice, kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def route_margin(z, correction, top, groups=None):
    """How close the choice is: the smallest gap between a taken and a refused choice score, groups included."""
    s = np.exp(z - z.max())
    choice = s / s.sum() + correction
    gap = np.inf
    if groups and groups["keep"] < groups["count"]:
        best = -np.sort(-choice.reshape(groups["count"], -1).max(axis=1))
        gap = best[groups["keep"] - 1] - best[groups["keep"]]
        kept = np.argsort(-choice.reshape(groups["count"], -1).max(axis=1), kind="stable")[:groups["keep"]]
        choice = choice.reshape(groups["count"], -1)[kept].ravel()
    choice = -np.sort(-choice)
    return min(gap, choice[top - 1] - choice[top]) if top < len(choice) else gap


def moe(h, w, p, f):
    r = f["router"]
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weight = route(w[p + "router"] @ h[t], w[p + "correction"], r["top"], r.get("groups"))
        for e, a in zip(chosen, weight):
            out[t] += a * (h[t] if e >= r["experts"] else glu(h[t], w, f"{p}e{e}.", silu))
    if f.get("shared"):
        out = out + glu(h, w, p + "shared.", silu) * sigmoid(h @ w[p + "shared.sg"].T)
    return out


def feed_forward(h, w, p, f):
    return glu(h, w, p, gelu_tanh) if f["kind"] == "dense" else moe(h, w, p, f)


# ---- model ----------------------------------------------------------------------------------------
def layer(x, w, p, lay, eps, groups):
    """x + gated (mixer of the shifted h) + gated (feed-forward of h), both from one norm."""
    h = grouped_rms_norm(x, w[p + "norm1"], eps, groups)
    y = MIXERS[lay["type"]](token_mix(h, w[p + "shift"]), w, p + "mix.", lay["mixer"], eps)
    y = y * sigmoid(h @ w[p + "rg1"].T + w[p + "rg1.b"])
    if lay.get("mlp"):
        y = y + feed_forward(h, w, p + "mlp.", lay["mlp"]) * sigmoid(h @ w[p + "rg2"].T + w[p + "rg2.b"])
    return x + y


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, F) for k, v in w.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        x = layer(x, w, f"l{lay.get('weights_of', i)}.", lay, eps, groups)
        if layers_out is not None:
            layers_out.append(x.copy())
    return grouped_rms_norm(x, w["final.norm"], eps, groups) @ w["head"].T
