"""CPU restatement (numpy, float64) of the decoder whose layers normalise after the sum
(Femolix): gated delta rule, and chunk-local grouped-query attention beside a linear attention
of constant decay, with dense or routed feed-forwards.

TEST INFRASTRUCTURE ONLY: imported by tests/ and smoke().  One function per mechanism, each
the plain equation evaluated token by token; nothing is shared with the shipped package.
Every function takes and returns arrays with one row per token.
"""
from __future__ import annotations

import numpy as np

from oracle.mixed_oracle import F, _sub, causal_conv, rms_norm, rotate_half, sigmoid, silu, softplus

UNIT_EPS = 1e-6


# ---- pieces ----------------------------------------------------------------------------
def unit(x):
    """x / |x|, with a constant under the root."""
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)


def norm_after_sum(x, y, w, alpha, eps):
    return rms_norm(alpha * x + y, w, eps)


def softcap(z, cap):
    return cap * np.tanh(z / cap)


# ---- attention -------------------------------------------------------------------------
def same_chunk(i, j, size):
    return i // size == j // size


def chunked_attention(q, k, v, scale, size):
    """q [tokens, H, d], k [tokens, G, d], v [tokens, G, e]; query head h reads key/value head
    h // (H / G); position i sees the positions up to i of its own chunk of `size`."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((n, H, v.shape[2]), F)
    for i in range(n):
        seen = [j for j in range(i // size * size if size else 0, i + 1) if not size or same_chunk(i, j, size)]
        for h in range(H):
            g = h // (H // G)
            s = (k[seen, g] @ q[i, h]) * scale
            p = np.exp(s - s.max())
            out[i, h] = (p @ v[seen, g]) / p.sum()
    return out


# ---- recurrences on a matrix per head ----------------------------------------------------
def delta_rule(q, k, v, g, beta):
    """q, k [tokens, H, d], v [tokens, H, e], g, beta [tokens, H]:
    the memory fades by g, what it holds under the key moves by the fraction beta towards the value,
    and the query reads the result."""
    n, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), F)
    out = np.zeros_like(v, dtype=F)
    for t in range(n):
        for h in range(H):
            S[h] *= g[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] += np.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out


def decayed_linear_attention(q, k, v, decay):
    """A memory per head that fades by its decay and adds each value under its key; the query reads."""
    n, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), F)
    out = np.zeros_like(v, dtype=F)
    for t in range(n):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out


# ---- mixers ----------------------------------------------------------------------------
def mixer_delta(x, c, W, eps):
    n, H, G, d, e = x.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def short(name):
        return silu(causal_conv(x @ W[name].T, W[name + ".conv"], 0.0))

    rep = H // G
    q = np.repeat(unit(short("q").reshape(n, G, d)) * d ** -0.5, rep, axis=1)
    k = np.repeat(unit(short("k").reshape(n, G, d)), rep, axis=1)
    v = short("v").reshape(n, H, e)
    beta = sigmoid(x @ W["b"].T)
    g = np.exp(-np.exp(W["A_log"]) * softplus(x @ W["a"].T + W["dt_bias"]))
    o = rms_norm(delta_rule(q, k, v, g, beta), W["norm"], eps)
    return (o.reshape(n, H * e) * silu(x @ W["g"].T)) @ W["o"].T


def mixer_attention(x, c, W, eps):
    n, H, G, d, e = x.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    pos = np.arange(n)
    q = rms_norm((x @ W["q"].T).reshape(n, H, d), W["q.norm"], eps)
    k = rms_norm((x @ W["k"].T).reshape(n, G, d), W["k.norm"], eps)
    v = (x @ W["v"].T).reshape(n, G, e)
    q, k = (rotate_half(t, pos, c["rot"]["base"], c["rot"]["dims"]) for t in (q, k))
    return chunked_attention(q, k, v, c["scale"], c["mask"]["size"]).reshape(n, H * e) @ W["o"].T


def mixer_linear_attention(x, c, W, eps):
    n, H, d, e = x.shape[0], c["heads"], c["dim"], c["vdim"]
    q, k = (silu(x @ W[t].T).reshape(n, H, d) for t in ("q", "k"))
    v = silu(x @ W["v"].T).reshape(n, H, e)
    o = decayed_linear_attention(q, k, v, c["decay"]).reshape(n, H * e)
    return (rms_norm(o, W["norm"], eps) * sigmoid(x @ W["g"].T)) @ W["o"].T


def mixer_parallel(x, c, W, eps):
    return (c["left_scale"] * mixer_attention(x, c["left"], _sub(W, "left."), eps) +
            c["right_scale"] * mixer_linear_attention(x, c["right"], _sub(W, "right."), eps))


# ---- feed-forwards -----------------------------------------------------------------------
def gated(x, W):
    return (silu(x @ W["gate"].T) * (x @ W["up"].T)) @ W["down"].T


def route(x, router, top):
    """The `top` experts of every token and the softmax over their logits."""
    z = x @ router.T
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=1)
    p = np.exp(zc - zc.max(axis=1, keepdims=True))
    return chosen, p / p.sum(axis=1, keepdims=True)


def mixture(x, top, W):
    chosen, p = route(x, W["router"], top)
    out = np.zeros_like(x)
    for e in range(W["router"].shape[0]):
        t, s = np.nonzero(chosen == e)
        if len(t):
            out[t] += p[t, s][:, None] * gated(x[t], _sub(W, f"e{e}."))
    return out


# ---- the model -------------------------------------------------------------------------
def forward(cfg, weights, tokens, taps=None):
    """Logits [tokens, vocab].  cfg: the parsed config.json; weights: name -> float array.
    taps: a list that receives the residual stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = weights["embed"][np.asarray(tokens)].astype(F)
    for i, L in enumerate(cfg["layers"]):
        W, mx = _sub(weights, f"l{i}."), _sub(weights, f"l{i}.mix.")
        y = {"delta": mixer_delta, "parallel": mixer_parallel}[L["type"]](x, L["mixer"], mx, eps)
        x = norm_after_sum(x, y, W["norm1"], alpha, eps)
        mlp = L["mlp"]
        if mlp is not None:
            ff = _sub(weights, f"l{i}.mlp.")
            y = gated(x, ff) if mlp["kind"] == "dense" else mixture(x, mlp["router"]["top"], ff)
            x = norm_after_sum(x, y, W["norm2"], alpha, eps)
        if taps is not None:
            taps.append(x.copy())
    return softcap(rms_norm(x, weights["final.norm"], eps) @ weights["head"].T, cfg["logit_softcap"])
