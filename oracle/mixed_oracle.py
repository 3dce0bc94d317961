"""CPU restatement (numpy, float64) of the decoder built from a list of mixer layers (Petulix).

TEST INFRASTRUCTURE ONLY: imported by tests/ and smoke().  One function per mechanism, each
the plain equation evaluated token by token; nothing is shared with the shipped package.
Every function takes and returns arrays with one row per token.
"""
from __future__ import annotations

import math

import numpy as np

F = np.float64


# ---- element-wise pieces ---------------------------------------------------------------
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def rotate_half(x, positions, base, dims):
    """x [tokens, ..., n]; the first `dims` entries of the last axis turn by position * base^(-2i/dims),
    entry i paired with entry i + dims/2; the rest pass."""
    out = np.array(x, dtype=F)
    hd = dims // 2
    for i in range(hd):
        a = np.asarray(positions, F) * F(base) ** (-2.0 * i / dims)
        a = a.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., i], x[..., i + hd]
        out[..., i] = u * np.cos(a) - v * np.sin(a)
        out[..., i + hd] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_conv(x, w, b):
    """Per channel: y_t = b + sum_j w[:, j] x_{t - taps + 1 + j}, zeros before the first token."""
    n, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x) + b
    for t in range(n):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


# ---- recurrences -----------------------------------------------------------------------
def selective_scan(x, dt, A, B, C, D):
    """x, dt [tokens, channels]; A [channels, states]; B, C [tokens, states]; D [channels]."""
    S = np.zeros(A.shape, F)
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def gated_linear_recurrence(u, r, i, lam, c=8.0):
    """a = exp(-c r softplus(lam)); S <- a S + sqrt(1 - a^2) i u."""
    S = np.zeros(u.shape[1], F)
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -c * r[t] * softplus(lam)
        a = np.exp(log_a)
        S = a * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def block_linear(u, w, b):
    """u [tokens, blocks * m] times a block-diagonal matrix w [blocks, m, m] ([out, in]) plus b."""
    nb, m = w.shape[0], w.shape[1]
    out = np.zeros((u.shape[0], nb * m), F)
    for k in range(nb):
        out[:, k * m:(k + 1) * m] = u[:, k * m:(k + 1) * m] @ w[k].T + b[k]
    return out


# ---- attention -------------------------------------------------------------------------
def sink_attention(q, k, v, scale, sink):
    """q [tokens, heads, d], k [tokens, heads, d], v [tokens, heads, e]: causal softmax whose
    denominator also holds exp(sink[head])."""
    n, H = q.shape[0], q.shape[1]
    out = np.zeros((n, H, v.shape[2]), F)
    for h in range(H):
        for t in range(n):
            s = (k[:t + 1, h] @ q[t, h]) * scale
            m = max(s.max(), sink[h])
            p = np.exp(s - m)
            out[t, h] = (p @ v[:t + 1, h]) / (p.sum() + math.exp(sink[h] - m))
    return out


# ---- mixers (h: the normalised input of the layer, one row per token) ------------------
def mixer_mamba1(h, c, W):
    inner, st, dr = c["inner"], c["state"], c["dt_rank"]
    xz = h @ W["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, W["conv"], W["conv.b"]))
    p = x @ W["x"].T
    dt = softplus(p[:, :dr] @ W["dt"].T + W["dt.b"])
    y = selective_scan(x, dt, -np.exp(W["A_log"]), p[:, dr:dr + st], p[:, dr + st:], W["D"])
    return (y * silu(z)) @ W["o"].T


def mixer_rglru(h, c, W):
    y = gelu_tanh(h @ W["y"].T + W["y.b"])
    u = causal_conv(h @ W["x"].T + W["x.b"], W["conv"], W["conv.b"])
    r = sigmoid(block_linear(u, W["ra"], W["ra.b"]))
    i = sigmoid(block_linear(u, W["ri"], W["ri.b"]))
    return (gated_linear_recurrence(u, r, i, W["lam"]) * y) @ W["o"].T


def mixer_latent_attention(h, c, W, eps):
    n, H, d, rd, e, R = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = np.arange(n)
    q = (h @ W["q"].T).reshape(n, H, d + rd)
    kv = h @ W["dkv"].T
    lat = rms_norm(kv[:, :R], W["dkv.norm"], eps)
    qr = rotate_half(q[:, :, d:], pos, c["rot"]["base"], c["rot"]["dims"])
    kr = rotate_half(kv[:, R:], pos, c["rot"]["base"], c["rot"]["dims"])
    k = (lat @ W["uk"].T).reshape(n, H, d)
    v = (lat @ W["uv"].T).reshape(n, H, e)
    q = np.concatenate([q[:, :, :d], qr], axis=2)
    k = np.concatenate([k, np.repeat(kr[:, None, :], H, axis=1)], axis=2)
    out = sink_attention(q, k, v, c["scale"], W["sink"])
    out = out * sigmoid(h @ W["g"].T)[:, :, None]
    return out.reshape(n, H * e) @ W["o"].T


def feed_forward(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


# ---- the model -------------------------------------------------------------------------
def run_order(cfg):
    """[(layer index, first layer of a repeated pass)] in execution order."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(lp["start"])]
    for p in range(lp["times"]):
        for i in range(lp["start"], lp["stop"]):
            order.append((i, p > 0 and i == lp["start"]))
    return order + [(i, False) for i in range(lp["stop"], n)]


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, taps=None):
    """Logits [tokens, vocab].  cfg: the parsed config.json; weights: name -> float array.
    taps: a list that receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    emb = weights["embed"][np.asarray(tokens)].astype(F)
    x = emb.copy()
    for i, again in run_order(cfg):
        L = cfg["layers"][i]
        if again:
            x = x + emb
        W, mx = _sub(weights, f"l{i}."), _sub(weights, f"l{i}.mix.")
        h = rms_norm(x, W["norm1"], eps)
        if L["type"] == "mamba1":
            y = mixer_mamba1(h, L["mixer"], mx)
        elif L["type"] == "rglru":
            y = mixer_rglru(h, L["mixer"], mx)
        elif L["type"] == "latent_attention":
            y = mixer_latent_attention(h, L["mixer"], mx, eps)
        else:
            raise ValueError(L["type"])
        x = x + rms_norm(y, W["norm1b"], eps)
        if L["mlp"] is not None:
            y = feed_forward(rms_norm(x, W["norm2"], eps), _sub(weights, f"l{i}.mlp."))
            x = x + rms_norm(y, W["norm2b"], eps)
        if taps is not None:
            taps.append(x.copy())
    return rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T
