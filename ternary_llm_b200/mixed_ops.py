"""Host-side mirror of the mixed-layer operators (include/tllm_b200_mixed.h) on torch tensors:
shape, dtype and device checks, then one call of the C ABI on torch's current stream.  The
activation type (bfloat16 or float32) is that of the first tensor; nothing here computes with
torch operations.
"""
from __future__ import annotations

import torch

from . import _lib
from .mixed import ACTIVATIONS
from .ops import _chk, _stream

_F = torch.float32


def _kind(t) -> int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"activations must be bfloat16 or float32, got {t.dtype}")
    return 1 if t.dtype == torch.bfloat16 else 0


def _opt(t, dtype, name, numel):
    return None if t is None else _chk(t, dtype, name, numel)


def dense_linear(x, w, y, rows: int, n: int, cols: int, bias=None, act=None, glu: bool = False) -> None:
    """y = act(x @ w.T + bias) in FP32; glu: w holds n gate rows, then n up rows, and
    y = act(gate) * up in the activation type."""
    d = x.dtype
    _lib.check(_lib.lib().tllm_b200_dense_linear(
        _kind(x), _chk(x, d, "x", rows * cols), _chk(w, d, "w", n * cols * (2 if glu else 1)), _opt(bias, _F, "bias", n),
        _chk(y, d if glu else _F, "y", rows * n), rows, n, cols, ACTIVATIONS[act], int(glu), _stream()))


def causal_conv(x, w, bias, state, y, channels: int, taps: int, n_seq: int, seq_len: int, start_pos: int, act=None) -> None:
    """Causal convolution per channel; state [n_seq, taps - 1, channels] carries the last inputs."""
    d, rows = x.dtype, n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_causal_conv(
        _kind(x), _chk(x, d, "x", rows * channels), _chk(w, _F, "w", channels * taps), _opt(bias, _F, "bias", channels),
        _opt(state, d, "state", n_seq * (taps - 1) * channels), _chk(y, d, "y", rows * channels), channels, taps,
        ACTIVATIONS[act], n_seq, seq_len, start_pos, _stream()))


def selective_scan(x, dt, bc, z, a2, d, state, y, channels: int, states: int, n_seq: int, seq_len: int, start_pos: int) -> None:
    """S = exp(dt A) S + dt x B, y = (S . C + D x) silu(z); a2 = A / ln 2, bc rows hold B then C,
    each padded to a multiple of 8; state [n_seq, channels, states]."""
    t, rows, ld = x.dtype, n_seq * seq_len, 2 * ((states + 7) // 8 * 8)
    _lib.check(_lib.lib().tllm_b200_selective_scan(
        _kind(x), _chk(x, t, "x", rows * channels), _chk(dt, _F, "dt", rows * channels), _chk(bc, t, "bc", rows * ld),
        _opt(z, t, "z", rows * channels), _chk(a2, _F, "a2", channels * states), _opt(d, _F, "d", channels),
        _chk(state, _F, "state", n_seq * channels * states), _chk(y, t, "y", rows * channels), channels, states, n_seq, seq_len,
        start_pos, _stream()))


def gated_scan(u, gates, soft_lam, y, state, out, channels: int, blocks: int, n_seq: int, seq_len: int, start_pos: int,
               decay: float = 8.0, act="gelu_tanh") -> None:
    """log a = -decay r softplus(lam), S = a S + sqrt(1 - a^2) i u, out = S act(y); gates
    [rows, blocks, 2, channels / blocks] = r, then i; soft_lam = softplus(lam)."""
    t, rows = u.dtype, n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_gated_scan(
        _kind(u), _chk(u, t, "u", rows * channels), _chk(gates, _F, "gates", rows * 2 * channels), _chk(soft_lam, _F, "soft_lam", channels),
        _chk(y, t, "y", rows * channels), _chk(state, _F, "state", n_seq * channels), _chk(out, t, "out", rows * channels), channels,
        blocks, decay, ACTIVATIONS[act], n_seq, seq_len, start_pos, _stream()))


def latent_attention(q, cache, sink, o, heads: int, rank: int, rot: int, scale: float, max_seq: int, n_seq: int, seq_len: int,
                     start_pos: int) -> None:
    """Absorbed latent attention: q [rows, heads, rank + rot], cache [n_seq, max_seq, rank + rot],
    o [rows, heads, rank]."""
    t, rows = q.dtype, n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_latent_attention(
        _kind(q), _chk(q, t, "q", rows * heads * (rank + rot)), _chk(cache, t, "cache", n_seq * max_seq * (rank + rot)),
        _opt(sink, _F, "sink", heads), _chk(o, t, "o", rows * heads * rank), heads, rank, rot, scale, max_seq, n_seq, seq_len,
        start_pos, _stream()))


def latent_attention_expanded(q, kx, vx, cache, sink, gate, o, heads: int, dim: int, rot: int, vdim: int, rank: int, scale: float,
                              max_seq: int, seq_len: int, start_pos: int) -> None:
    """Latent attention of one sequence over expanded keys and values (BF16)."""
    t, ctx = torch.bfloat16, start_pos + seq_len
    _lib.check(_lib.lib().tllm_b200_latent_attention_expanded(
        _chk(q, t, "q", seq_len * heads * (dim + rot)), _chk(kx, t, "kx", ctx * heads * dim), _chk(vx, t, "vx", ctx * heads * vdim),
        _chk(cache, t, "cache", max_seq * (rank + rot)), _opt(sink, _F, "sink", heads), _opt(gate, t, "gate", seq_len * heads),
        _chk(o, t, "o", seq_len * heads * vdim), heads, dim, rot, vdim, rank, scale, max_seq, seq_len, start_pos, _stream()))


def grouped_attention(proj, q_norm, k_norm, eps: float, rope, rot_dims: int, kc, vc, o, heads: int, kv_heads: int, dim: int, vdim: int,
                      chunk: int, cache_rows: int, max_seq: int, scale: float, n_seq: int, seq_len: int, start_pos: int,
                      out_scale: float = 1.0) -> None:
    """Per-head norms, rotation, cache append and attention of a step; proj [rows, q | k | v]
    (q is overwritten), rope [max_seq, rot_dims / 2, 2] = cos, sin, caches [n_seq, cache_rows, ..]."""
    t, rows = proj.dtype, n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_grouped_attention(
        _kind(proj), _chk(proj, t, "proj", rows * (heads * dim + kv_heads * (dim + vdim))), _opt(q_norm, _F, "q_norm", dim),
        _opt(k_norm, _F, "k_norm", dim), eps, _opt(rope, _F, "rope", max_seq * rot_dims), rot_dims,
        _chk(kc, t, "kc", n_seq * cache_rows * kv_heads * dim), _chk(vc, t, "vc", n_seq * cache_rows * kv_heads * vdim),
        _chk(o, t, "o", rows * heads * vdim), heads, kv_heads, dim, vdim, chunk, cache_rows, max_seq, scale, out_scale, n_seq, seq_len,
        start_pos, _stream()))


def linear_attention(qkv, decay, state, o, heads: int, dim: int, vdim: int, n_seq: int, seq_len: int, start_pos: int) -> None:
    """S_t = decay S_(t-1) + v k', o = S_t q; qkv [rows, q | k | v], state [n_seq, heads, vdim, dim]."""
    rows = n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_matrix_scan(
        _kind(qkv), 0, _chk(qkv, qkv.dtype, "qkv", rows * heads * (2 * dim + vdim)), _chk(decay, _F, "decay", heads), None, None, None, None, 1.0,
        _chk(state, _F, "state", n_seq * heads * dim * vdim), _chk(o, _F, "o", rows * heads * vdim), heads, heads, dim, vdim, n_seq, seq_len,
        start_pos, _stream()))


def delta_rule(qkv, a, b, neg_a, dt_bias, q_scale: float, state, o, heads: int, kv_heads: int, dim: int, vdim: int, n_seq: int, seq_len: int,
               start_pos: int) -> None:
    """S_t = g S_(t-1) + beta (v - g S_(t-1) k) k', o = S_t q with unit-length q (times q_scale)
    and k, g = exp(neg_a softplus(a + dt_bias)), beta = sigmoid(b)."""
    rows = n_seq * seq_len
    _lib.check(_lib.lib().tllm_b200_matrix_scan(
        _kind(qkv), 1, _chk(qkv, qkv.dtype, "qkv", rows * (2 * kv_heads * dim + heads * vdim)), None, _chk(a, _F, "a", rows * heads),
        _chk(b, _F, "b", rows * heads), _chk(neg_a, _F, "neg_a", heads), _chk(dt_bias, _F, "dt_bias", heads), q_scale,
        _chk(state, _F, "state", n_seq * heads * dim * vdim), _chk(o, _F, "o", rows * heads * vdim), heads, kv_heads, dim, vdim, n_seq, seq_len,
        start_pos, _stream()))


def gated_norm(o, w, gate, out, rows: int, groups: int, n: int, eps: float, act="silu", out_scale: float = 1.0) -> None:
    """out = out_scale * o / rms(o) * w * act(gate), the norm over each group of n entries."""
    t = gate.dtype
    _lib.check(_lib.lib().tllm_b200_gated_norm(
        _kind(gate), _chk(o, _F, "o", rows * groups * n), _chk(w, _F, "w", n), _chk(gate, t, "gate", rows * groups * n),
        _chk(out, t, "out", rows * groups * n), rows, groups, n, eps, out_scale, ACTIVATIONS[act], _stream()))


def experts(h, z, gate_up, down, y, rows: int, width: int, ff: int, n: int, top: int, act="silu") -> None:
    """Weighted sum of the outputs of the `top` experts with the largest z, softmax over them."""
    t = h.dtype
    _lib.check(_lib.lib().tllm_b200_experts(
        _kind(h), _chk(h, t, "h", rows * width), _chk(z, _F, "z", rows * n), _chk(gate_up, t, "gate_up", n * 2 * ff * width),
        _chk(down, t, "down", n * width * ff), _chk(y, _F, "y", rows * width), rows, width, ff, n, top, ACTIVATIONS[act], _stream()))
