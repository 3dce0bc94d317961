"""Each mixed-layer operator alone against the oracle's equation for it: sizes that are not
multiples of a tile, portions of a sequence down to one token with the state carried between
them, several sequences in one call, and inputs built so that one far, first or border position
decides the result."""
import numpy as np
import pytest
import torch

import ternary_llm_b200 as tl
from oracle import mixed_oracle as O
from ternary_llm_b200 import mixed_ops as ops

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
REL = {"float32": 2e-5, "bfloat16": 6e-3}


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).cuda().to(dtype)


def rounded(a, dt):
    """The values the kernel sees."""
    return torch.from_numpy(np.asarray(a, np.float32)).to(DT[dt]).double().numpy()


def close(got, want, rel, what=""):
    got = got.double().cpu().numpy() if isinstance(got, torch.Tensor) else got
    assert np.isfinite(got).all(), what
    err = np.abs(got - want).max() / max(1e-3, np.abs(want).max())
    assert err <= rel, f"{what}: {err:.2e} > {rel:.0e}"


ACT = {None: lambda v: v, "silu": O.silu, "gelu_tanh": O.gelu_tanh}


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("rows", [1, 2, 3, 5, 8, 9, 64, 129, 300])
def test_dense_linear(rows, dt):
    rng = np.random.default_rng(rows)
    for n, k, act, glu, bias in ((100, 200, None, False, False), (33, 8, "silu", False, True), (1000, 1032, None, False, True),
                                 (72, 64, "gelu_tanh", True, False), (520, 136, "gelu_tanh", True, False)):
        x, w = rounded(rng.standard_normal((rows, k)), dt), rounded(rng.standard_normal((n * (2 if glu else 1), k)) * k ** -0.5, dt)
        b = rng.standard_normal(n).astype(np.float32) if bias else None
        y = torch.full((rows, n), float("nan"), device="cuda", dtype=DT[dt] if glu else torch.float32)
        ops.dense_linear(dev(x, DT[dt]), dev(w, DT[dt]), y, rows, n, k, bias=dev(b) if bias else None, act=act, glu=glu)
        p = x @ w.T
        want = ACT[act](p[:, :n]) * p[:, n:] if glu else ACT[act](p + (b if bias else 0))
        close(y, want, REL[dt] if glu else 2e-5, f"n={n} k={k} glu={glu}")
    tl.check_device_errors()


def cuts_of(n):
    """Ways to cut n tokens: whole, two at a time after an odd start, one by one at the end."""
    yield [n]
    odd = [5] + [2] * ((n - 5) // 2)
    yield odd + [n - sum(odd)] * (n > sum(odd))
    if n > 70:
        yield [1, 64, 1] + [1] * 3 + [n - 69]
    yield [n - 3, 1, 1, 1]


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_causal_conv(taps, dt):
    rng = np.random.default_rng(taps)
    n, C = 75, 40
    x = rounded(rng.standard_normal((2, n, C)), dt)
    w, b = rng.standard_normal((C, taps)).astype(np.float32), rng.standard_normal(C).astype(np.float32)
    for act in (None, "silu"):
        want = np.stack([ACT[act](O.causal_conv(x[s], w.astype(np.float64), b.astype(np.float64))) for s in range(2)])
        for cuts in cuts_of(n):
            state = torch.full((2, max(taps - 1, 1), C), float("nan"), device="cuda", dtype=DT[dt])   # a new sequence must not read it
            got, pos = [], 0
            for c in cuts:
                y = torch.empty(2, c, C, device="cuda", dtype=DT[dt])
                ops.causal_conv(dev(x[:, pos:pos + c], DT[dt]), dev(w), dev(b), state, y, C, taps, 2, c, pos, act)
                got.append(y)
                pos += c
            close(torch.cat(got, dim=1), want, REL[dt], f"cuts {cuts[:4]}")


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("states,channels", [(1, 24), (5, 40), (16, 24), (40, 8), (130, 24), (300, 8)])
def test_selective_scan(states, channels, dt):
    rng = np.random.default_rng(states)
    n, C, S = 150, channels, states
    s8 = (S + 7) // 8 * 8
    x, z = rounded(rng.standard_normal((2, n, C)), dt), rounded(rng.standard_normal((2, n, C)), dt)
    B, Cm = rounded(rng.standard_normal((2, n, S)), dt), rounded(rng.standard_normal((2, n, S)) * S ** -0.5, dt)
    t = rng.uniform(0.001, 0.3, (2, n, C)).astype(np.float32)
    A, D = -np.exp(rng.uniform(-5, 2, (C, S))).astype(np.float32), rng.standard_normal(C).astype(np.float32)
    x[:, 0] *= 8                                     # the first token must still be felt much later
    want = np.stack([O.selective_scan(x[s], t[s].astype(np.float64), A.astype(np.float64), B[s], Cm[s], D.astype(np.float64)) * O.silu(z[s])
                     for s in range(2)])
    bc = np.zeros((2, n, 2 * s8))
    bc[..., :S], bc[..., s8:s8 + S] = B, Cm
    a2 = dev(A.astype(np.float64) / np.log(2))
    for cuts in cuts_of(n):
        state = torch.full((2, C, S), float("nan"), device="cuda")
        got, pos = [], 0
        for c in cuts:
            p = slice(pos, pos + c)
            y = torch.empty(2, c, C, device="cuda", dtype=DT[dt])
            ops.selective_scan(dev(x[:, p], DT[dt]), dev(t[:, p]), dev(bc[:, p], DT[dt]), dev(z[:, p], DT[dt]), a2, dev(D), state, y, C, S,
                               2, c, pos)
            got.append(y)
            pos += c
        close(torch.cat(got, dim=1), want, REL[dt], f"cuts {cuts[:4]}")


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("channels,blocks", [(8, 1), (40, 5), (64, 2), (104, 13)])
def test_gated_scan(channels, blocks, dt):
    rng = np.random.default_rng(channels)
    n, C, m = 600, channels, channels // blocks
    u, y = rounded(rng.standard_normal((2, n, C)), dt), rounded(rng.standard_normal((2, n, C)), dt)
    r, i = rng.uniform(0.01, 1, (2, n, C)).astype(np.float32), rng.uniform(0, 1, (2, n, C)).astype(np.float32)
    lam = rng.uniform(-12, 1, C).astype(np.float32)     # decays from almost 1 (a cancelling 1 - a^2) to almost 0
    want = np.stack([O.gated_linear_recurrence(u[s], r[s].astype(np.float64), i[s].astype(np.float64), lam.astype(np.float64)) *
                     O.gelu_tanh(y[s]) for s in range(2)])
    gates = np.stack([r.reshape(2, n, blocks, m), i.reshape(2, n, blocks, m)], axis=3)
    soft = dev(O.softplus(lam.astype(np.float64)))
    for cuts in cuts_of(n):
        state = torch.full((2, C), float("nan"), device="cuda")
        got, pos = [], 0
        for c in cuts:
            p = slice(pos, pos + c)
            out = torch.empty(2, c, C, device="cuda", dtype=DT[dt])
            ops.gated_scan(dev(u[:, p], DT[dt]), dev(gates[:, p]), soft, dev(y[:, p], DT[dt]), state, out, C, blocks, 2, c, pos)
            got.append(out)
            pos += c
        close(torch.cat(got, dim=1), want, REL[dt], f"cuts {cuts[:4]}")


def attention_case(rng, n, ctx, H, rank, rot, hot, dt):
    """Queries and cache rows where each listed (query, position) pair has one score that stands
    out of all others of its query."""
    q = rng.standard_normal((n, H, rank + rot)) * 0.3
    c = rng.standard_normal((ctx, rank + rot)) * 0.3
    for qi, ki in hot:
        q[qi] += 6.0 * c[ki] / np.linalg.norm(c[ki]) * np.sqrt(rank + rot) / np.linalg.norm(c[ki])
    return rounded(q, dt), rounded(c, dt)


def plain_attention(q, k, v, scale, sink, start):
    """Queries at positions start.. over keys and values [positions, heads, .]."""
    H = q.shape[1]
    none = np.full(H, -1e30) if sink is None else sink
    pad = np.zeros((start,) + q.shape[1:])
    return O.sink_attention(np.concatenate([pad, q]), k, v, scale, none)[start:]


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("H,rank,rot", [(1, 8, 8), (3, 40, 8), (7, 56, 24), (20, 128, 0), (16, 512, 64), (4, 896, 128), (2, 1104, 8)])
def test_absorbed_attention(H, rank, rot, dt):
    """Edges: the first position, the borders of the 64-position tiles and of the splits, the
    query's own position, and the one after it (which must not be seen)."""
    rng = np.random.default_rng(rank)
    ctx = 330
    scale = (rank + rot) ** -0.5
    for n in (1, 2, 5):
        start = ctx - n
        hots = [0, 63, 64, 127, 128, 191, 192, 255, 256, start]
        for sink in (None, np.linspace(-2, 5, H)):
            hot = [(j % n, h) for j, h in enumerate(hots[:n])] if sink is None else [(0, hots[3]), (n - 1, 0)][:n]
            q, c = attention_case(rng, n, ctx, H, rank, rot, hot, dt)
            if n > 1:
                q[0] += 4.0 * c[start + 1]           # position after the first query: masked for it
                q = rounded(q, dt)
            k = np.repeat(c[:, None], H, axis=1)
            want = plain_attention(q, k, k[..., :rank], scale, sink, start)
            cache = torch.full((1, ctx + 9, rank + rot), float("nan"), device="cuda", dtype=DT[dt])   # unused rows must not be read
            cache[0, :ctx] = dev(c, DT[dt])
            o = torch.empty(n, H, rank, device="cuda", dtype=DT[dt])
            ops.latent_attention(dev(q, DT[dt]), cache, dev(sink) if sink is not None else None, o, H, rank, rot, scale, ctx + 9, 1, n, start)
            close(o, want, REL[dt], f"n={n} sink={sink is not None}")


@pytest.mark.parametrize("dt", list(DT))
def test_absorbed_attention_single_hot_positions_and_short_contexts(dt):
    rng = np.random.default_rng(9)
    H, rank, rot, ctx = 4, 32, 8, 200
    scale = 1.0
    for hot in (0, 1, 62, 63, 64, 65, 127, 128, 198, 199):
        q, c = attention_case(rng, 1, ctx, H, rank, rot, [(0, hot)], dt)
        k = np.repeat(c[:, None], H, axis=1)
        cache = dev(c, DT[dt])[None].contiguous()
        o = torch.empty(1, H, rank, device="cuda", dtype=DT[dt])
        ops.latent_attention(dev(q, DT[dt]), cache, None, o, H, rank, rot, scale, ctx, 1, 1, ctx - 1)
        want = plain_attention(q, k, k[..., :rank], scale, None, ctx - 1)
        assert np.abs(want - c[hot, :rank]).max() < 0.05 * np.abs(c[hot]).max()        # the case is what it says
        close(o, want, REL[dt], f"hot {hot}")
    for ctx in (1, 2, 3, 17):                                                           # the first tokens, with a strong sink
        q, c = attention_case(rng, ctx, ctx, H, rank, rot, [], dt)
        k, sink = np.repeat(c[:, None], H, axis=1), np.full(H, 3.0)
        o = torch.empty(ctx, H, rank, device="cuda", dtype=DT[dt])
        ops.latent_attention(dev(q, DT[dt]), dev(c, DT[dt])[None].contiguous(), dev(sink), o, H, rank, rot, scale, ctx, 1, ctx, 0)
        close(o, plain_attention(q, k, k[..., :rank], scale, sink, 0), REL[dt], f"ctx {ctx}")


@pytest.mark.parametrize("dt", list(DT))
def test_absorbed_attention_of_several_sequences_is_each_alone(dt):
    rng = np.random.default_rng(4)
    H, rank, rot, ctx, B = 5, 48, 16, 140, 6
    q = dev(rng.standard_normal((B, H, rank + rot)), DT[dt])
    cache = dev(rng.standard_normal((B, ctx, rank + rot)), DT[dt])
    o = torch.empty(B, H, rank, device="cuda", dtype=DT[dt])
    ops.latent_attention(q, cache, None, o, H, rank, rot, 0.2, ctx, B, 1, ctx - 1)
    for b in range(B):
        one = torch.empty(1, H, rank, device="cuda", dtype=DT[dt])
        ops.latent_attention(q[b:b + 1].contiguous(), cache[b:b + 1].contiguous(), None, one, H, rank, rot, 0.2, ctx, 1, 1, ctx - 1)
        close(o[b:b + 1], one.double().cpu().numpy(), REL[dt], f"sequence {b}")


@pytest.mark.parametrize("H,dim,rot,vdim", [(1, 8, 8, 8), (3, 24, 8, 40), (2, 40, 24, 72), (4, 128, 64, 128), (2, 64, 0, 256), (2, 200, 56, 24)])
def test_expanded_attention(H, dim, rot, vdim):
    rng = np.random.default_rng(dim)
    dt, rank = "bfloat16", 16
    scale = (dim + rot) ** -0.5
    for n, start in ((1, 0), (63, 0), (64, 1), (65, 64), (9, 200), (130, 77)):
        ctx = start + n
        k, v = rounded(rng.standard_normal((ctx, H, dim)), dt), rounded(rng.standard_normal((ctx, H, vdim)), dt)
        kr, q = rounded(rng.standard_normal((ctx, rot)), dt), rng.standard_normal((n, H, dim + rot))
        full = np.concatenate([k, np.repeat(kr[:, None], H, axis=1)], axis=2)
        for qi, ki in ((0, 0), (n - 1, 0), (n - 1, max(0, start - 1)), (n // 2, start + n // 2), (n - 1, min(63, ctx - 1)), (n - 1, min(64, ctx - 1))):
            q[qi] += 0.7 * full[ki]
        if n > 2:
            q[1] += 2.0 * full[start + 2]            # the next position, which it must not see
        q = rounded(q, dt)
        sink, gate = rng.standard_normal(H) * 2, rounded(rng.standard_normal((n, H)), dt)
        for s, g in ((None, None), (sink, gate)):
            want = plain_attention(q, full, v, scale, s, start)
            if g is not None:
                want = want * O.sigmoid(g)[:, :, None]
            cache = torch.full((ctx + 3, rank + rot), float("nan"), device="cuda", dtype=torch.bfloat16)
            cache[:ctx, rank:] = dev(kr, torch.bfloat16)
            o = torch.empty(n, H, vdim, device="cuda", dtype=torch.bfloat16)
            ops.latent_attention_expanded(dev(q, torch.bfloat16), dev(k, torch.bfloat16), dev(v, torch.bfloat16), cache,
                                          dev(s) if s is not None else None, dev(g, torch.bfloat16) if g is not None else None, o, H, dim, rot,
                                          vdim, rank, scale, ctx + 3, n, start)
            close(o, want, REL[dt], f"n={n} start={start} sink={s is not None}")


def test_operators_refuse_short_tensors():
    x = torch.zeros(2, 16, device="cuda")
    with pytest.raises(ValueError, match="holds"):
        ops.dense_linear(x, torch.zeros(3, 16, device="cuda"), torch.zeros(2, 4, device="cuda"), 2, 4, 16)
    with pytest.raises(TypeError):
        ops.dense_linear(x.half(), x.half(), x, 2, 2, 16)
