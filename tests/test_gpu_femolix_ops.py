"""The operators of the Femolix design alone against the oracle's equation for each: sizes that are
not multiples of a tile, portions down to one token with cache or state carried between them,
several sequences in one call, and inputs built so that one far, first or border position decides
the result."""
import numpy as np
import pytest
import torch

import ternary_llm_b200 as tl
from oracle import femolix_oracle as O
from oracle.mixed_oracle import rms_norm, rotate_half, sigmoid, silu, softplus
from tests.test_gpu_mixed_ops import DT, close, dev, rounded
from ternary_llm_b200 import mixed_ops as ops

pytestmark = pytest.mark.gpu
REL = {"float32": 2e-5, "bfloat16": 1e-2}


def portions(n):
    """Ways to cut n tokens: whole; two at a time after an odd start; one by one; the end token by token."""
    yield [n]
    yield [5] + [2] * ((n - 5) // 2) + [1] * ((n - 5) % 2)
    yield [n - 3, 1, 1, 1]
    if n > 130:
        yield [1, 64, 1, 2, 60, n - 128]
    if n <= 40:
        yield [1] * n


# ---- grouped attention ---------------------------------------------------------------------
def rope_table(n, base, dims):
    a = np.arange(n)[:, None] * np.float64(base) ** (-2.0 * np.arange(dims // 2) / dims)
    return torch.from_numpy(np.stack([np.cos(a), np.sin(a)], axis=-1).astype(np.float32)).cuda()


def attend(x, qn, kn, eps, base, rot, scale, chunk, H, G, d, e):
    """The oracle on the projected rows x [tokens, q | k | v]."""
    n = len(x)
    q, k, v = x[:, :H * d].reshape(n, H, d), x[:, H * d:(H + G) * d].reshape(n, G, d), x[:, (H + G) * d:].reshape(n, G, e)
    if qn is not None:
        q, k = rms_norm(q, qn, eps), rms_norm(k, kn, eps)
    if rot:
        q, k = rotate_half(q, np.arange(n), base, rot), rotate_half(k, np.arange(n), base, rot)
    return O.chunked_attention(q, k, v, scale, chunk).reshape(n, H * e)


CASES = [  # heads, kv heads, dim, vdim, rotated, chunk, tokens, cache rows (0: all), norms
    (4, 2, 24, 40, 8, 50, 210, 0, True), (3, 3, 8, 8, 8, 64, 150, 0, True), (8, 1, 64, 32, 32, 33, 140, 180, True), (5, 5, 16, 72, 0, 0, 90, 0, False),
    (12, 1, 40, 16, 40, 7, 100, 0, True), (2, 1, 128, 136, 64, 1, 20, 0, True), (2, 2, 136, 264, 16, 100, 150, 0, True), (16, 2, 32, 64, 2, 65, 131, 0, True)]


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("case", CASES, ids=[f"{c[0]}x{c[1]}x{c[2]}x{c[3]}c{c[5]}" for c in CASES])
def test_grouped_attention(case, dt):
    H, G, d, e, rot, chunk, n, ring, norms = case
    rng = np.random.default_rng(d + e)
    x = rounded(rng.standard_normal((2, n, H * d + G * (d + e))), dt)
    qn, kn = (rng.uniform(0.5, 2, d), rng.uniform(0.5, 2, d)) if norms else (None, None)
    qn, kn = (a if a is None else a.astype(np.float32).astype(np.float64) for a in (qn, kn))
    scale, rows = 3.0 * d ** -0.5, ring or n
    want = np.stack([0.6 * attend(s, qn, kn, 1e-5, 300.0, rot, scale, chunk, H, G, d, e) for s in x])
    rope = rope_table(n, 300.0, rot) if rot else None
    for cuts in portions(n):
        if ring and max(cuts) > ring - chunk:
            continue
        kc = torch.full((2, rows, G * d), float("nan"), device="cuda", dtype=DT[dt])     # what was not written must not be read
        vc = torch.full((2, rows, G * e), float("nan"), device="cuda", dtype=DT[dt])
        got, pos = [], 0
        for c in cuts:
            o = torch.full((2, c, H * e), float("nan"), device="cuda", dtype=DT[dt])
            ops.grouped_attention(dev(x[:, pos:pos + c], DT[dt]), dev(qn) if norms else None, dev(kn) if norms else None, 1e-5, rope, rot, kc, vc, o,
                                  H, G, d, e, chunk, rows, n, scale, 2, c, pos, out_scale=0.6)
            got.append(o)
            pos += c
        close(torch.cat(got, dim=1), want, 3e-5 if dt == "float32" else 2e-2, f"cuts {cuts[:4]}")


@pytest.mark.parametrize("d,e", [(64, 64), (64, 128), (128, 64), (128, 128)])
@pytest.mark.parametrize("chunk,ring", [(0, 0), (100, 0), (128, 512), (300, 768), (1, 0)])
def test_grouped_attention_over_long_prompts(chunk, ring, d, e):
    """Head sizes and lengths of the tensor-memory kernel: portions of 128 tokens and more from
    positions inside a tile, chunks of every alignment, a ring of cache rows, a sharp softmax whose
    maximum keeps growing."""
    H, G, n = 4, 2, 700
    rng = np.random.default_rng(chunk + d)
    x = rounded(rng.standard_normal((1, n, H * d + G * (d + e))), "bfloat16")
    x[0, :, H * d:(H + G) * d] *= np.linspace(0.2, 3.0, n)[:, None]           # scores grow along the sequence
    x = rounded(x, "bfloat16")
    scale, rows = 4.0 * d ** -0.5, ring or n
    want = attend(x[0], None, None, 1e-5, 300.0, 32, scale, chunk, H, G, d, e)[None]
    for cuts in ([700], [128, 130, 442], [5, 300, 200, 195], [130, 1, 1, 568]):
        if ring and max(cuts) > ring - chunk:
            continue
        kc = torch.full((1, rows, G * d), float("nan"), device="cuda", dtype=torch.bfloat16)
        vc = torch.full((1, rows, G * e), float("nan"), device="cuda", dtype=torch.bfloat16)
        got, pos = [], 0
        for c in cuts:
            o = torch.full((1, c, H * e), float("nan"), device="cuda", dtype=torch.bfloat16)
            ops.grouped_attention(dev(x[:, pos:pos + c], torch.bfloat16), None, None, 1e-5, rope_table(n, 300.0, 32), 32, kc, vc, o, H, G, d, e, chunk,
                                  rows, n, scale, 1, c, pos)
            got.append(o)
            pos += c
        close(torch.cat(got, dim=1), want, 2e-2, f"cuts {cuts}")
    tl.check_device_errors()


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("chunk", [0, 190])
@pytest.mark.parametrize("d", [16, 64])
def test_grouped_attention_finds_one_key_just_inside_and_never_outside(dt, chunk, d):
    """One key matches the query of every position; its value is the output exactly where the mask
    shows it: from its own position to the end of its chunk."""
    H, G, e, n = 2, 1, {16: 8, 64: 64}[d], 470
    for at in (0, 63, 64, 189, 190, 379):
        x = np.zeros((1, n, H * d + G * (d + e)))
        x[..., d - 1:H * d:d] = 1.0
        x[:, :, H * d] = 1.0                                     # every other key: orthogonal to the queries
        x[:, at, H * d], x[:, at, H * d + d - 1] = 0.0, 1.0
        x[:, at, (H + G) * d:] = 5.0
        # decode: the last positions one by one, from just before the next chunk's edge
        for cuts in ([n], [370] + [1] * 100, [180] + [1] * 25 + [265]):
            kc, vc = (torch.zeros(1, n, w, device="cuda", dtype=DT[dt]) for w in (d, e))
            got, pos = [], 0
            for c in cuts:
                o = torch.empty(1, c, H * e, device="cuda", dtype=DT[dt])
                ops.grouped_attention(dev(x[:, pos:pos + c], DT[dt]), None, None, 1e-5, None, 0, kc, vc, o, H, G, d, e, chunk, n, n, 30.0, 1, c, pos)
                got.append(o)
                pos += c
            got = torch.cat(got, dim=1)[0].float().cpu().numpy()
            end = (at // chunk + 1) * chunk if chunk else n
            seen = np.zeros(n, bool)
            seen[at:end] = True
            assert np.allclose(got[seen], 5.0, atol=1e-2) and np.allclose(got[~seen], 0.0, atol=1e-6), f"key {at} cuts {cuts[:2]}"


# ---- matrix recurrences ------------------------------------------------------------------------
@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("heads,dim,vdim", [(3, 8, 8), (2, 24, 40), (4, 64, 32), (1, 16, 136), (2, 128, 64), (1, 200, 24), (1, 264, 16)])
def test_linear_attention(heads, dim, vdim, dt):
    rng = np.random.default_rng(dim)
    n, H = 203, heads
    qkv = rounded(rng.standard_normal((2, n, H * (2 * dim + vdim))) * np.repeat([dim ** -0.5, 1.0], [2 * H * dim, H * vdim]), dt)
    qkv[:, 0] *= 4                                                # the first token must still be felt much later
    decay = np.linspace(0.9997, 0.2, H).astype(np.float32)
    want = []
    for s in qkv:
        q, k, v = s[:, :H * dim].reshape(n, H, dim), s[:, H * dim:2 * H * dim].reshape(n, H, dim), s[:, 2 * H * dim:].reshape(n, H, vdim)
        want.append(O.decayed_linear_attention(q, k, v, decay.astype(np.float64)).reshape(n, -1))
    want = np.stack(want)
    for cuts in portions(n):
        state = torch.full((2, H, vdim, dim), float("nan"), device="cuda")
        got, pos = [], 0
        for c in cuts:
            o = torch.full((2, c, H * vdim), float("nan"), device="cuda")
            ops.linear_attention(dev(qkv[:, pos:pos + c], DT[dt]), dev(decay), state, o, H, dim, vdim, 2, c, pos)
            got.append(o)
            pos += c
        close(torch.cat(got, dim=1), want, 2e-5 if dt == "float32" else 3e-4, f"cuts {cuts[:4]}")


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(2, 1, 8, 16), (4, 2, 24, 40), (3, 3, 64, 32), (2, 2, 16, 136), (4, 1, 128, 64), (1, 1, 200, 24),
                                                     (1, 1, 264, 16)])
def test_delta_rule(heads, kv_heads, dim, vdim, dt):
    """Inputs enter the recurrence without rounding: only the products' own rounding remains."""
    rng = np.random.default_rng(dim + 1)
    n, H, G = 203, heads, kv_heads
    qkv = rounded(rng.standard_normal((2, n, 2 * G * dim + H * vdim)), dt)
    base = rng.standard_normal((G, dim))
    qkv[..., G * dim:2 * G * dim] = rounded(qkv[..., G * dim:2 * G * dim] + 1.5 * base.reshape(-1), dt)    # keys that overlap
    a, b = rng.standard_normal((2, n, H)).astype(np.float32), 2 * rng.standard_normal((2, n, H)).astype(np.float32)
    neg_a, bias = -np.geomspace(1e-4, 3.0, H).astype(np.float32), rng.standard_normal(H).astype(np.float32)
    want = []
    for s in range(2):
        q, k = (O.unit(qkv[s][:, i * G * dim:(i + 1) * G * dim].reshape(n, G, dim)).repeat(H // G, axis=1) for i in (0, 1))
        g = np.exp(neg_a.astype(np.float64) * softplus(a[s].astype(np.float64) + bias))
        v = qkv[s][:, 2 * G * dim:].reshape(n, H, vdim)
        want.append(O.delta_rule(0.3 * q, k, v, g, sigmoid(b[s].astype(np.float64))).reshape(n, -1))
    want = np.stack(want)
    for cuts in portions(n):
        state = torch.full((2, H, vdim, dim), float("nan"), device="cuda")
        got, pos = [], 0
        for c in cuts:
            o = torch.full((2, c, H * vdim), float("nan"), device="cuda")
            p = slice(pos, pos + c)
            ops.delta_rule(dev(qkv[:, p], DT[dt]), dev(a[:, p]), dev(b[:, p]), dev(neg_a), dev(bias), 0.3, state, o, H, G, dim, vdim, 2, c, pos)
            got.append(o)
            pos += c
        close(torch.cat(got, dim=1), want, 2e-5 if dt == "float32" else 3e-4, f"cuts {cuts[:4]}")


@pytest.mark.parametrize("dt", list(DT))
def test_delta_rule_returns_what_was_written_far_back(dt):
    """Without decay and with orthogonal keys a value written once is read back any time later, until its
    key is written again: positions around the borders of 64 tokens."""
    n, d, e = 400, 32, 8
    for at in (0, 62, 63, 64, 127, 128):
        qkv = np.zeros((1, n, 2 * d + e))
        qkv[:, :, d + 1] = 1.0                                    # all other tokens write under key 1
        qkv[:, at, d + 1], qkv[:, at, d + 2], qkv[:, at, 2 * d:] = 0.0, 1.0, 7.0
        qkv[:, :, 2] = 1.0                                        # every query asks for key 2
        qkv[:, 300, d + 1], qkv[:, 300, d + 2], qkv[:, 300, 2 * d:] = 0.0, 1.0, -2.0
        a, b = np.full((1, n, 1), -60.0), np.full((1, n, 1), 40.0)
        want = np.zeros((n, e))
        want[at:], want[300:] = 7.0, -2.0
        for cuts in ([n], [at + 1] + [1] * 5 + [n - at - 6], [290] + [1] * 30 + [80]):
            state = torch.zeros(1, 1, e, d, device="cuda")
            got, pos = [], 0
            for c in cuts:
                o, p = torch.empty(1, c, e, device="cuda"), slice(pos, pos + c)
                ops.delta_rule(dev(qkv[:, p], DT[dt]), dev(a[:, p]), dev(b[:, p]), dev(-np.ones(1)), dev(np.zeros(1)), 1.0, state, o, 1, 1, d, e, 1, c,
                               pos)
                got.append(o[0])
                pos += c
            assert np.abs(torch.cat(got).cpu().numpy() - want).max() < 1e-3, f"written at {at}, cuts {cuts[:2]}"


@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("rows,groups,n,act", [(1, 1, 8, "silu"), (3, 5, 24, "silu"), (9, 1, 1000, "sigmoid"), (2, 40, 128, "sigmoid"), (70, 3, 136, "silu")])
def test_gated_norm(rows, groups, n, act, dt):
    rng = np.random.default_rng(n)
    o, w = rng.standard_normal((rows, groups, n)).astype(np.float32), rng.standard_normal(n).astype(np.float32)
    z = rounded(rng.standard_normal((rows, groups, n)), dt)
    want = 0.7 * rms_norm(o.astype(np.float64), w, 1e-3) * {"silu": silu, "sigmoid": sigmoid}[act](z)
    out = torch.empty(rows, groups, n, device="cuda", dtype=DT[dt])
    ops.gated_norm(dev(o), dev(w), dev(z, DT[dt]), out, rows, groups, n, 1e-3, act, 0.7)
    close(out, want, REL[dt])


# ---- experts -------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", list(DT))
@pytest.mark.parametrize("n,top,ff,width", [(4, 1, 24, 40), (8, 3, 40, 72), (5, 5, 8, 16), (70, 6, 16, 24), (1, 1, 136, 64)])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 130, 700])
def test_experts(rows, n, top, ff, width, dt):
    rng = np.random.default_rng(rows + n)
    h, z = rounded(rng.standard_normal((rows, width)), dt), 2 * rng.standard_normal((rows, n)).astype(np.float32)
    if rows > 9:
        z[:, 0] += 4                                              # one expert that nearly all tokens choose
    gu, dn = rounded(rng.standard_normal((n, 2 * ff, width)) * width ** -0.5, dt), rounded(rng.standard_normal((n, width, ff)) * ff ** -0.5, dt)
    W = {"router": np.eye(n)}
    want = np.zeros((rows, width))
    chosen, p = O.route(z.astype(np.float64), W["router"], top)
    for t in range(rows):
        for s, e in enumerate(chosen[t]):
            want[t] += p[t, s] * O.gated(h[t:t + 1], {"gate": gu[e, :ff], "up": gu[e, ff:], "down": dn[e]})[0]
    for _ in range(2):                                            # the second call meets the first one's leftovers
        y = torch.full((rows, width), float("nan"), device="cuda")
        ops.experts(dev(h, DT[dt]), dev(z), dev(gu, DT[dt]), dev(dn, DT[dt]), y, rows, width, ff, n, top)
        close(y, want, REL[dt], f"rows={rows}")
    tl.check_device_errors()


def test_equal_router_logits_choose_the_lower_index():
    rows, n, top, ff, width = 20, 6, 2, 8, 16
    rng = np.random.default_rng(0)
    h, z = rng.standard_normal((rows, width)), np.zeros((rows, n))
    z[::2, 4] = 1.0
    gu, dn = rng.standard_normal((n, 2 * ff, width)) * 0.3, rng.standard_normal((n, width, ff)) * 0.3
    want = np.zeros((rows, width))
    for t in range(rows):
        es = [4, 0] if t % 2 == 0 else [0, 1]
        p = np.exp(z[t, es]) / np.exp(z[t, es]).sum()
        want[t] = sum(p[i] * O.gated(h[t:t + 1], {"gate": gu[e, :ff], "up": gu[e, ff:], "down": dn[e]})[0] for i, e in enumerate(es))
    for m in (1, 4, 20):
        y = torch.empty(m, width, device="cuda")
        ops.experts(dev(h[:m]), dev(z[:m]), dev(gu), dev(dn), y, m, width, ff, n, top)
        close(y, want[:m], 2e-5)
