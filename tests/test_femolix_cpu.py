"""The Femolix design, what needs no GPU: the oracle's mechanisms against independent forms of the
same equations, the sensitivity of the comparison to mistakes, loading and its refusals."""
import ctypes
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import femolix_oracle as O
from tests import _femolix as X
from tests.test_mixed_cpu import write_model
from ternary_llm_b200 import _lib, mixed, models

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- the oracle against other forms of the same equations ------------------------------
def test_delta_rule_is_a_triangular_system():
    rng = np.random.default_rng(0)
    n, H, d, e = 9, 2, 5, 3
    q, k, v = O.unit(rng.standard_normal((n, H, d))), O.unit(rng.standard_normal((n, H, d))), rng.standard_normal((n, H, e))
    g, beta = rng.uniform(0.3, 1, (n, H)), rng.uniform(0, 1, (n, H))
    got = O.delta_rule(q, k, v, g, beta)
    for h in range(H):
        G = np.cumprod(g[:, h])
        ratio = np.tril(G[:, None] / G[None, :])
        A = np.tril(beta[:, h, None] * ratio * (k[:, h] @ k[:, h].T), -1)
        u = np.linalg.solve(np.eye(n) + A, beta[:, h, None] * v[:, h])
        assert np.allclose(got[:, h], (ratio * (q[:, h] @ k[:, h].T)) @ u)


def test_delta_rule_replaces_what_a_key_held():
    k = np.zeros((3, 1, 4))
    k[0, 0, 0] = k[1, 0, 1] = k[2, 0, 0] = 1.0
    v = np.arange(6.0).reshape(3, 1, 2)
    one = np.ones((3, 1))
    o = O.delta_rule(k, k, v, one, one)
    assert np.allclose(o, v)                                  # the third write replaces the first's value
    assert not np.allclose(O.decayed_linear_attention(k, k, v, [1.0]), v)


def test_decayed_linear_attention_is_a_weighted_sum_of_the_past():
    rng = np.random.default_rng(1)
    n, H, d, e = 7, 2, 4, 3
    q, k, v, dec = rng.standard_normal((n, H, d)), rng.standard_normal((n, H, d)), rng.standard_normal((n, H, e)), [0.5, 0.9]
    got = O.decayed_linear_attention(q, k, v, dec)
    for h in range(H):
        for t in range(n):
            want = sum(dec[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(got[t, h], want)


def test_chunked_attention_restarts_at_every_chunk():
    rng = np.random.default_rng(2)
    n, H, G, d, e, size = 11, 4, 2, 6, 5, 4
    q, k, v = rng.standard_normal((n, H, d)), rng.standard_normal((n, G, d)), rng.standard_normal((n, G, e))
    got = O.chunked_attention(q, k, v, 0.3, size)
    for c in range(0, n, size):
        p = slice(c, min(n, c + size))
        assert np.allclose(got[p], O.chunked_attention(q[p], k[p], v[p], 0.3, 0))
    assert np.allclose(got[[0, 4, 8]], np.repeat(v[[0, 4, 8]], H // G, axis=1))       # a chunk's first token sees itself
    s = (k[4:7, 1] @ q[6, 2]) * 0.3
    p = np.exp(s) / np.exp(s).sum()
    assert np.allclose(got[6, 2], p @ v[4:7, 1])


def test_routing_weights_and_mixture():
    rng = np.random.default_rng(3)
    x, W = rng.standard_normal((6, 5)), {"router": rng.standard_normal((4, 5))}
    for e in range(4):
        W.update({f"e{e}.gate": rng.standard_normal((3, 5)), f"e{e}.up": rng.standard_normal((3, 5)), f"e{e}.down": rng.standard_normal((5, 3))})
    chosen, p = O.route(x, W["router"], 2)
    z = x @ W["router"].T
    for t in range(6):
        order = sorted(range(4), key=lambda i: -z[t, i])[:2]
        assert list(chosen[t]) == order
        w = np.exp(z[t, order]) / np.exp(z[t, order]).sum()
        assert np.allclose(p[t], w)
        want = sum(w[i] * O.gated(x[t:t + 1], O._sub(W, f"e{e}."))[0] for i, e in enumerate(order))
        assert np.allclose(O.mixture(x, 2, W)[t], want)
    p_all = O.route(x, W["router"], 4)[1]
    assert np.allclose(p_all.sum(axis=1), 1) and np.allclose(O.route(x, W["router"], 1)[1], 1)


CFG = X.config([X.delta(mlp=X.dense(30)), X.parallel(mlp=X.moe(6, 2, 18), size=7), X.delta(mlp=X.moe(5, 3, 20), conv=2)])
MISTAKES = ["chunk", "rotation", "qk_norm", "scale", "left_scale", "right_scale", "decay", "beta", "g", "conv", "unit", "q_scale", "out_norm",
            "out_gate", "router", "top", "alpha", "norm2", "softcap", "eps_inside", "read_before_write"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_a_mistake_in_any_mechanism_shows_in_the_logits(mistake, monkeypatch):
    """The comparison of the GPU tests is only worth something if a wrong mechanism moves the
    logits by far more than its tolerance: each mistake is planted in the oracle."""
    cfg = json.loads(json.dumps(CFG))
    _, W = X.random_model(cfg, 5)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 24)
    want = O.forward(cfg, W, toks)
    mixer = cfg["layers"][1]["mixer"]
    zero = {"beta": "mix.b", "out_gate": "right.g"}
    if mistake == "chunk":
        mixer["left"]["mask"]["size"] += 1
    elif mistake == "rotation":
        monkeypatch.setattr(O, "rotate_half", lambda x, p, b, d: x)
    elif mistake == "qk_norm":
        W = {k: (v * 0 + 1 if k.endswith(("q.norm", "k.norm")) else v) for k, v in W.items()}
    elif mistake == "scale":
        mixer["left"]["scale"] *= 2
    elif mistake in ("left_scale", "right_scale"):
        mixer[mistake] = 1.0
    elif mistake == "decay":
        mixer["right"]["decay"] = [d * 0.8 for d in mixer["right"]["decay"]]
    elif mistake in zero:
        W = {k: (v * 0 if k.endswith(zero[mistake]) else v) for k, v in W.items()}
    elif mistake == "g":
        W = {k: (v + 2 if k.endswith("dt_bias") else v) for k, v in W.items()}
    elif mistake == "conv":
        W = {k: (np.roll(v, 1, axis=1) if k.endswith("k.conv") else v) for k, v in W.items()}
    elif mistake == "unit":
        monkeypatch.setattr(O, "unit", lambda x: x)
    elif mistake == "q_scale":                              # hidden by the norm of the output, except for its eps
        cfg["norm"]["eps"] = 0.05
        want = O.forward(cfg, W, toks)
        monkeypatch.setattr(O, "unit", lambda x, f=O.unit: f(x) * 3.0)
    elif mistake == "out_norm":
        W = {k: (v * 0 + 1 if k.endswith("mix.norm") else v) for k, v in W.items()}
    elif mistake == "router":
        monkeypatch.setattr(O, "route", lambda x, r, t, f=O.route: (f(x, r, t)[0], 0 * f(x, r, t)[1] + 1.0 / t))
    elif mistake == "top":
        cfg["layers"][2]["mlp"]["router"]["top"] = 2
    elif mistake == "alpha":
        cfg["postln_alpha"] = 1.0
    elif mistake == "norm2":
        W = {k: (v * 0 + 1 if k.endswith("norm2") else v) for k, v in W.items()}
    elif mistake == "softcap":
        monkeypatch.setattr(O, "softcap", lambda z, c: z)
    elif mistake == "eps_inside":
        cfg["norm"]["eps"] = 0.5
    elif mistake == "read_before_write":
        monkeypatch.setattr(O, "delta_rule", lambda q, k, v, g, b, f=O.delta_rule: f(q, k, v, g, b) - (q * k).sum(-1, keepdims=True) * v * b[..., None])
    assert X.row_error(O.forward(cfg, W, toks), want).max() > 0.07


# ---- loading -----------------------------------------------------------------------------
def test_a_folder_loads_by_its_architecture(tmp_path):
    raw, _ = X.random_model(CFG, 1)
    write_model(str(tmp_path), CFG, raw)
    m = models.load(str(tmp_path))
    assert isinstance(m, mixed.Femolix) and m.residual_scale == CFG["postln_alpha"] and m.logit_softcap == CFG["logit_softcap"]
    assert [layer.type for layer in m.layers] == [mixed.DELTA_RULE, mixed.ATTENTION, mixed.DELTA_RULE]
    assert m.layers[1].beside.type == mixed.LINEAR_ATTENTION and m.layers[0].beside is None
    assert m.layers[1].sizes["experts"] == 6 and len(m.layers[1].tensors["gate"]) == 6
    assert (m.layers[1].tensors["gate"][5] == raw["l1.mlp.e5.gate"]).all()
    held = sorted(X.model(CFG, raw).tensor_shapes(CFG)) == sorted(raw)
    assert held


def test_a_description_carries_the_mixer_beside_and_the_experts():
    raw, _ = X.random_model(CFG, 1)
    m, seen = X.model(CFG, raw), []

    def up(a):
        seen.append(a)
        return len(seen)

    d = m.fill_desc(up, 64)
    assert d.norm_after_sum == 1 and abs(d.residual_scale - 1.7) < 1e-6 and d.logit_softcap == 9.0 and d.head
    L = d.layers[1]
    other = _lib.MixedLayerDesc.from_address(L.beside)
    assert (other.type, other.heads, other.dim, other.vdim) == (mixed.LINEAR_ATTENTION, 3, 10, 14)
    assert np.allclose([other.head_decay[i] for i in range(3)], CFG["layers"][1]["mixer"]["right"]["decay"])
    assert (L.chunk, L.experts, L.top, L.ff) == (7, 6, 2, 18) and abs(other.out_scale - 0.45) < 1e-7
    assert isinstance(seen[L.t[mixed.TENSOR_SLOTS.index("down")] - 1], list) and d.layers[0].beside is None


@pytest.mark.parametrize("change,match", [
    (lambda c, r: r.pop("l1.mlp.e3.up"), "l1.mlp.e3.up is missing"),
    (lambda c, r: r.update({"l1.mlp.e3.up": r["l1.mlp.e3.up"][:-1]}), "up of layer 1"),
    (lambda c, r: r.update({"l0.mix.q.conv": r["l0.mix.q.conv"][:, :-1]}), "q_conv of layer 0"),
    (lambda c, r: c["layers"][1]["mixer"]["right"]["decay"].pop(), "decays"),
    (lambda c, r: c["layers"][1]["mlp"]["router"].update(top=9), "9 of 6"),
    (lambda c, r: c["layers"][1]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c, r: c["layers"][0].update(type="lstm"), "unknown mixer"),
    (lambda c, r: r.update(head=r["head"][:-1]), "head"),
    (lambda c, r: c["layers"][1]["mixer"]["right"].update(vdim=15), "of layer 1"),
])
def test_a_model_that_does_not_fit_its_configuration_is_refused(change, match):
    cfg = json.loads(json.dumps(CFG))
    raw, _ = X.random_model(cfg, 1)
    change(cfg, raw)
    with pytest.raises(ValueError, match=match):
        X.model(cfg, raw)


def test_ctypes_structures_match_the_header(tmp_path):
    src = tmp_path / "s.c"
    src.write_text('#include <stdio.h>\n#include <stddef.h>\n#include "tllm_b200_mixed.h"\n#define L(f) offsetof(tllm_b200_mixed_layer, f)\n'
                   '#define D(f) offsetof(tllm_b200_mixed_desc, f)\n'
                   'int main(void){printf("%zu %zu %zu %zu %zu %zu %zu %d %d %d", L(experts), L(out_scale), L(head_decay), L(beside), D(logit_softcap),'
                   'D(head), D(layers), TLLM_T_K, TLLM_T_ROUTER, TLLM_MIXER_DELTA_RULE);return 0;}')
    exe = str(tmp_path / "s")
    subprocess.check_call(["gcc", "-I", os.path.join(ROOT, "include"), "-o", exe, str(src)])
    got = [int(v) for v in subprocess.check_output([exe]).split()]
    L, D, slot = _lib.MixedLayerDesc, _lib.MixedDesc, mixed.TENSOR_SLOTS.index
    assert got == [L.experts.offset, L.out_scale.offset, L.head_decay.offset, L.beside.offset, D.logit_softcap.offset, D.head.offset,
                   D.layers.offset, slot("k"), slot("router"), mixed.DELTA_RULE]


def test_argument_errors_need_no_gpu():
    h = _lib.lib()
    buf = ctypes.create_string_buffer(4096 + 64)
    p = (ctypes.addressof(buf) + 63) & ~63
    att = [1e-5, p, 8, p, p, p, 4, 2, 16, 8]
    assert h.tllm_b200_grouped_attention(1, None, None, None, *att, 0, 32, 32, 1.0, 1.0, 1, 4, 0, None) == -1
    assert h.tllm_b200_grouped_attention(1, p, None, None, *att, 0, 16, 32, 1.0, 1.0, 1, 4, 0, None) == -3      # a ring without chunks
    assert h.tllm_b200_grouped_attention(1, p, None, None, *att, 8, 11, 32, 1.0, 1.0, 1, 4, 0, None) == -3      # a ring too short
    assert h.tllm_b200_grouped_attention(1, p, None, None, 1e-5, p, 8, p, p, p, 5, 2, 16, 8, 0, 32, 32, 1.0, 1.0, 1, 4, 0, None) == -3
    assert h.tllm_b200_matrix_scan(1, 1, p, p, None, p, p, p, 1.0, p, p, 2, 1, 8, 8, 1, 1, 0, None) == -1
    assert h.tllm_b200_matrix_scan(1, 0, p, p, None, None, None, None, 1.0, p, p, 2, 2, 12, 8, 1, 1, 0, None) == -3
    assert h.tllm_b200_gated_norm(1, p, p, p, p, 1, 1, 12, 1e-5, 1.0, 2, None) == -3
    assert h.tllm_b200_experts(1, p, p, p, p, p, 1, 16, 8, 4, 5, 2, None) == -3
