"""Models of mixer layers, what needs no GPU: the oracle's mechanisms against independent forms
of the same equations, the sensitivity of the comparison to mistakes, the safetensors container,
the registry and its refusals, and the trace replay on a stand-in decoder."""
import ctypes
import io
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import mixed_oracle as O
from tests import _mixed as M
from ternary_llm_b200 import _lib, generate, mixed, models, trace
from ternary_llm_b200 import safetensors_io as st

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- the oracle against other forms of the same equations ------------------------------
def test_oracle_convolution_is_numpys():
    rng = np.random.default_rng(0)
    x, w, b = rng.standard_normal((9, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    y = O.causal_conv(x, w, b)
    for c in range(3):
        assert np.allclose(y[:, c], b[c] + np.convolve(x[:, c], w[c, ::-1])[:9])


def test_oracle_scans_are_weighted_sums_of_the_past():
    rng = np.random.default_rng(1)
    n, C, S = 6, 3, 4
    x, dt = rng.standard_normal((n, C)), rng.uniform(0.1, 1, (n, C))
    A, B, Cm, D = -rng.uniform(0.1, 2, (C, S)), rng.standard_normal((n, S)), rng.standard_normal((n, S)), rng.standard_normal(C)
    want = np.zeros((n, C))
    for t in range(n):
        for s in range(t + 1):
            decay = np.exp(dt[s + 1:t + 1].sum(axis=0)[:, None] * A)
            want[t] += ((decay * B[s]) * Cm[t]).sum(axis=1) * dt[s] * x[s]
        want[t] += D * x[t]
    assert np.allclose(O.selective_scan(x, dt, A, B, Cm, D), want)
    r, i, lam = rng.uniform(0, 1, (n, C)), rng.uniform(0, 1, (n, C)), rng.standard_normal(C)
    la = -8.0 * r * np.log1p(np.exp(lam))
    want = np.zeros((n, C))
    for t in range(n):
        for s in range(t + 1):
            want[t] += np.exp(la[s + 1:t + 1].sum(axis=0)) * np.sqrt(1 - np.exp(2 * la[s])) * i[s] * x[s]
    assert np.allclose(O.gated_linear_recurrence(x, r, i, lam), want)


def test_oracle_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))
    dots = [(O.rotate_half(q, [p + 7], 100.0, 8) * O.rotate_half(k, [p], 100.0, 8)).sum() for p in (0, 5, 300)]
    assert np.allclose(dots, dots[0]) and not np.isclose(dots[0], (q * k).sum())
    assert np.allclose(O.rotate_half(q, [9], 100.0, 8)[:, 8:], q[:, 8:])


def test_oracle_attention_sink_is_a_key_of_value_zero():
    rng = np.random.default_rng(3)
    n, H, d = 5, 2, 4
    q, k, v, sink = rng.standard_normal((n, H, d)), rng.standard_normal((n, H, d)), rng.standard_normal((n, H, 3)), rng.standard_normal(H)
    out = O.sink_attention(q, k, v, 0.7, sink)
    for h in range(H):
        for t in range(n):
            s = np.append((k[:t + 1, h] @ q[t, h]) * 0.7, sink[h])
            p = np.exp(s) / np.exp(s).sum()
            assert np.allclose(out[t, h], p[:-1] @ v[:t + 1, h])


CFG = dict(layers=[M.attention(ff=40), M.mamba(), M.rglru(ff=24)], loop={"start": 0, "stop": 2, "times": 2})


@pytest.mark.parametrize("mistake", ["sink", "gate", "rotation", "conv", "scan_skip", "lam", "inject", "post_norm", "conv_bias"])
def test_a_mistake_in_any_mechanism_shows_in_the_logits(mistake, monkeypatch):
    """The comparison of the GPU tests is only worth something if a wrong mechanism moves the
    logits by far more than its tolerance: each mistake is planted in the oracle."""
    cfg = M.config(**CFG)
    _, W = M.random_model(cfg, 5)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 24)
    want = O.forward(cfg, W, toks)
    if mistake == "sink":
        W = {k: (v * 0 - 1e4 if k.endswith("sink") else v) for k, v in W.items()}
    elif mistake == "gate":
        W = {k: (v * 0 if k.endswith("mix.g") else v) for k, v in W.items()}
    elif mistake == "rotation":
        monkeypatch.setattr(O, "rotate_half", lambda x, p, b, d: x)
    elif mistake == "conv":
        W = {k: (np.roll(v, 1, axis=1) if k.endswith("conv") else v) for k, v in W.items()}
    elif mistake == "conv_bias":
        W = {k: (v * 0 if k.endswith("conv.b") else v) for k, v in W.items()}
    elif mistake == "scan_skip":
        W = {k: (v * 0 if k.endswith(".D") else v) for k, v in W.items()}
    elif mistake == "lam":
        W = {k: (v + 3 if k.endswith("lam") else v) for k, v in W.items()}
    elif mistake == "inject":
        monkeypatch.setattr(O, "run_order", lambda c, f=O.run_order: [(i, False) for i, _ in f(c)])
    elif mistake == "post_norm":
        W = {k: (v * 0 + 1 if k.endswith("norm1b") else v) for k, v in W.items()}
    err = M.row_error(O.forward(cfg, W, toks), want)
    assert err.max() > 0.1


def test_run_order_of_a_loop():
    cfg = M.config([M.mamba()] * 5, loop={"start": 1, "stop": 3, "times": 3})
    assert O.run_order(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]


# ---- container, registry, configuration --------------------------------------------------
def test_safetensors_round_trip(tmp_path):
    rng = np.random.default_rng(0)
    t = {"a": st.to_bf16(rng.standard_normal((3, 5)).astype(np.float32)), "b.c": np.arange(7, dtype=np.int32),
         "d": rng.standard_normal(4).astype(np.float32)}
    p = str(tmp_path / "x.safetensors")
    st.write_safetensors(p, t)
    f = st.SafetensorsFile(p)
    assert set(f.keys()) == set(t) and f.dtypes == {"a": "BF16", "b.c": "I32", "d": "F32"}
    for k in t:
        assert (f[k] == t[k]).all() and f[k].shape == t[k].shape
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-4])
    with pytest.raises(ValueError):
        st.SafetensorsFile(p)


def test_bf16_conversion_rounds_to_nearest_even():
    import torch
    x = np.random.default_rng(0).standard_normal(1000).astype(np.float32)
    want = torch.from_numpy(x).to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16)
    assert (st.to_bf16(x) == want).all()
    assert (st.from_bf16(want) == torch.from_numpy(x).to(torch.bfloat16).float().numpy()).all()


def write_model(path, cfg, raw):
    os.makedirs(path, exist_ok=True)
    json.dump(cfg, open(os.path.join(path, "config.json"), "w"))
    st.write_safetensors(os.path.join(path, "model.safetensors"), raw)


def test_a_folder_loads_by_its_architecture(tmp_path):
    cfg = M.config(**CFG)
    raw, _ = M.random_model(cfg, 1)
    write_model(str(tmp_path), cfg, raw)
    m = models.load(str(tmp_path))
    assert isinstance(m, mixed.Petulix) and m.vocab_size == cfg["vocab"] and m.loop == (0, 2, 2, True)
    assert [layer.type for layer in m.layers] == [mixed.LATENT_ATTENTION, mixed.SELECTIVE_SCAN, mixed.GATED_RECURRENCE]
    cfg["architecture"] = "Unheard"
    write_model(str(tmp_path), cfg, raw)
    with pytest.raises(ValueError, match="unknown architecture"):
        models.load(str(tmp_path))


@pytest.mark.parametrize("change,match", [
    (lambda c, r: r.pop("l1.mix.dt"), "l1.mix.dt is missing"),
    (lambda c, r: r.update({"l0.mix.sink": r["l0.mix.sink"][:-1]}), "sink of layer 0"),
    (lambda c, r: c.update(width=c["width"] + 1), "embedding"),
    (lambda c, r: c["layers"][2].update(type="lstm"), "unknown mixer"),
    (lambda c, r: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c, r: c["layers"][2]["mixer"].update(blocks=7), "does not split"),
])
def test_a_model_that_does_not_fit_its_configuration_is_refused(change, match):
    cfg = json.loads(json.dumps(M.config(**CFG)))
    raw, _ = M.random_model(cfg, 1)
    change(cfg, raw)
    with pytest.raises(ValueError, match=match):
        M.model(cfg, raw)


def test_ctypes_structures_match_the_header(tmp_path):
    src = tmp_path / "s.c"
    src.write_text('#include <stdio.h>\n#include <stddef.h>\n#include "tllm_b200_mixed.h"\n'
                   'int main(void){printf("%zu %zu %d %zu %zu %d %d", sizeof(tllm_b200_mixed_layer), sizeof(tllm_b200_mixed_desc),'
                   'TLLM_T_COUNT, offsetof(tllm_b200_mixed_layer, t), offsetof(tllm_b200_mixed_layer, rot_base), TLLM_T_LAM, TLLM_T_Q);return 0;}')
    exe = str(tmp_path / "s")
    subprocess.check_call(["gcc", "-I", os.path.join(ROOT, "include"), "-o", exe, str(src)])
    got = [int(v) for v in subprocess.check_output([exe]).split()]
    assert got == [ctypes.sizeof(_lib.MixedLayerDesc), ctypes.sizeof(_lib.MixedDesc), _lib.TENSORS_PER_LAYER, _lib.MixedLayerDesc.t.offset,
                   _lib.MixedLayerDesc.rot_base.offset, mixed.TENSOR_SLOTS.index("lam"), mixed.TENSOR_SLOTS.index("q")]
    assert len(mixed.TENSOR_SLOTS) == _lib.TENSORS_PER_LAYER


def test_argument_errors_need_no_gpu():
    h = _lib.lib()
    buf = ctypes.create_string_buffer(4096 + 64)
    p = (ctypes.addressof(buf) + 63) & ~63
    out = ctypes.c_void_p()
    assert h.tllm_b200_mixed_decoder_create(None, 0, 1, ctypes.byref(out)) == -1
    d = _lib.MixedDesc()
    d.layers, d.embedding, d.final_norm = (_lib.MixedLayerDesc * 1)(), p, p
    assert h.tllm_b200_mixed_decoder_create(ctypes.byref(d), 0, 65, ctypes.byref(out)) == -5
    assert h.tllm_b200_mixed_decoder_create(ctypes.byref(d), 0, 1, ctypes.byref(out)) == -3
    assert h.tllm_b200_mixed_decoder_runs(None) == 0
    assert h.tllm_b200_decoder_forward_logits(None, 0, p, 1, 0, None, 0, None, None, None) == -1
    assert h.tllm_b200_dense_linear(1, p, p, None, p, 1, 8, 12, 0, 0, None) == -3
    assert h.tllm_b200_causal_conv(1, p, p, None, None, p, 8, 2, 0, 1, 1, 0, None) == -1
    assert h.tllm_b200_causal_conv(1, p, p, None, p, p, 9, 2, 0, 1, 1, 0, None) == -3
    assert h.tllm_b200_selective_scan(1, p, p, p, None, p, None, p, p, 8, 0, 1, 1, 0, None) == -3
    assert h.tllm_b200_gated_scan(1, p, p, p, p, p, p, 24, 2, 8.0, 1, 1, 1, 0, None) == -3
    assert h.tllm_b200_latent_attention(1, p, p, None, p, 2, 16, 8, 1.0, 4, 1, 5, 0, None) == -3
    assert h.tllm_b200_latent_attention_expanded(p, p, p, p, None, None, p, 2, 12, 8, 8, 16, 1.0, 8, 4, 0, None) == -3


# ---- trace replay on a stand-in decoder ----------------------------------------------------
class _FakeDecoder:
    vocab_size, device = 4, "cpu"

    def __init__(self):
        self.calls = []

    def forward_logits(self, slot, ids, start, want):
        import torch
        self.calls.append((slot, ids.tolist(), start, list(want)))
        return torch.tensor([[float(ids[w]), start + w, slot, 0.5] for w in want], dtype=torch.float32).reshape(len(want), 4)


def test_trace_replay_positions_slots_and_files(tmp_path, monkeypatch):
    import torch
    monkeypatch.setattr(torch.cuda, "synchronize", lambda *a: None)
    dec, said = _FakeDecoder(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [0], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [2], "want": [0]}, {"id": "c", "tokens": [3, 3], "want": [1]}], "end": ["a", "c"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [1], "want": [0]}], "end": []}]
    trace.run(dec, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), said.append, 2)
    assert said == ["done 0", "done 1", "done 2", "done 3"]
    assert [c[2] for c in dec.calls] == [0, 0, 3, 0, 0]                 # positions; "a" starts anew after its end
    assert dec.calls[1][0] != dec.calls[0][0] and dec.calls[3][0] == dec.calls[1][0]
    assert not os.path.exists(tmp_path / "1.f32")
    got = np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 4)
    assert got[:, 0].tolist() == [3.0, 1.0] and got[:, 1].tolist() == [2.0, 0.0]
    assert np.fromfile(tmp_path / "2.f32", "<f4").reshape(-1, 4)[:, 1].tolist() == [3.0, 1.0]
    with pytest.raises(ValueError, match="token id"):
        trace.run(dec, io.StringIO(json.dumps({"step": 0, "entries": [{"id": "z", "tokens": [4], "want": []}], "end": []})),
                  str(tmp_path), said.append, 2)
    with pytest.raises(RuntimeError, match="slots"):
        t = trace.SlotTable(1)
        t.slot("a"), t.slot("b")


def test_generation_command_line_arguments(capsys):
    assert generate.parse_tokens("5, 17,3") == [5, 17, 3]
    for bad in (["--model", "m", "--tokens", "a"], ["--model", "m", "--tokens", "-1"], ["--tokens", "1"], ["--model", "m", "--tokens", "1", "--dtype", "int8"]):
        with pytest.raises(SystemExit):
            generate.main(bad)
    capsys.readouterr()
