"""Femolix models through the Decoder against the oracle: whole prompts, portions, decoding, slots
used again, sequences in lock step, keys and states just inside and outside their reach, the
residual stream after every layer, rings of cache rows, greedy generation, and the programs."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import ternary_llm_b200 as tl
from oracle import femolix_oracle as O
from tests import _femolix as X
from tests.test_gpu_mixed_decoder import ids, run
from tests.test_mixed_cpu import write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {"float32": 1e-4, "bfloat16": 6e-2}

CONFIGS = {
    "all": X.config([X.delta(mlp=X.dense(40)), X.parallel(mlp=X.moe(6, 2, 24)), X.parallel(size=16, mlp=X.dense(18)), X.delta(conv=2, mlp=X.moe(5, 3, 20))]),
    "delta": X.config([X.delta(heads=3, kv_heads=1, dim=64, vdim=80, conv=4), X.delta(heads=3, kv_heads=3, dim=9, vdim=7, conv=1, mlp=X.dense(11)),
                       X.delta(heads=4, kv_heads=4, dim=24, vdim=72, conv=5)], width=72, vocab=257, eps=1e-3, alpha=1.0),
    "parallel": X.config([X.parallel(heads=8, kv_heads=8, dim=24, vdim=24, size=50, rot=24, r_heads=2, r_dim=40, r_vdim=72),
                          X.parallel(heads=5, kv_heads=1, dim=10, vdim=9, size=1, rot=2, r_heads=1, r_dim=7, r_vdim=33, decay=[0.999]),
                          X.parallel(heads=4, kv_heads=2, size=130, rot=4, left=1.0, right=1.0, r_heads=6, r_dim=16, r_vdim=8)], width=50, alpha=2.5),
    "experts": X.config([X.delta(mlp=X.moe(3, 3, 9)), X.delta(mlp=X.moe(12, 1, 16)), X.parallel(mlp=X.moe(9, 4, 33))], width=30, cap=3.0),
    "narrow": X.config([X.delta(heads=1, kv_heads=1, dim=4, vdim=5, conv=4, mlp=X.dense(6)), X.parallel(heads=2, kv_heads=1, dim=4, vdim=3, rot=2, r_heads=1)],
                       width=9, vocab=17, alpha=0.8),
}
_cache = {}


def setup(name, n=150, seed=0):
    """(configuration, tensors, floats, tokens, oracle logits, oracle residuals), computed once."""
    key = (name, n, seed)
    if key not in _cache:
        cfg = CONFIGS[name]
        raw, W = X.random_model(cfg, sum(map(ord, name)))
        toks = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], n).astype(np.int32)
        taps = []
        _cache[key] = (cfg, raw, W, toks, O.forward(cfg, W, toks, taps), np.stack(taps))
    return _cache[key]


def near(err, dtype):
    """In BF16 a close call of a router goes either way and moves single positions: nearly all within
    the limit, and the bulk well within."""
    if dtype == "float32":
        return err.max() <= LIMIT[dtype]
    return (err > LIMIT[dtype]).mean() <= 0.06 and np.median(err) <= LIMIT[dtype] / 2


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    """Whole prompt, portions of several sizes down to two tokens, and token by token after a
    prefix: all equal to the oracle; the slot carries another sequence's state before each."""
    cfg, raw, _, toks, want, _ = setup(name)
    n = len(toks)
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_batch=2, max_seq_len=n)
    cuts = {"whole": [n], "decode": [n - 40] + [1] * 40, "tokens": [1] * n, "pairs": [2] * (n // 2), "portions": [2, 3, 9, 1, 16, 33, 2, 64, n - 130]}
    for what, c in cuts.items():
        err = X.row_error(run(dec, toks, c, seq=1), want)
        assert near(err, dtype), f"{what}: {err.max():.2e} at {int(err.argmax())}"
    tl.check_device_errors()
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_residual_after_every_layer(dtype):
    cfg, raw, _, toks, _, taps = setup("all")
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=len(toks))
    _, got = dec.forward_logits(0, ids(toks), 0, [], taps=True)
    assert got.shape == taps.shape
    for r in range(len(taps)):
        err = np.abs(got[r].double().cpu().numpy() - taps[r]).max(axis=1) / np.abs(taps[r]).max()
        assert np.quantile(err, 1.0 if dtype == "float32" else 0.95) <= {"float32": 1e-4, "bfloat16": 5e-2}[dtype], f"layer {r}: {err.max():.2e}"
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("at", [0, 3, 89, 90, 179])
def test_a_key_is_found_until_its_chunk_ends(at, dtype):
    """Attention whose every query picks one token, wherever in the chunk: exactly the positions of
    that chunk behind it feel the token, in prompts and in decoding."""
    cfg = X.config([X.parallel(heads=4, kv_heads=2, dim=16, vdim=24, size=90, rot=4, scale=1.0, left=1.0, right=0.0)], width=48, vocab=61)
    raw, W = X.finder_model(cfg, 77)
    toks = np.random.default_rng(3).integers(0, 60, 230).astype(np.int32)
    other = toks.copy()
    toks[at] = 60                              # the only token of its kind
    want, without = O.forward(cfg, W, toks), O.forward(cfg, W, other)
    moved = np.sqrt(((want - without) ** 2).mean(axis=1)) / np.std(want)
    end = (at // 90 + 1) * 90
    inside = np.zeros(230, bool)
    inside[at:min(end, 230)] = True
    assert moved[inside].min() > 0.2 and moved[~inside].max() < 1e-9           # the case is what it says
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=230)
    for cuts in ([230], [60] + [1] * 50 + [120], [170] + [1] * 60, [88, 2, 2, 2, 136]):
        err = X.row_error(run(dec, toks, cuts), want)
        assert err.max() <= LIMIT[dtype], f"{cuts[:3]}: {err.max():.2e} at {int(err.argmax())}"
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("kind", ["linear", "delta"])
def test_the_first_token_is_remembered(kind, dtype):
    """States that hardly decay: the first token still decides hundreds of positions later."""
    if kind == "linear":
        cfg = X.config([X.parallel(left=0.0, right=1.0, r_heads=2, r_dim=12, r_vdim=20, decay=[0.99995, 0.9999])], width=40, vocab=50, alpha=0.5)
    else:
        cfg = X.config([X.delta(heads=2, kv_heads=1, dim=48, vdim=24, conv=4)], width=40, vocab=50, alpha=0.5)
    raw, W = X.random_model(cfg, 9)
    if kind == "linear":
        W["embed"][49] *= 12.0
    else:                                      # the first token's key is its own, and nothing decays
        W["l0.mix.A_log"] = W["l0.mix.A_log"] * 0 - 12.0
        W["embed"][:, 0], W["embed"][:, 1] = 0.0, 1.0
        W["embed"][49], W["embed"][49, 0] = 3 * W["embed"][49], 30.0
        W["l0.mix.q"][:, 0], W["l0.mix.k"][:, 1] = 0.0, 0.0
        W["l0.mix.k"][0], W["l0.mix.q"][0], W["l0.mix.k"][0, 0], W["l0.mix.q"][0, 1] = 0.0, 0.0, 2.0, 3.0
        for t in ("q", "k"):
            W[f"l0.mix.{t}.conv"][0] = [0.0, 0.0, 0.0, 1.0]
    raw, W = X.refloat(W)
    toks = np.random.default_rng(5).integers(0, 49, 420).astype(np.int32)
    other = toks.copy()
    toks[0] = 49
    want, without = O.forward(cfg, W, toks), O.forward(cfg, W, other)
    moved = np.sqrt(((want - without) ** 2).mean(axis=1)) / np.std(want)
    assert np.median(moved[300:]) > 0.1
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=420)
    for cuts in ([420], [2] * 20 + [380], [1, 63, 1, 255] + [1] * 100, [64, 64, 128, 164]):
        err = X.row_error(run(dec, toks, cuts), want)
        assert err.max() <= LIMIT[dtype], f"{cuts[:3]}: {err.max():.2e} at {int(err.argmax())}"
    dec.close()


def test_slots_are_independent_and_used_again():
    """Requests of unequal length interleaved over two slots that change owners."""
    cfg, raw, W, toks, want, _ = setup("all")
    dec = tl.Decoder(X.model(cfg, raw), dtype="float32", max_batch=3, max_seq_len=160)
    toks2 = np.random.default_rng(11).integers(0, cfg["vocab"], 90).astype(np.int32)
    want2 = O.forward(cfg, W, toks2)
    a = [dec.forward_logits(2, ids(toks[:70]), 0, [69])]
    b = [dec.forward_logits(0, ids(toks2[:33]), 0, [0, 32])]
    a.append(dec.forward_logits(2, ids(toks[70:72]), 70, [0, 1]))
    b.append(dec.forward_logits(0, ids(toks2[33:90]), 33, [56]))
    a.append(dec.forward_logits(2, ids(toks[72:150]), 72, [77]))
    c = dec.forward_logits(0, ids(toks[:60]), 0, [59])           # slot 0 starts anew
    for got, w in ((torch.cat(a), want[[69, 70, 71, 149]]), (torch.cat(b), want2[[0, 32, 89]]), (c, want[[59]])):
        assert X.row_error(got.cpu().numpy(), w).max() <= LIMIT["float32"]
    for bad in (59, 61, 149):                                     # a recurrent state cannot be rewound
        with pytest.raises(tl.TllmError, match="continue"):
            dec.forward_logits(0, ids(toks[:1]), bad, [])
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("batch", [2, 5, 12])
def test_lock_step_batches(batch, dtype):
    """One token of several sequences per step against each sequence in the oracle."""
    cfg, raw, W, _, _, _ = setup("all")
    toks = np.random.default_rng(batch).integers(0, cfg["vocab"], (batch, 54)).astype(np.int32)
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_batch=batch, max_seq_len=60)
    want, errs = [O.forward(cfg, W, t) for t in toks], []
    for b in range(batch):
        errs.append(X.row_error(dec.forward_seq(b, ids(toks[b, :50]), 0).cpu().numpy()[None], want[b][49:50])[0])
    for t in range(50, 54):
        got = dec.forward_batch(ids(toks[:, t]), t).cpu().numpy()
        errs += [X.row_error(got[b][None], want[b][t:t + 1])[0] for b in range(batch)]
    assert near(np.array(errs), dtype), max(errs)
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_a_ring_of_cache_rows(dtype):
    """A sequence far longer than the cache of its chunked layers: prompts of more tokens than one
    pass, wanted logits from every part, and decoding across further chunks."""
    cfg = X.config([X.parallel(heads=2, kv_heads=1, dim=8, vdim=8, size=60, rot=4, r_heads=1, r_dim=8, r_vdim=8, mlp=X.dense(16)),
                    X.parallel(heads=2, kv_heads=2, dim=8, vdim=16, size=150, rot=8, scale=1.5, r_heads=2, r_dim=8, r_vdim=8),
                    X.delta(heads=1, kv_heads=1, dim=8, vdim=8, mlp=X.moe(4, 2, 8))], width=24, vocab=40)
    raw, W = X.random_model(cfg, 8)
    n = 2600
    toks = np.random.default_rng(8).integers(0, 40, n).astype(np.int32)
    want = O.forward(cfg, W, toks)
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=n)
    at = [0, 59, 60, 149, 150, 2047, 2048, 2049, 2099, 2100, 2499]
    got = [dec.forward_logits(0, ids(toks[:2500]), 0, at)] + [dec.forward_logits(0, ids(toks[p:p + 1]), p, [0]) for p in range(2500, n)]
    assert near(X.row_error(torch.cat(got).cpu().numpy(), want[at + list(range(2500, n))]), dtype)
    cuts = [1000, 2, 1046, 90, 1, 1, 200, n - 2340]
    assert near(X.row_error(run(dec, toks, cuts), want), dtype)
    with pytest.raises(tl.TllmError, match="continue"):
        dec.forward_logits(0, ids(toks[:1]), 30, [])
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_greedy_generation_through_the_graph_replayed_loop(dtype):
    """generate() against the oracle fed with the same tokens: every token is the oracle's best
    (or within rounding of it), over a long run, from a prompt, from nothing, and continued."""
    cfg, raw, W, toks, _, _ = setup("all")
    dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=400)
    slack = LIMIT[dtype] * 6

    def check(seq, n_prompt):
        lg = O.forward(cfg, W, seq)
        bad = [p for p in range(n_prompt - 1, len(seq) - 1) if lg[p, seq[p + 1]] < lg[p].max() - slack * lg[p].std()]
        assert len(bad) <= (0 if dtype == "float32" else 0.05 * len(seq)), bad

    first = int(dec.forward(ids(toks[:20]), 0).argmax())
    out, _ = dec.generate(first, 20, 100)
    more, _ = dec.generate(out[-1], 120, 30)                     # continues where it ended
    check(np.concatenate([toks[:20], [first], out, more]), 20)
    out2, _ = dec.generate(int(toks[0]), 0, 15)                  # position 0: a new sequence in the slot
    check(np.concatenate([toks[:1], out2]), 1)
    dec.reset()
    dec.forward(ids(toks[:20]), 0)
    again, _ = dec.generate(first, 20, 100)
    assert again == out
    dec.forward(ids(toks[:20]), 0)                               # the same tokens step by step through forward()
    tok = first
    for i in range(12):
        tok_next = int(dec.forward(ids([tok]), 20 + i).argmax())
        assert tok_next == out[i]
        tok = tok_next
    dec.close()


def test_sizes_of_a_real_layer_agree_between_the_two_precisions():
    """Wide layers take other kernel instances; BF16 against the 32-bit mode on the same weights."""
    cfg = X.config([X.delta(heads=8, kv_heads=4, dim=128, vdim=128, conv=4, mlp=X.dense(1536)),
                    X.parallel(heads=16, kv_heads=2, dim=128, vdim=128, size=256, rot=64, scale=128 ** -0.5, r_heads=4, r_dim=128, r_vdim=128),
                    X.delta(heads=2, kv_heads=2, dim=256, vdim=64, conv=3, mlp=X.dense(512))], width=640, vocab=1000)
    raw, _ = X.random_model(cfg, 3)
    toks = np.random.default_rng(0).integers(0, 1000, 700).astype(np.int32)
    out = {}
    for dtype in LIMIT:
        dec = tl.Decoder(X.model(cfg, raw), dtype=dtype, max_seq_len=720)
        out[dtype] = [run(dec, toks, c) for c in ([700], [680] + [1] * 20, [100, 9, 150, 2, 400, 39])]
        tl.check_device_errors()
        dec.close()
    for a, b in zip(out["float32"], out["bfloat16"]):
        assert X.row_error(a, out["float32"][0]).max() <= LIMIT["float32"]
        assert X.row_error(b, out["float32"][0]).max() <= LIMIT["bfloat16"]


def test_programs(tmp_path):
    """Trace replay and the command line."""
    cfg, raw, _, toks, want, _ = setup("all")
    write_model(str(tmp_path / "m"), cfg, raw)
    os.makedirs(tmp_path / "out")
    env = dict(os.environ, PATH=os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:50].tolist(), "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[50:51].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:9].tolist(), "want": [8]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600, env=env)
    assert r.returncode == 0, r.stderr[-2000:]
    for step, places in ((0, [49, 3]), (1, [50]), (2, [8])):
        got = np.fromfile(tmp_path / "out" / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert X.row_error(got, want[places]).max() <= LIMIT["float32"]
    r = subprocess.run([sys.executable, "-m", "ternary_llm_b200.generate", "--model", str(tmp_path / "m"), "--tokens", ",".join(map(str, toks[:12])),
                        "--steps", "9", "--dtype", "float32"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    dec = tl.Decoder(str(tmp_path / "m"), dtype="float32", max_seq_len=64)
    tok, expect = int(dec.forward(ids(toks[:12]), 0).argmax()), []
    for i in range(9):
        expect.append(tok)
        tok = int(dec.forward(ids([tok]), 12 + i).argmax())
    assert [int(v) for v in r.stdout.strip().splitlines()[-1].split(",")] == expect
    dec.close()
