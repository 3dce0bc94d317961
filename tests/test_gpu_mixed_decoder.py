"""Models of mixer layers through the Decoder against the oracle: whole prompts, portions,
decoding, slots used again, sequences in lock step, loops, the residual stream after every layer
run, greedy generation through the graph-replayed loop, and the trace replay program."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import ternary_llm_b200 as tl
from oracle import mixed_oracle as O
from tests import _mixed as M
from tests.test_mixed_cpu import write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {"float32": 1e-4, "bfloat16": 6e-2}

CONFIGS = {
    "all": M.config([M.attention(ff=40), M.mamba(), M.rglru(ff=24), M.attention(heads=5, dim=16, rot_dim=4, vdim=8, kv_rank=24, base=500.0)],
                    loop={"start": 1, "stop": 3, "times": 3}),
    "attention": M.config([M.attention(heads=8, dim=24, rot_dim=16, vdim=36, kv_rank=72, ff=100), M.attention(heads=1, vdim=9, dim=1, rot_dim=2, kv_rank=11)],
                          width=72, vocab=257, loop={"start": 0, "stop": 2, "times": 2}, eps=1e-3),
    "mamba": M.config([M.mamba(inner=88, state=33, dt_rank=1, conv=2, ff=16), M.mamba(inner=7, state=1, dt_rank=9, conv=1)], width=50),
    "rglru": M.config([M.rglru(width=33, blocks=1, conv=4), M.rglru(width=64, blocks=8, conv=1, ff=9), M.rglru(width=6, blocks=6, conv=5)], width=30,
                      loop={"start": 2, "stop": 3, "times": 4}),
    "one_layer_loop": M.config([M.rglru(), M.mamba(ff=8), M.attention(kv_rank=16)], width=64, vocab=64, loop={"start": 2, "stop": 3, "times": 2}),
}
_cache = {}


def setup(name, n=150, seed=0):
    """(configuration, tensors, tokens, oracle logits, oracle residuals), computed once."""
    key = (name, n, seed)
    if key not in _cache:
        cfg = CONFIGS[name]
        raw, W = M.random_model(cfg, sum(map(ord, name)))
        toks = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], n).astype(np.int32)
        taps = []
        _cache[key] = (cfg, raw, toks, O.forward(cfg, W, toks, taps), np.stack(taps))
    return _cache[key]


def ids(t):
    return torch.from_numpy(np.asarray(t, np.int32)).cuda()


def run(dec, toks, cuts, seq=0):
    out, pos = [], 0
    for c in cuts:
        out.append(dec.forward_logits(seq, ids(toks[pos:pos + c]), pos, list(range(c))).cpu().numpy())
        pos += c
    assert pos == len(toks)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    """Whole prompt, portions of several sizes down to two tokens, and token by token after a
    prefix: all equal to the oracle; the slot carries another sequence's state before each."""
    cfg, raw, toks, want, _ = setup(name)
    n = len(toks)
    dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_batch=2, max_seq_len=n)
    cuts = {"whole": [n], "decode": [n - 40] + [1] * 40, "tokens": [1] * n, "pairs": [2] * (n // 2),
            "portions": [2, 3, 9, 1, 16, 33, 2, 64, n - 130]}
    for what, c in cuts.items():
        err = M.row_error(run(dec, toks, c, seq=1), want)
        assert err.max() <= LIMIT[dtype], f"{what}: {err.max():.2e} at {int(err.argmax())}"
    tl.check_device_errors()
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_residual_after_every_layer_run(dtype):
    cfg, raw, toks, _, taps = setup("all")
    dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_seq_len=len(toks))
    _, got = dec.forward_logits(0, ids(toks), 0, [], taps=True)
    assert got.shape == taps.shape
    for r in range(len(taps)):
        err = np.abs(got[r].double().cpu().numpy() - taps[r]).max() / np.abs(taps[r]).max()
        assert err <= {"float32": 1e-4, "bfloat16": 5e-2}[dtype], f"layer run {r}: {err:.2e}"
    dec.close()


def test_a_far_token_is_found_again():
    """Attention whose query reaches a token hundreds of positions back, through the prompt and
    through the decode kernels: the logits change when that one token changes, as the oracle's do."""
    cfg = M.config([M.attention(heads=2, dim=16, rot_dim=2, vdim=32, kv_rank=32, base=2e5, scale=2.0)], width=48, vocab=61)
    raw, W = M.finder_model(cfg, 77)
    toks = np.random.default_rng(3).integers(0, 60, 400).astype(np.int32)
    toks[3] = 60                              # the only token of its kind
    other = toks.copy()
    other[3] = 1
    want, want2 = O.forward(cfg, W, toks), O.forward(cfg, W, other)
    moved = np.sqrt(((want - want2) ** 2).mean(axis=1)) / np.std(want)
    far = [t for t in range(300, 400) if moved[t] > 0.2]
    assert far                                # the case is what it says
    for dtype in LIMIT:
        dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_seq_len=400)
        for cuts in ([400], [300] + [1] * 100, [190, 2, 100, 108]):
            err = M.row_error(run(dec, toks, cuts), want)
            assert err.max() <= LIMIT[dtype] and err[far].max() <= LIMIT[dtype], f"{dtype} {cuts[:3]}: {err.max():.2e}"
        dec.close()


def test_slots_are_independent_and_used_again():
    """Requests of unequal length interleaved over two slots that change owners."""
    cfg, raw, toks, want, _ = setup("all")
    dec = tl.Decoder(M.model(cfg, raw), dtype="float32", max_batch=3, max_seq_len=160)
    toks2 = np.random.default_rng(11).integers(0, cfg["vocab"], 90).astype(np.int32)
    _, W = M.random_model(cfg, sum(map(ord, "all")))
    want2 = O.forward(cfg, W, toks2)
    a = [dec.forward_logits(2, ids(toks[:70]), 0, [69])]
    b = [dec.forward_logits(0, ids(toks2[:33]), 0, [0, 32])]
    a.append(dec.forward_logits(2, ids(toks[70:72]), 70, [0, 1]))
    b.append(dec.forward_logits(0, ids(toks2[33:90]), 33, [56]))
    a.append(dec.forward_logits(2, ids(toks[72:150]), 72, [77]))
    c = dec.forward_logits(0, ids(toks[:60]), 0, [59])           # slot 0 starts anew
    for got, w in ((torch.cat(a), want[[69, 70, 71, 149]]), (torch.cat(b), want2[[0, 32, 89]]), (c, want[[59]])):
        assert M.row_error(got.cpu().numpy(), w).max() <= LIMIT["float32"]
    for bad in (59, 61, 149):                                     # a recurrent state cannot be rewound
        with pytest.raises(tl.TllmError, match="continue"):
            dec.forward_logits(0, ids(toks[:1]), bad, [])
    with pytest.raises(tl.TllmError):
        dec.forward_logits(3, ids(toks[:1]), 0, [])
    with pytest.raises(tl.TllmError):
        dec.forward_logits(0, ids(toks[:2]), 0, [2])
    with pytest.raises(tl.TllmError):
        dec.forward_logits(0, ids(np.zeros(161)), 0, [])
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("batch", [2, 5, 12])
def test_lock_step_batches(batch, dtype):
    """One token of several sequences per step against each sequence in the oracle."""
    cfg, raw, _, _, _ = setup("all")
    _, W = M.random_model(cfg, sum(map(ord, "all")))
    rng = np.random.default_rng(batch)
    toks = rng.integers(0, cfg["vocab"], (batch, 74)).astype(np.int32)
    dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_batch=batch, max_seq_len=80)
    want = [O.forward(cfg, W, t) for t in toks]
    for b in range(batch):
        last = dec.forward_seq(b, ids(toks[b, :70]), 0)
        assert last.dtype == torch.float32
        assert M.row_error(last.cpu().numpy()[None], want[b][69:70]).max() <= LIMIT[dtype]
    for t in range(70, 74):
        got = dec.forward_batch(ids(toks[:, t]), t).cpu().numpy()
        for b in range(batch):
            err = M.row_error(got[b][None], want[b][t:t + 1]).max()
            assert err <= LIMIT[dtype], f"sequence {b} position {t}: {err:.2e}"
    dec.close()


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_greedy_generation_through_the_graph_replayed_loop(dtype):
    """generate() against the oracle fed with the same tokens: every token is the oracle's best
    (or within rounding of it), over a long run, from a prompt, from nothing, and continued."""
    cfg, raw, toks, _, _ = setup("all")
    _, W = M.random_model(cfg, sum(map(ord, "all")))
    dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_seq_len=400)
    slack = LIMIT[dtype] * 6

    def check(seq, n_prompt):
        lg = O.forward(cfg, W, seq)
        for p in range(n_prompt - 1, len(seq) - 1):
            assert lg[p, seq[p + 1]] >= lg[p].max() - slack * lg[p].std(), f"position {p}"

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
    # the same tokens step by step through forward()
    dec.forward(ids(toks[:20]), 0)
    tok = first
    for i in range(12):
        tok_next = int(dec.forward(ids([tok]), 20 + i).argmax())
        assert tok_next == out[i]
        tok = tok_next
    with pytest.raises(tl.TllmError, match="continue"):
        dec.generate(tok, 40, 2)
    dec.close()


def test_generation_from_the_command_line(tmp_path):
    cfg, raw, toks, _, _ = setup("one_layer_loop", n=60)
    write_model(str(tmp_path / "m"), cfg, raw)
    r = subprocess.run([sys.executable, "-m", "ternary_llm_b200.generate", "--model", str(tmp_path / "m"), "--tokens",
                        ",".join(map(str, toks[:12])), "--steps", "9", "--dtype", "float32"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    dec = tl.Decoder(str(tmp_path / "m"), dtype="float32", max_seq_len=64)
    tok, want = int(dec.forward(ids(toks[:12]), 0).argmax()), []
    for i in range(9):
        want.append(tok)
        tok = int(dec.forward(ids([tok]), 12 + i).argmax())
    assert [int(v) for v in r.stdout.strip().splitlines()[-1].split(",")] == want
    dec.close()


def test_prompt_longer_than_one_pass_through_the_layers():
    """A prompt of more tokens than the activation buffers hold goes through in portions, wanted
    logits from each; decode steps far behind it read the whole cache."""
    cfg = M.config([M.attention(heads=2, dim=8, rot_dim=8, vdim=16, kv_rank=16), M.mamba(inner=16, state=4, dt_rank=2), M.rglru(width=16, blocks=2)],
                   width=24, vocab=40)
    raw, _ = M.random_model(cfg, 8)
    n = 2300
    toks = np.random.default_rng(8).integers(0, 40, n).astype(np.int32)
    want_at = [0, 2047, 2048, 2049, 2299]
    ref = tl.Decoder(M.model(cfg, raw), dtype="float32", max_seq_len=n)
    want = []
    pos = 0
    for c in (1000, 1047, 1, 1, 251):                            # other cuts, the same sequence
        want.append(ref.forward_logits(0, ids(toks[pos:pos + c]), pos, list(range(c))))
        pos += c
    want = torch.cat(want).double().cpu().numpy()
    for dtype in LIMIT:
        dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_seq_len=n)
        got = dec.forward_logits(0, ids(toks), 0, want_at).cpu().numpy()
        assert M.row_error(got, want[want_at]).max() <= LIMIT[dtype]
        last = dec.forward(ids(toks), 0)
        assert M.row_error(last.cpu().numpy()[None], want[-1:]).max() <= LIMIT[dtype]
        got = np.concatenate([dec.forward_logits(0, ids(toks[:2290]), 0, []).cpu().numpy().reshape(0, 40)] +
                             [dec.forward_logits(0, ids(toks[p:p + 1]), p, [0]).cpu().numpy() for p in range(2290, 2300)])
        assert M.row_error(got, want[2290:]).max() <= LIMIT[dtype]
        dec.close()
    ref.close()


def test_sizes_of_a_real_layer_agree_between_the_two_precisions():
    """Wide layers take other kernel instances (two-wide GEMM tiles, long latents); BF16 against
    the 32-bit mode on the same weights."""
    cfg = M.config([M.attention(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, ff=1024), M.mamba(inner=1024, state=16, dt_rank=32, ff=512),
                    M.rglru(width=1280, blocks=10, conv=4)], width=640, vocab=1000)
    raw, _ = M.random_model(cfg, 3)
    toks = np.random.default_rng(0).integers(0, 1000, 300).astype(np.int32)
    out = {}
    for dtype in LIMIT:
        dec = tl.Decoder(M.model(cfg, raw), dtype=dtype, max_seq_len=320)
        out[dtype] = [run(dec, toks, c) for c in ([300], [280] + [1] * 20, [100, 9, 150, 2, 39])]
        tl.check_device_errors()
        dec.close()
    for a, b in zip(out["float32"], out["bfloat16"]):
        assert M.row_error(a, out["float32"][0]).max() <= LIMIT["float32"]
        assert M.row_error(b, out["float32"][0]).max() <= LIMIT["bfloat16"]


def test_trace_replay_program(tmp_path):
    cfg, raw, toks, want, _ = setup("one_layer_loop", n=60)
    write_model(str(tmp_path / "m"), cfg, raw)
    os.makedirs(tmp_path / "out")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:50].tolist(), "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[50:51].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[51:60].tolist(), "want": [0, 8]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:9].tolist(), "want": [8]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600,
                       env=dict(os.environ, PATH=os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"]))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [s for s in r.stdout.splitlines() if s.startswith("done")] == [f"done {i}" for i in range(4)]
    for step, places in ((0, [49, 3]), (2, [51, 59]), (3, [8])):
        got = np.fromfile(tmp_path / "out" / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert M.row_error(got, want[places]).max() <= LIMIT["float32"]
    assert not os.path.exists(tmp_path / "out" / "1.f32")
