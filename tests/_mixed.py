"""Small random models of mixer layers for the tests, in the form both sides take: a parsed
configuration and tensors by file name (BF16 bit patterns for the library, floats for the oracle)."""
import numpy as np

from ternary_llm_b200 import safetensors_io as st
from ternary_llm_b200.mixed import Petulix


def attention(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=40, base=10000.0, ff=None, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba(inner=56, state=12, dt_rank=5, conv=4, ff=None):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def rglru(width=60, blocks=5, conv=3, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=44, vocab=101, loop=None, eps=1e-5):
    return {"architecture": "Petulix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "loop": loop or {"start": 0, "stop": len(layers), "times": 1}}


def random_model(cfg, seed):
    """(tensors as BF16 bit patterns, the same as floats).  Attention is sharpened (queries scaled
    up), sinks are of the size of the scores, decays leave memories from a few to thousands of
    tokens, and norm weights, biases and skip terms all differ from 0 and 1."""
    rng = np.random.default_rng(seed)
    raw = {}
    for name, shape in Petulix.tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        a = rng.standard_normal(shape)
        if last in ("norm1", "norm2", "norm1b", "norm2b", "norm"):
            a = 1.0 + 0.3 * a
        elif last == "A_log":
            a = np.log(rng.uniform(0.02, 8.0, shape))
        elif name.endswith("dt.b"):
            a = a - 2.0
        elif last == "lam":
            a = 2.0 * a - 5.0
        elif last == "sink":
            a = 1.0 + a
        elif last in ("b", "D", "conv"):
            a = 0.5 * a
        elif last == "q":
            a = a * 2.0 * shape[-1] ** -0.5
        elif name != "embed":
            a = a * shape[-1] ** -0.5
        raw[name] = st.to_bf16(a.astype(np.float32))
    return raw, {k: st.from_bf16(v).astype(np.float64) for k, v in raw.items()}


def finder_model(cfg, seed):
    """A model of one attention layer whose every query picks the last vocabulary entry, however
    far back: that entry alone has a component which the first latent reads, the first key
    dimension repeats it, and the first query dimension is the same for all tokens."""
    raw, W = random_model(cfg, seed)
    m = cfg["layers"][0]["mixer"]
    per = m["dim"] + m["rot_dim"]
    e = 0.5 * W["embed"]
    e[:, 0], e[:, 1] = 2.0, 0.0
    e[-1] = 0.0
    e[-1, 0], e[-1, 1] = 2.0, 8.0
    q, dkv, uk = 0.3 * W["l0.mix.q"], 0.3 * W["l0.mix.dkv"], 0.3 * W["l0.mix.uk"]
    dkv[0] = 0.0
    dkv[0, 1] = 1.0
    for h in range(m["heads"]):
        q[h * per], uk[h * m["dim"]] = 0.0, 0.0
        q[h * per, 0], uk[h * m["dim"], 0] = 0.75, 1.0
    W.update({"embed": e, "l0.mix.q": q, "l0.mix.dkv": dkv, "l0.mix.uk": uk, "l0.norm1": 0 * W["l0.norm1"] + 1,
              "l0.mix.dkv.norm": 0 * W["l0.mix.dkv.norm"] + 1, "l0.mix.sink": 0 * W["l0.mix.sink"]})
    raw = {k: st.to_bf16(v.astype(np.float32)) for k, v in W.items()}
    return raw, {k: st.from_bf16(v).astype(np.float64) for k, v in raw.items()}


def model(cfg, raw):
    return Petulix.from_config(cfg, raw)


def row_error(got, want):
    """Root mean square of the difference per row (means taken off), relative to the spread of
    the expected logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.std(want)
