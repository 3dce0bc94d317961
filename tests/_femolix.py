"""Small random models of the Femolix design for the tests: a parsed configuration, tensors by file
name (BF16 bit patterns for the library, floats for the oracle), and models planted so that one
token decides the result."""
import numpy as np

from ternary_llm_b200 import safetensors_io as st
from ternary_llm_b200.mixed import Femolix
from tests._mixed import row_error  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def parallel(heads=6, kv_heads=2, dim=16, vdim=12, size=37, base=5000.0, rot=8, scale=0.4, r_heads=3, r_dim=10, r_vdim=14, decay=None, left=0.7,
             right=0.45, mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                               "rot": {"base": base, "dims": rot}, "scale": scale}, "left_scale": left, "right_scale": right,
                      "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay or np.linspace(0.55, 0.9995, r_heads).tolist()}}}


def config(layers, width=44, vocab=101, eps=1e-5, alpha=1.7, cap=9.0):
    return {"architecture": "Femolix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha,
            "logit_softcap": cap}


def random_model(cfg, seed):
    """(tensors as BF16 bit patterns, the same as floats).  Decays leave memories from a token to
    thousands, routers are decided, norm weights differ from 1, and the head is large enough for
    the soft cap to bend the logits."""
    rng = np.random.default_rng(seed)
    raw = {}
    for name, shape in Femolix.tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        a = rng.standard_normal(shape)
        if last in ("norm1", "norm2", "norm"):
            a = 1.0 + 0.3 * a
        elif last == "A_log":
            a = np.log(rng.uniform(0.001, 4.0, shape))
        elif last == "dt_bias":
            a = a - 1.5
        elif last == "conv":
            a = 0.7 * a
        elif last == "router":
            a = a * 3.0 * shape[-1] ** -0.5
        elif last == "head":
            a = a * 6.0 * shape[-1] ** -0.5
        elif name != "embed":
            a = a * shape[-1] ** -0.5
        raw[name] = st.to_bf16(a.astype(np.float32))
    return raw, {k: st.from_bf16(v).astype(np.float64) for k, v in raw.items()}


def model(cfg, raw):
    return Femolix.from_config(cfg, raw)


def refloat(W):
    raw = {k: st.to_bf16(v.astype(np.float32)) for k, v in W.items()}
    return raw, {k: st.from_bf16(v).astype(np.float64) for k, v in raw.items()}


def finder_model(cfg, seed):
    """One `parallel` layer whose every query picks the last vocabulary entry if its chunk holds it:
    that entry alone has a component which the last key dimension (not rotated) reads, and the last
    query dimension is the same for all tokens."""
    raw, W = random_model(cfg, seed)
    m = cfg["layers"][0]["mixer"]["left"]
    assert m["rot"]["dims"] < m["dim"]
    e = 0.5 * W["embed"]
    e[:, 0], e[:, 1] = 2.0, 0.0
    e[-1, 1] = 8.0
    q, k = 0.2 * W["l0.mix.left.q"], 0.1 * W["l0.mix.left.k"]
    for h in range(m["heads"]):
        q[(h + 1) * m["dim"] - 1] = 0.0
        q[(h + 1) * m["dim"] - 1, 0] = 2.0
    for g in range(m["kv_heads"]):
        k[(g + 1) * m["dim"] - 1] = 0.0
        k[(g + 1) * m["dim"] - 1, 1] = 2.0
    W.update({"embed": e, "l0.mix.left.q": q, "l0.mix.left.k": k, "l0.mix.left.v": 2.0 * W["l0.mix.left.v"],
              "l0.mix.left.q.norm": 0 * W["l0.mix.left.q.norm"] + 1, "l0.mix.left.k.norm": 0 * W["l0.mix.left.k.norm"] + 1})
    return refloat(W)
