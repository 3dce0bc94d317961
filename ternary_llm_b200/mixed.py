"""Models made of a list of mixer layers (include/tllm_b200_mixed.h): the description that the
C decoder takes, and the designs that map onto it.

Petulix: latent attention with a softmax sink and an output gate, Mamba, and Griffin's RG-LRU
block in any order, a norm before and after every sublayer, an optional gated feed-forward per
layer, a run of layers repeated with the embedding output added before each further pass, and
the embedding table as output head.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np

from . import _lib
from .models import register

LATENT_ATTENTION, SELECTIVE_SCAN, GATED_RECURRENCE = 1, 2, 3
ACTIVATIONS = {None: 0, "gelu_tanh": 1, "silu": 2}

# order of the TLLM_T_... enumeration
TENSOR_SLOTS = ("norm1", "norm1b", "norm2", "norm2b", "gate", "up", "down", "out",
                "q", "kv_down", "kv_norm", "k_up", "v_up", "sink", "head_gate",
                "in", "in_bias", "conv", "conv_bias", "x", "dt", "dt_bias", "a_log", "d",
                "y", "y_bias", "ra", "ra_bias", "ri", "ri_bias", "lam")


@dataclass
class MixedLayer:
    """Sizes of one layer and its tensors (slot of TENSOR_SLOTS -> array of BF16 bit patterns or
    a torch BF16 tensor)."""
    type: int
    sizes: dict                                   # fields of tllm_b200_mixed_layer
    tensors: dict
    shapes: dict = field(default_factory=dict)    # slot -> shape the sizes imply


@dataclass
class MixedModel:
    vocab_size: int
    width: int
    norm_eps: float
    layers: list
    embedding: object
    final_norm: object
    loop: tuple = (0, 0, 1, False)                # start, stop, times, add the embedding output before further passes
    architecture = "mixed"

    def check(self) -> None:
        """Every tensor has the shape that the sizes imply."""
        def shape(name, t, want):
            if tuple(t.shape) != tuple(want):
                raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration implies {tuple(want)}")
        shape("embedding", self.embedding, (self.vocab_size, self.width))
        shape("final norm", self.final_norm, (self.width,))
        for i, layer in enumerate(self.layers):
            for slot, t in layer.tensors.items():
                shape(f"{slot} of layer {i}", t, layer.shapes[slot])

    def fill_desc(self, up, max_seq_len: int):
        """tllm_b200_mixed_desc for this model; up(array) -> device pointer."""
        self.check()
        layers = (_lib.MixedLayerDesc * len(self.layers))()
        for dst, layer in zip(layers, self.layers):
            dst.type = layer.type
            for k, v in layer.sizes.items():
                setattr(dst, k, v)
            for slot, t in layer.tensors.items():
                dst.t[TENSOR_SLOTS.index(slot)] = up(t)
        d = _lib.MixedDesc()
        d.vocab_size, d.width, d.n_layers, d.max_seq_len = self.vocab_size, self.width, len(self.layers), max_seq_len
        d.norm_eps = self.norm_eps
        d.loop_start, d.loop_stop, d.loop_times, d.loop_inject = self.loop
        d.embedding, d.final_norm = up(self.embedding), up(self.final_norm)
        d.layers = layers
        return d


def _latent_attention(m, width):
    H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    sizes = dict(heads=H, dim=d, rot_dim=r, rot_dims=rot["dims"], vdim=e, kv_rank=R, scale=m["scale"], rot_base=rot["base"])
    names = {"q": ("q", (H * (d + r), width)), "kv_down": ("dkv", (R + r, width)), "kv_norm": ("dkv.norm", (R,)),
             "k_up": ("uk", (H * d, R)), "v_up": ("uv", (H * e, R)), "sink": ("sink", (H,)), "head_gate": ("g", (H, width)),
             "out": ("o", (width, H * e))}
    return LATENT_ATTENTION, sizes, names


def _mamba1(m, width):
    C, st, dr, taps = m["inner"], m["state"], m["dt_rank"], m["conv"]
    sizes = dict(channels=C, taps=taps, state=st, dt_rank=dr)
    names = {"in": ("in", (2 * C, width)), "conv": ("conv", (C, taps)), "conv_bias": ("conv.b", (C,)), "x": ("x", (dr + 2 * st, C)),
             "dt": ("dt", (C, dr)), "dt_bias": ("dt.b", (C,)), "a_log": ("A_log", (C, st)), "d": ("D", (C,)), "out": ("o", (width, C))}
    return SELECTIVE_SCAN, sizes, names


RGLRU_DECAY = 8.0


def _rglru(m, width):
    C, nb, taps = m["width"], m["blocks"], m["conv"]
    if nb < 1 or C % nb:
        raise ValueError(f"rglru: width {C} does not split into {nb} blocks")
    b = C // nb
    sizes = dict(channels=C, taps=taps, blocks=nb, decay=RGLRU_DECAY, gate_act=ACTIVATIONS["gelu_tanh"])
    names = {"y": ("y", (C, width)), "y_bias": ("y.b", (C,)), "in": ("x", (C, width)), "in_bias": ("x.b", (C,)),
             "conv": ("conv", (C, taps)), "conv_bias": ("conv.b", (C,)), "ra": ("ra", (nb, b, b)), "ra_bias": ("ra.b", (nb, b)),
             "ri": ("ri", (nb, b, b)), "ri_bias": ("ri.b", (nb, b)), "lam": ("lam", (C,)), "out": ("o", (width, C))}
    return GATED_RECURRENCE, sizes, names


_MIXERS = {"latent_attention": _latent_attention, "mamba1": _mamba1, "rglru": _rglru}


@register("Petulix")
class Petulix(MixedModel):
    @staticmethod
    def tensor_shapes(cfg: dict) -> dict:
        """File name -> shape of every tensor of a model with this configuration."""
        out = {"embed": (cfg["vocab"], cfg["width"])}
        for i, entry in enumerate(cfg["layers"]):
            _, _, names = Petulix._layer(cfg, i, entry)
            out.update({name: shape for name, shape in names.values()})
        out["final.norm"] = (cfg["width"],)
        return out

    @staticmethod
    def _layer(cfg, i, entry):
        w, p = cfg["width"], f"l{i}."
        if entry["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r} (known: {', '.join(sorted(_MIXERS))})")
        kind, sizes, mix = _MIXERS[entry["type"]](entry["mixer"], w)
        names = {"norm1": (p + "norm1", (w,)), "norm1b": (p + "norm1b", (w,))}
        names.update({slot: (p + "mix." + name, shape) for slot, (name, shape) in mix.items()})
        mlp = entry.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            ff = mlp["ff"]
            sizes.update(ff=ff, ff_act=ACTIVATIONS["gelu_tanh"])
            names.update({"norm2": (p + "norm2", (w,)), "norm2b": (p + "norm2b", (w,)), "gate": (p + "mlp.gate", (ff, w)),
                          "up": (p + "mlp.up", (ff, w)), "down": (p + "mlp.down", (w, ff))})
        return kind, sizes, names

    @classmethod
    def from_config(cls, cfg: dict, tensors) -> "Petulix":
        dtypes = getattr(tensors, "dtypes", {})

        def take(name):
            if name not in tensors:
                raise ValueError(f"tensor {name} is missing")
            if dtypes.get(name, "BF16") != "BF16":
                raise ValueError(f"tensor {name} is {dtypes[name]}, expected BF16")
            return tensors[name]

        layers = []
        for i, entry in enumerate(cfg["layers"]):
            kind, sizes, names = cls._layer(cfg, i, entry)
            layers.append(MixedLayer(kind, sizes, {slot: take(name) for slot, (name, _) in names.items()},
                                     {slot: shape for slot, (_, shape) in names.items()}))
        lp = cfg.get("loop")
        loop = (lp["start"], lp["stop"], lp["times"], True) if lp else (0, 0, 1, False)
        m = cls(cfg["vocab"], cfg["width"], cfg["norm"]["eps"], layers, take("embed"), take("final.norm"), loop)
        m.check()
        return m


def random_tensors(shapes: dict, seed: int, device=None) -> dict:
    """Seeded random BF16 weights for benchmarks and examples, file name -> tensor: matrices scaled
    by 1/sqrt(fan-in), norms 1, decays spread over their usual ranges.  With a device, torch
    tensors drawn there; else arrays of BF16 bit patterns."""
    import torch
    gen = torch.Generator(device=device or "cpu").manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        last = name.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=gen, device=device or "cpu")
        if last in ("norm1", "norm2", "norm1b", "norm2b", "norm"):
            t = torch.ones_like(t)
        elif last == "A_log":
            t = torch.log(torch.arange(1, shape[1] + 1, device=t.device, dtype=torch.float32)).expand(shape) + 0.1 * t
        elif last == "D":
            t = 1.0 + 0.1 * t
        elif name.endswith("dt.b"):
            t = t - 4.0
        elif last == "lam":
            t = 0.5 * t - 2.0
        elif last in ("b", "sink"):
            t = 0.1 * t
        elif name == "embed":
            t = t * shape[-1] ** -0.5
        else:
            t = t * shape[-1] ** -0.5
        t = t.to(torch.bfloat16).contiguous()
        out[name] = t if device is not None else t.view(torch.int16).numpy().view(np.uint16)
    return out
