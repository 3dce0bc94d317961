"""Models made of a list of mixer layers (include/tllm_b200_mixed.h): the description that the
C decoder takes, and the designs that map onto it.

Petulix: latent attention with a softmax sink and an output gate, Mamba, and Griffin's RG-LRU
block in any order, a norm before and after every sublayer, an optional gated feed-forward per
layer, a run of layers repeated with the embedding output added before each further pass, and
the embedding table as output head.

Femolix: gated delta rule, or chunk-local grouped-query attention beside linear attention of
constant decay, in any order; a norm behind every sum of scaled residual and sublayer; a dense
feed-forward, a mixture of experts or none per layer; a head of its own with a soft cap.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field

import numpy as np

from . import _lib
from .models import register

LATENT_ATTENTION, SELECTIVE_SCAN, GATED_RECURRENCE, ATTENTION, LINEAR_ATTENTION, DELTA_RULE = range(1, 7)
ACTIVATIONS = {None: 0, "gelu_tanh": 1, "silu": 2, "sigmoid": 4}

# order of the TLLM_T_... enumeration
TENSOR_SLOTS = ("norm1", "norm1b", "norm2", "norm2b", "gate", "up", "down", "out",
                "q", "kv_down", "kv_norm", "k_up", "v_up", "sink", "head_gate",
                "in", "in_bias", "conv", "conv_bias", "x", "dt", "dt_bias", "a_log", "d",
                "y", "y_bias", "ra", "ra_bias", "ri", "ri_bias", "lam",
                "k", "v", "q_norm", "k_norm", "q_conv", "k_conv", "v_conv", "step", "decay_in", "mix_norm", "mix_gate", "router")


@dataclass
class MixedLayer:
    """Sizes of one layer and its tensors (slot of TENSOR_SLOTS -> array of BF16 bit patterns or
    a torch BF16 tensor; a list of equal ones is laid out one behind the other)."""
    type: int
    sizes: dict                                   # fields of tllm_b200_mixed_layer
    tensors: dict
    shapes: dict = field(default_factory=dict)    # slot -> shape the sizes imply (of each in a list)
    head_decay: object = None                     # floats, one per head
    beside: "MixedLayer | None" = None            # a second mixer added to this layer's


@dataclass
class MixedModel:
    vocab_size: int
    width: int
    norm_eps: float
    layers: list
    embedding: object
    final_norm: object
    loop: tuple = (0, 0, 1, False)                # start, stop, times, add the embedding output before further passes
    head: object = None                           # None: the embedding
    residual_scale: float | None = None           # not None: norm(scale * x + sublayer(x)) instead of x + sublayer(norm(x))
    logit_softcap: float = 0.0
    architecture = "mixed"

    def check(self) -> None:
        """Every tensor has the shape that the sizes imply."""
        def shape(name, t, want):
            if tuple(t.shape) != tuple(want):
                raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration implies {tuple(want)}")

        def mixer(layer, i):
            for slot, t in layer.tensors.items():
                for one in t if isinstance(t, list) else [t]:
                    shape(f"{slot} of layer {i}", one, layer.shapes[slot])
            if layer.head_decay is not None and len(layer.head_decay) != layer.sizes["heads"]:
                raise ValueError(f"layer {i}: {len(layer.head_decay)} decays for {layer.sizes['heads']} heads")
            if layer.beside is not None:
                mixer(layer.beside, i)

        shape("embedding", self.embedding, (self.vocab_size, self.width))
        shape("final norm", self.final_norm, (self.width,))
        if self.head is not None:
            shape("head", self.head, (self.vocab_size, self.width))
        for i, layer in enumerate(self.layers):
            mixer(layer, i)

    def fill_desc(self, up, max_seq_len: int):
        """tllm_b200_mixed_desc for this model; up(array or list of arrays) -> device pointer."""
        self.check()
        keep = []                                 # what the structures point to

        def fill(dst, layer):
            dst.type = layer.type
            for k, v in layer.sizes.items():
                setattr(dst, k, v)
            for slot, t in layer.tensors.items():
                dst.t[TENSOR_SLOTS.index(slot)] = up(t)
            if layer.head_decay is not None:
                dst.head_decay = (ctypes.c_float * len(layer.head_decay))(*layer.head_decay)
            if layer.beside is not None:
                other = _lib.MixedLayerDesc()
                fill(other, layer.beside)
                keep.append(other)
                dst.beside = ctypes.addressof(other)

        layers = (_lib.MixedLayerDesc * len(self.layers))()
        for dst, layer in zip(layers, self.layers):
            fill(dst, layer)
        d = _lib.MixedDesc()
        d.vocab_size, d.width, d.n_layers, d.max_seq_len = self.vocab_size, self.width, len(self.layers), max_seq_len
        d.norm_eps = self.norm_eps
        d.loop_start, d.loop_stop, d.loop_times, d.loop_inject = self.loop
        d.norm_after_sum, d.residual_scale = self.residual_scale is not None, self.residual_scale or 0.0
        d.logit_softcap = self.logit_softcap
        d.embedding, d.final_norm = up(self.embedding), up(self.final_norm)
        d.head = up(self.head) if self.head is not None else None
        d.layers = layers
        d.keep = keep
        return d


def _taker(tensors):
    """name -> BF16 tensor of a model file, with the refusals."""
    dtypes = getattr(tensors, "dtypes", {})

    def take(name):
        if isinstance(name, list):
            return [take(n) for n in name]
        if name not in tensors:
            raise ValueError(f"tensor {name} is missing")
        if dtypes.get(name, "BF16") != "BF16":
            raise ValueError(f"tensor {name} is {dtypes[name]}, expected BF16")
        return tensors[name]

    return take


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
        take = _taker(tensors)
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


# ---- Femolix -------------------------------------------------------------------------------
def _delta(m, width, prefix):
    H, G, d, e, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    sizes = dict(heads=H, kv_heads=G, dim=d, vdim=e, taps=taps, in_act=ACTIVATIONS["silu"], gate_act=ACTIVATIONS["silu"], out_scale=1.0)
    names = {"q": ("q", (G * d, width)), "k": ("k", (G * d, width)), "v": ("v", (H * e, width)), "q_conv": ("q.conv", (G * d, taps)),
             "k_conv": ("k.conv", (G * d, taps)), "v_conv": ("v.conv", (H * e, taps)), "step": ("b", (H, width)), "decay_in": ("a", (H, width)),
             "a_log": ("A_log", (H,)), "dt_bias": ("dt_bias", (H,)), "mix_norm": ("norm", (e,)), "mix_gate": ("g", (H * e, width)),
             "out": ("o", (width, H * e))}
    return DELTA_RULE, sizes, {slot: (prefix + n, shape) for slot, (n, shape) in names.items()}


def _chunked_attention(m, width, prefix, out_scale):
    H, G, d, e, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    sizes = dict(heads=H, kv_heads=G, dim=d, vdim=e, rot_dims=rot["dims"], rot_base=rot["base"], scale=m["scale"], chunk=m["mask"]["size"],
                 out_scale=out_scale)
    names = {"q": ("q", (H * d, width)), "k": ("k", (G * d, width)), "v": ("v", (G * e, width)), "q_norm": ("q.norm", (d,)),
             "k_norm": ("k.norm", (d,)), "out": ("o", (width, H * e))}
    return ATTENTION, sizes, {slot: (prefix + n, shape) for slot, (n, shape) in names.items()}


def _lightning(m, width, prefix, out_scale):
    H, d, e = m["heads"], m["dim"], m["vdim"]
    sizes = dict(heads=H, kv_heads=H, dim=d, vdim=e, in_act=ACTIVATIONS["silu"], gate_act=ACTIVATIONS["sigmoid"], out_scale=out_scale)
    names = {"q": ("q", (H * d, width)), "k": ("k", (H * d, width)), "v": ("v", (H * e, width)), "mix_norm": ("norm", (H * e,)),
             "mix_gate": ("g", (H * e, width)), "out": ("o", (width, H * e))}
    return LINEAR_ATTENTION, sizes, {slot: (prefix + n, shape) for slot, (n, shape) in names.items()}


@register("Femolix")
class Femolix(MixedModel):
    @staticmethod
    def tensor_shapes(cfg: dict) -> dict:
        """File name -> shape of every tensor of a model with this configuration."""
        out = {"embed": (cfg["vocab"], cfg["width"])}
        for i, entry in enumerate(cfg["layers"]):
            for _, _, names in Femolix._mixers(cfg, i, entry):
                for name, shape in names.values():
                    out.update({n: shape for n in (name if isinstance(name, list) else [name])})
        out["final.norm"] = (cfg["width"],)
        out["head"] = (cfg["vocab"], cfg["width"])
        return out

    @staticmethod
    def _mixers(cfg, i, entry):
        """(type, sizes, slot -> (file name or names, shape)) of the layer, then of the mixer beside it."""
        w, p, m = cfg["width"], f"l{i}.", entry["mixer"]
        if entry["type"] == "delta":
            mixers = [_delta(m, w, p + "mix.")]
        elif entry["type"] == "parallel":
            mixers = [_chunked_attention(m["left"], w, p + "mix.left.", m["left_scale"]),
                      _lightning(m["right"], w, p + "mix.right.", m["right_scale"])]
        else:
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r} (known: delta, parallel)")
        _, sizes, names = mixers[0]
        names["norm1"] = (p + "norm1", (w,))
        mlp = entry.get("mlp")
        if mlp is None:
            return mixers
        if mlp["kind"] not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        names["norm2"] = (p + "norm2", (w,))
        sizes["ff_act"] = ACTIVATIONS["silu"]
        if mlp["kind"] == "dense":
            ff = sizes["ff"] = mlp["ff"]
            names.update({"gate": (p + "mlp.gate", (ff, w)), "up": (p + "mlp.up", (ff, w)), "down": (p + "mlp.down", (w, ff))})
            return mixers
        ff, n, top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
        if not 1 <= top <= n:
            raise ValueError(f"layer {i}: {top} of {n} experts")
        sizes.update(ff=ff, experts=n, top=top)
        names["router"] = (p + "mlp.router", (n, w))
        for slot, shape in (("gate", (ff, w)), ("up", (ff, w)), ("down", (w, ff))):
            names[slot] = ([f"{p}mlp.e{e}.{slot}" for e in range(n)], shape)
        return mixers

    @classmethod
    def from_config(cls, cfg: dict, tensors) -> "Femolix":
        take = _taker(tensors)
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            made = [MixedLayer(kind, sizes, {slot: take(name) for slot, (name, _) in names.items()},
                               {slot: shape for slot, (_, shape) in names.items()}) for kind, sizes, names in cls._mixers(cfg, i, entry)]
            if len(made) == 2:
                made[0].beside = made[1]
                made[1].head_decay = list(entry["mixer"]["right"]["decay"])
            layers.append(made[0])
        m = cls(cfg["vocab"], cfg["width"], cfg["norm"]["eps"], layers, take("embed"), take("final.norm"), head=take("head"),
                residual_scale=cfg["postln_alpha"], logit_softcap=cfg["logit_softcap"])
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
            t = torch.log(torch.arange(1, shape[-1] + 1, device=t.device, dtype=torch.float32)).expand(shape) + 0.1 * t
        elif last == "D":
            t = 1.0 + 0.1 * t
        elif name.endswith("dt.b") or last == "dt_bias":
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
