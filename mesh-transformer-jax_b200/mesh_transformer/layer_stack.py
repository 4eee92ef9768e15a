"""Layer-stack models: configuration, tensor names and random initialisation.

Configuration keys (config.json):
    architecture, vocab, width, norm {eps}
    layers: list of {type, mixer, mlp}; mlp {kind "dense", ff} or null
Keselix (RMS norms before and after every sublayer, SwiGLU feed-forwards), further keys
    residual_mult
    loop: {start, stop, times} or absent
    type "latent_attention", mixer {heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {base, dims}}
    type "mamba1",           mixer {inner, state, conv, dt_rank}
Bavutar (a layer norm behind every residual sum, squared-relu feed-forwards), further keys
    postln_alpha, embedding {scale}, logit_softcap
    type "attention",        mixer {heads, kv_heads, dim, vdim, scale, q_temp {coef, every}, kv_from}; the last two may be
                             absent
    type "mamba2",           mixer {heads, vdim, state, groups, conv, norm_groups}
    type "channel_delta",    mixer {heads, kv_heads, dim, vdim, conv}; the widths of its low-rank decay and gate
                             projections are the tensors' (``decay_rank``, ``gate_rank``, filled in by ``fit_tensors``)
A mixer is described once, in MIXERS, and any family may list it.

Runtime keys a caller may add: ``seq`` (longest prompt, default 2048), ``mtj_dtype`` ("bfloat16", the default, or
"float32": fp32 activations and caches throughout), ``mtj_tc_min_rows`` (prompt rows from which a call takes the
tensor-core path).

Tensors keep their own names ("embed", "l0.mix.q", ...) as the leaves of one module; linear weights are [out, in].
"""
from __future__ import annotations

import ctypes

import numpy as np
import torch

from . import registry
from ._lib import MtjConfig, MtjLayerDesc, MtjStackDesc, lib

MODULE = "layer_stack"
DTYPES = ("bfloat16", "float32")
SANDWICH_RMS, POST_LN = 0, 1                         # MTJ_RESIDUAL_*
SWIGLU, SQUARED_RELU = 0, 1                          # MTJ_FF_*


# ------------------------------------------------------------------- mixers ----
class LatentAttention:
    code = 0                                         # MTJ_MIXER_*

    @staticmethod
    def shapes(m, d):
        H, r = m["heads"], m["rot_dim"]
        return {"q": (H * (m["dim"] + r), d), "dkv": (m["kv_rank"] + r, d), "dkv.norm": (m["kv_rank"],),
                "uk": (H * m["dim"], m["kv_rank"]), "uv": (H * m["vdim"], m["kv_rank"]), "o": (d, H * m["vdim"])}

    @staticmethod
    def describe(m, desc):
        for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"):
            setattr(desc, k, m[k])
        desc.window, desc.rot_base = m["mask"]["size"], m["rot"]["base"]

    @staticmethod
    def check(m):
        if m["rot"].get("dims", m["rot_dim"]) != m["rot_dim"]:
            raise NotImplementedError("the rotated part is rotated as a whole")


class Mamba1:
    code = 1

    @staticmethod
    def shapes(m, d):
        n = m["inner"]
        return {"in": (2 * n, d), "conv": (n, m["conv"]), "conv.b": (n,), "dt.b": (n,), "D": (n,),
                "x": (m["dt_rank"] + 2 * m["state"], n), "dt": (n, m["dt_rank"]), "A_log": (n, m["state"]), "o": (d, n)}

    @staticmethod
    def describe(m, desc):
        for k in ("inner", "state", "conv", "dt_rank"):
            setattr(desc, k, m[k])

    @staticmethod
    def check(m):
        pass


class GroupedAttention:
    code = 2

    @staticmethod
    def shapes(m, d):
        nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        out = {"q": (nq, d), "q.norm": (nq,), "o": (d, m["heads"] * m["vdim"])}
        if m.get("kv_from") is None:
            out.update({"k": (nk, d), "k.norm": (nk,), "v": (m["kv_heads"] * m["vdim"], d)})
        return out

    @staticmethod
    def describe(m, desc):
        for k in ("heads", "kv_heads", "dim", "vdim", "scale"):
            setattr(desc, k, m[k])
        if m.get("kv_from") is not None:
            desc.kv_from = m["kv_from"]
        if m.get("q_temp"):
            desc.q_temp_coef, desc.q_temp_every = m["q_temp"]["coef"], m["q_temp"]["every"]

    @staticmethod
    def check(m):
        if m["heads"] % m["kv_heads"]:
            raise ValueError("heads must be a multiple of kv_heads")
        if m.get("q_temp") and not m["q_temp"]["every"] > 0:
            raise ValueError("q_temp.every must be positive")


class Mamba2:
    code = 3

    @staticmethod
    def shapes(m, d):
        H, inner = m["heads"], m["heads"] * m["vdim"]
        ch = inner + 2 * m["groups"] * m["state"]
        return {"in": (inner + ch + H, d), "conv": (ch, m["conv"]), "conv.b": (ch,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                "norm": (inner,), "o": (d, inner)}

    @staticmethod
    def describe(m, desc):
        for k in ("heads", "vdim", "conv", "norm_groups"):
            setattr(desc, k, m[k])
        desc.dim, desc.kv_heads = m["state"], m["groups"]

    @staticmethod
    def check(m):
        if m["heads"] % m["groups"] or m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ValueError("heads must be a multiple of groups, and inner of norm_groups")


class ChannelDelta:
    code = 4
    RANKS = {"decay_rank": "a1", "gate_rank": "g1"}  # widths that only the tensors tell

    @staticmethod
    def shapes(m, d):
        H, n, nv = m["heads"], m["dim"], m["vdim"]
        out = {"b": (H, d), "A_log": (H,), "dt_bias": (H * n,), "norm": (nv,), "o": (d, H * nv),
               "a1": (m["decay_rank"], d), "a2": (H * n, m["decay_rank"]), "g1": (m["gate_rank"], d), "g2": (H * nv, m["gate_rank"])}
        for name, rows in (("q", m["kv_heads"] * n), ("k", m["kv_heads"] * n), ("v", H * nv)):
            out[name], out[name + ".conv"] = (rows, d), (rows, m["conv"])
        return out

    @staticmethod
    def describe(m, desc):
        for k in ("heads", "kv_heads", "dim", "vdim", "conv", "decay_rank", "gate_rank"):
            setattr(desc, k, m[k])

    @staticmethod
    def check(m):
        if m["heads"] % m["kv_heads"]:
            raise ValueError("heads must be a multiple of kv_heads")
        if "decay_rank" not in m or "gate_rank" not in m:
            raise ValueError("decay_rank and gate_rank are missing: load the model's folder or set them")


MIXERS = {"latent_attention": LatentAttention, "mamba1": Mamba1, "attention": GroupedAttention, "mamba2": Mamba2,
          "channel_delta": ChannelDelta}


# -------------------------------------------------------------------- stacks ----
def _family(config):
    return registry.family(config)


def tensor_shapes(config: dict) -> dict:
    """{tensor name: shape}."""
    d, V, fam = config["width"], config["vocab"], _family(config)
    out = {"embed": (V, d), "head": (V, d)}
    out.update({n: (d,) for n in (("final.norm",) if fam.residual == SANDWICH_RMS else fam.norm_names("final.norm"))})
    if _loop(config)[2]:
        out["loop.in"] = (d, 2 * d)
    for i, layer in enumerate(config["layers"]):
        t = {n: (d,) for n in fam.norm_names("norm1")}
        t.update({"mix." + k: v for k, v in MIXERS[layer["type"]].shapes(layer["mixer"], d).items()})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            t.update({n: (d,) for n in fam.norm_names("norm2")})
            if fam.ff == SWIGLU:
                t["mlp.gate"] = (f, d)
            t["mlp.up"], t["mlp.down"] = (f, d), (d, f)
        out.update({f"l{i}.{k}": v for k, v in t.items()})
    return out


def _loop(config):
    """(start, stop, times); times 0 = no loop."""
    loop = config.get("loop")
    return (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)


def describe(config: dict):
    """The ctypes description of the stack (keep the returned object alive while it is used)."""
    fam = _family(config)
    layers = (MtjLayerDesc * len(config["layers"]))()
    for desc, layer in zip(layers, config["layers"]):
        mixer = MIXERS[layer["type"]]
        desc.mixer, desc.kv_from = mixer.code, -1
        desc.ff = layer["mlp"]["ff"] if layer["mlp"] is not None else 0
        desc.ff_kind = fam.ff
        mixer.describe(layer["mixer"], desc)
    start, stop, times = _loop(config)
    return MtjStackDesc(layers=layers, n_layers=len(layers), loop_start=start, loop_stop=stop, loop_times=times,
                        residual=fam.residual, norm_eps=config["norm"]["eps"], act_f32=1 if config["mtj_dtype"] == "float32" else 0,
                        tc_min_rows=config.get("mtj_tc_min_rows", 0), **fam.constants(config))


class LayerStack:
    """What the families share."""
    mixers: tuple = ()
    residual, ff = SANDWICH_RMS, SWIGLU

    @classmethod
    def prepare(cls, config: dict) -> dict:
        if "n_vocab" in config and "mtj_dtype" in config:
            return config                              # already prepared
        out = dict(config, n_vocab=config["vocab"], d_model=config["width"])
        for k, v in (("seq", 2048), ("cores_per_replica", 1), ("mtj_dtype", "bfloat16")):
            out.setdefault(k, v)
        return out

    @staticmethod
    def fit_tensors(config: dict, shapes: dict) -> dict:
        """The configuration with the sizes that only the tensors' shapes ({name: shape}) tell."""
        layers = []
        for i, layer in enumerate(config["layers"]):
            ranks = getattr(MIXERS.get(layer["type"]), "RANKS", {})
            found = {k: int(shapes[f"l{i}.mix.{t}"][0]) for k, t in ranks.items() if f"l{i}.mix.{t}" in shapes}
            layers.append(dict(layer, mixer=dict(layer["mixer"], **found)))
        return dict(config, layers=layers)

    @classmethod
    def validate(cls, config: dict) -> None:
        if config["cores_per_replica"] != 1:
            raise NotImplementedError("layer-stack models run on one GPU (cores_per_replica 1)")
        if config["mtj_dtype"] not in DTYPES:
            raise ValueError(f"mtj_dtype must be one of {DTYPES}")
        for i, layer in enumerate(config["layers"]):
            if layer["type"] not in cls.mixers:
                raise NotImplementedError(f"layer {i}: no mixer {layer['type']!r}")
            if layer["mlp"] is not None and layer["mlp"].get("kind", "dense") != "dense":
                raise NotImplementedError(f"layer {i}: no feed-forward {layer['mlp']['kind']!r}")
            try:
                MIXERS[layer["type"]].check(layer["mixer"])
            except (ValueError, NotImplementedError) as e:
                raise type(e)(f"layer {i}: {e}") from None
        start, stop, times = _loop(config)
        if times and not 0 <= start < stop <= len(config["layers"]):
            raise ValueError("loop must name a range of layers")

    @staticmethod
    def param_shapes(config: dict) -> dict:
        return {MODULE: tensor_shapes(config)}

    @staticmethod
    def create(config: dict, caps: dict, handle) -> int:
        cfg = MtjConfig(layers=len(config["layers"]), d_model=config["d_model"], n_heads=1, n_vocab=config["n_vocab"],
                        pe_rotary_dims=0, seq=config["seq"], cores_per_replica=1, **caps)
        desc = describe(config)
        return lib.mtj_create_stack(ctypes.byref(cfg), ctypes.byref(desc), handle)

    @staticmethod
    def state_from_tensors(config: dict, tensors: dict) -> dict:
        """The two-level parameter tree of ``network.state`` from tensors by name."""
        shapes = tensor_shapes(config)
        missing, extra = sorted(set(shapes) - set(tensors)), sorted(set(tensors) - set(shapes))
        if missing or extra:
            raise ValueError(f"tensors do not fit the configuration: missing {missing}, unknown {extra}")
        for n, s in shapes.items():
            if tuple(tensors[n].shape) != tuple(s):
                raise ValueError(f"tensor {n}: shape {tuple(tensors[n].shape)}, expected {tuple(s)}")
        return {MODULE: {n: torch.as_tensor(t)[None] for n, t in tensors.items()}}

    @staticmethod
    def init_state(config: dict, rank: int, device, seed: int) -> dict:
        """Random weights: norms at one, linear maps with unit gain, decays exp(-dt A) with A = 1 .. state (one per
        head: uniform in 1 .. 16) and step sizes softplus^-1 of values between 1e-3 and 0.1."""
        gen = torch.Generator(device=device)
        gen.manual_seed(seed)

        def normal(shape, std):
            return torch.randn(shape, generator=gen, device=device) * std

        out = {}
        for name, shape in tensor_shapes(config).items():
            leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
            if leaf.endswith("norm.b") or leaf in ("norm1.b", "norm2.b"):
                t = torch.zeros(shape, device=device)
            elif "norm" in leaf or leaf == "mix.D":
                t = torch.ones(shape, device=device)
            elif leaf == "mix.A_log" and len(shape) == 1:
                t = (1 + 15 * torch.rand(shape, generator=gen, device=device)).log()
            elif leaf == "mix.A_log":
                t = torch.arange(1, shape[1] + 1, device=device).float().log().expand(shape).contiguous()
            elif leaf in ("mix.dt.b", "mix.dt_bias"):
                dt = torch.exp(torch.rand(shape, generator=gen, device=device) * np.log(100.0) + np.log(1e-3))
                t = dt + torch.log(-torch.expm1(-dt))
            elif leaf == "mix.conv.b":
                t = torch.zeros(shape, device=device)
            elif leaf == "embed":
                t = normal(shape, 1.0)
            else:
                t = normal(shape, shape[-1] ** -0.5)
            out[name] = t.to(torch.bfloat16)[None]
        return {"params": {MODULE: out}, "step": np.array(0), "opt_state": None}


@registry.register("Keselix")
class Keselix(LayerStack):
    mixers = ("latent_attention", "mamba1")

    @staticmethod
    def norm_names(name):
        return (name, name + "b")                      # before and after the sublayer

    @staticmethod
    def constants(config):
        return {"residual_mult": config["residual_mult"]}


@registry.register("Bavutar")
class Bavutar(LayerStack):
    mixers = ("attention", "mamba2", "channel_delta")
    residual, ff = POST_LN, SQUARED_RELU

    @staticmethod
    def norm_names(name):
        return (name, name + ".b")                     # weight and bias

    @staticmethod
    def constants(config):
        return {"residual_mult": config["postln_alpha"], "embed_scale": config["embedding"]["scale"],
                "logit_softcap": config.get("logit_softcap") or 0.0}

    @classmethod
    def validate(cls, config):
        super().validate(config)
        if config.get("loop"):
            raise NotImplementedError("Bavutar models have no loop")
        for i, layer in enumerate(config["layers"]):
            j = layer["mixer"].get("kv_from")
            if j is None:
                continue
            src = config["layers"][j] if 0 <= j < i else {"type": None}
            if src["type"] != "attention" or src["mixer"].get("kv_from") is not None or \
                    any(src["mixer"][k] != layer["mixer"][k] for k in ("kv_heads", "dim", "vdim")):
                raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own and "
                                 "the same head sizes")
