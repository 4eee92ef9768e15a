"""Layer-stack models (Keselix): configuration, tensor names and random initialisation.

Configuration keys (config.json):
    architecture, vocab, width, norm {eps}, residual_mult
    layers: list of {type, mixer, mlp}
        type "latent_attention", mixer {heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {base, dims}}
        type "mamba1",           mixer {inner, state, conv, dt_rank}
        mlp {kind "dense", ff} or null
    loop: {start, stop, times} or absent
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
MIXERS = {"latent_attention": 0, "mamba1": 1}        # MTJ_MIXER_*
DTYPES = ("bfloat16", "float32")


def tensor_shapes(config: dict) -> dict:
    """{tensor name: shape}."""
    d, V = config["width"], config["vocab"]
    out = {"embed": (V, d), "final.norm": (d,), "head": (V, d)}
    if _loop(config)[2]:
        out["loop.in"] = (d, 2 * d)
    for i, layer in enumerate(config["layers"]):
        m, t = layer["mixer"], {}
        t["norm1"] = t["norm1b"] = (d,)
        if layer["type"] == "latent_attention":
            H, r = m["heads"], m["rot_dim"]
            t["mix.q"] = (H * (m["dim"] + r), d)
            t["mix.dkv"] = (m["kv_rank"] + r, d)
            t["mix.dkv.norm"] = (m["kv_rank"],)
            t["mix.uk"] = (H * m["dim"], m["kv_rank"])
            t["mix.uv"] = (H * m["vdim"], m["kv_rank"])
            t["mix.o"] = (d, H * m["vdim"])
        else:
            n = m["inner"]
            t["mix.in"] = (2 * n, d)
            t["mix.conv"] = (n, m["conv"])
            t["mix.conv.b"] = t["mix.dt.b"] = t["mix.D"] = (n,)
            t["mix.x"] = (m["dt_rank"] + 2 * m["state"], n)
            t["mix.dt"] = (n, m["dt_rank"])
            t["mix.A_log"] = (n, m["state"])
            t["mix.o"] = (d, n)
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            t["norm2"] = t["norm2b"] = (d,)
            t["mlp.gate"] = t["mlp.up"] = (f, d)
            t["mlp.down"] = (d, f)
        out.update({f"l{i}.{k}": v for k, v in t.items()})
    return out


def _loop(config):
    """(start, stop, times); times 0 = no loop."""
    loop = config.get("loop")
    return (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)


def describe(config: dict):
    """The ctypes description of the stack (keep the returned object alive while it is used)."""
    layers = (MtjLayerDesc * len(config["layers"]))()
    for desc, layer in zip(layers, config["layers"]):
        m = layer["mixer"]
        desc.mixer = MIXERS[layer["type"]]
        desc.ff = layer["mlp"]["ff"] if layer["mlp"] is not None else 0
        if layer["type"] == "latent_attention":
            for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"):
                setattr(desc, k, m[k])
            desc.window, desc.rot_base = m["mask"]["size"], m["rot"]["base"]
        else:
            for k in ("inner", "state", "conv", "dt_rank"):
                setattr(desc, k, m[k])
    start, stop, times = _loop(config)
    return MtjStackDesc(layers=layers, n_layers=len(layers), loop_start=start, loop_stop=stop, loop_times=times,
                        residual_mult=config["residual_mult"], norm_eps=config["norm"]["eps"],
                        act_f32=1 if config["mtj_dtype"] == "float32" else 0,
                        tc_min_rows=config.get("mtj_tc_min_rows", 0))


@registry.register("Keselix")
class LayerStack:
    @staticmethod
    def prepare(config: dict) -> dict:
        if "n_vocab" in config and "mtj_dtype" in config:
            return config                              # already prepared
        out = dict(config, n_vocab=config["vocab"], d_model=config["width"])
        for k, v in (("seq", 2048), ("cores_per_replica", 1), ("mtj_dtype", "bfloat16")):
            out.setdefault(k, v)
        return out

    @staticmethod
    def validate(config: dict) -> None:
        if config["cores_per_replica"] != 1:
            raise NotImplementedError("layer-stack models run on one GPU (cores_per_replica 1)")
        if config["mtj_dtype"] not in DTYPES:
            raise ValueError(f"mtj_dtype must be one of {DTYPES}")
        for i, layer in enumerate(config["layers"]):
            if layer["type"] not in MIXERS:
                raise NotImplementedError(f"layer {i}: no mixer {layer['type']!r}")
            if layer["mlp"] is not None and layer["mlp"].get("kind", "dense") != "dense":
                raise NotImplementedError(f"layer {i}: no feed-forward {layer['mlp']['kind']!r}")
            if layer["type"] == "latent_attention" and layer["mixer"]["rot"].get("dims", layer["mixer"]["rot_dim"]) \
                    != layer["mixer"]["rot_dim"]:
                raise NotImplementedError(f"layer {i}: the rotated part is rotated as a whole")
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
        """Random weights: norms at one, linear maps with unit gain, decays exp(-dt A) with A = 1 .. state and step
        sizes softplus^-1 of values between 1e-3 and 0.1."""
        gen = torch.Generator(device=device)
        gen.manual_seed(seed)

        def normal(shape, std):
            return torch.randn(shape, generator=gen, device=device) * std

        out = {}
        for name, shape in tensor_shapes(config).items():
            leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
            if "norm" in leaf or leaf == "mix.D":
                t = torch.ones(shape, device=device)
            elif leaf == "mix.A_log":
                t = torch.arange(1, shape[1] + 1, device=device).float().log().expand(shape).contiguous()
            elif leaf == "mix.dt.b":
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
