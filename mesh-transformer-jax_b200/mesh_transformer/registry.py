"""Model families by the configuration's ``architecture`` key.

A family is a class with static methods
    prepare(config)       the configuration with the keys every runtime call reads filled in
                          (``n_vocab``, ``d_model``, ``seq``, ``cores_per_replica``)
    validate(config)      raises for configurations it cannot run
    param_shapes(config)  {module: {leaf: per-shard shape}}
    create(config, caps, handle)   makes the library handle, returns its status
    init_state(config, rank, device, seed)   random ``state``
and, to load model folders,
    fit_tensors(config, shapes)   the configuration with the sizes that only the tensors' shapes tell
    state_from_tensors(config, tensors)   the parameter tree of ``state``
A configuration without the key is the reference's GPT-J (its config JSON has no such key).
"""
from __future__ import annotations

import importlib
import json
import os

_FAMILIES: dict = {}
_MODULES = {"gptj": "_runtime", "Keselix": "layer_stack", "Bavutar": "layer_stack"}     # where each family registers itself


def register(*names):
    def wrap(cls):
        for n in names:
            _FAMILIES[n] = cls
        return cls
    return wrap


def names():
    return sorted(_MODULES)


def family(config: dict):
    name = config.get("architecture", "gptj")
    if name not in _FAMILIES:
        if name not in _MODULES:
            raise NotImplementedError(f"no model family {name!r}; known: {', '.join(names())}")
        importlib.import_module("." + _MODULES[name], __package__)
    return _FAMILIES[name]


def prepare(config: dict) -> dict:
    return family(config).prepare(config)


def read_config(folder: str, **overrides) -> dict:
    """``config.json`` of a model folder, with overrides for the runtime keys."""
    with open(os.path.join(folder, "config.json")) as f:
        return prepare(dict(json.load(f), **overrides))


def load_network(folder: str, device=None, **overrides):
    """A ``CausalTransformer`` with the configuration and weights of a model folder (config.json and
    model.safetensors)."""
    import numpy as np
    from .checkpoint import read_safetensors
    from .transformer_shard import CausalTransformer
    config = read_config(folder, **overrides)
    fam = family(config)
    if not hasattr(fam, "state_from_tensors"):
        raise NotImplementedError("this family does not load model folders; use load_ckpt or hf_interchange")
    tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
    config = fam.fit_tensors(config, {n: tuple(t.shape) for n, t in tensors.items()})
    net = CausalTransformer(config, device=device, init_weights=False)
    net.state = {"params": fam.state_from_tensors(config, tensors), "step": np.array(0), "opt_state": None}
    return net
