"""
Architectures by name. A model folder (config.json + model.safetensors) names its architecture in config.json; the
.pt checkpoints of training runs hold GPT models.
"""

import json
import os


class Architecture:
    def __init__(self, name, config_from_dict, build, load_folder):
        self.name, self.config_from_dict, self.build, self.load_folder = name, config_from_dict, build, load_folder


def _gpt():
    from dataclasses import fields
    import torch
    from nanochat_b200 import common
    from nanochat_b200.models.gpt import GPT, GPTConfig
    from nanochat_b200.utils.safetensors import read_safetensors

    def config_from_dict(d, **serving):
        names = {f.name for f in fields(GPTConfig)}
        return GPTConfig(**{k: v for k, v in {**d, **serving}.items() if k in names})

    def build(config, device, dtype=None):
        if dtype is not None and dtype != common.COMPUTE_DTYPE:
            raise ValueError(f"GPT computes in {common.COMPUTE_DTYPE} in this process (NANOCHAT_DTYPE), not {dtype}")
        with torch.device("meta"):
            model = GPT(config)
        model.to_empty(device=device)
        model.init_weights()
        return model.eval()

    def load_folder(path, device, dtype=None, **serving):
        with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as f:
            model = build(config_from_dict(json.load(f), **serving), device, dtype)
        tensors = {k: v.to(device) for k, v in read_safetensors(os.path.join(path, "model.safetensors")).items()}
        wte = next(v for k, v in model.state_dict().items() if k.endswith("wte.weight")).dtype
        for k in tensors:
            if k.endswith("wte.weight") or k.startswith("value_embeds."):
                tensors[k] = tensors[k].to(wte)
            else:
                tensors[k] = tensors[k].float()
        model.load_state_dict(tensors, strict=True, assign=True)
        return model.eval()

    return Architecture("GPT", config_from_dict, build, load_folder)


def _served(name):
    """A model that is served only: module models/<name>, class <Name>, configuration <Name>Config."""
    import importlib
    m = importlib.import_module(f"nanochat_b200.models.{name.lower()}")
    model = getattr(m, name)

    def build(config, device, dtype=None):
        return model(config, dtype).init_weights(device)

    return Architecture(name, getattr(m, name + "Config").from_dict, build, m.load_folder)


_ARCHITECTURES = {"GPT": _gpt, "Lupodra": lambda: _served("Lupodra"), "Safepel": lambda: _served("Safepel")}


def architectures():
    return sorted(_ARCHITECTURES)


def get_architecture(name):
    if name not in _ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {architectures()}")
    return _ARCHITECTURES[name]()


def load_model_folder(path, device, dtype=None, **serving):
    """The model of a folder with config.json and model.safetensors, in `dtype` (default: the compute type).
    `serving` overrides configuration fields that are limits of the server, such as sequence_len."""
    config = os.path.join(path, "config.json")
    if not os.path.exists(config):
        raise FileNotFoundError(f"no config.json in {path}")
    with open(config, "r", encoding="utf-8") as f:
        name = json.load(f).get("architecture", "GPT")
    return get_architecture(name).load_folder(path, device, dtype, **serving).eval()
