"""
What models that are served only share: weights packed into the layouts of the serving kernels (row sizes padded to
multiples of 8 with zeros), loading by tensor name with every shape checked, random initialisation, model folders.

A model defines `tensor_shapes()` (names and shapes of the stored tensors), `pack(take, device)` (fetch every tensor
through `take(name, *shape)`) and, where the default does not fit, `init_tensor(name, shape, normal)`.
"""

import json
import os

import torch
import torch.nn as nn


def padded(n, m=8):
    """n rounded up to a multiple of m."""
    return -(-n // m) * m


def fit(w, *shape):
    """w at the origin of a zero tensor of `shape`."""
    if tuple(w.shape) == shape:
        return w
    out = w.new_zeros(shape)
    out[tuple(slice(0, s) for s in w.shape)] = w
    return out


def fit_heads(w, heads, size):
    """Rows of a per-head projection (heads * size, n) with every head's rows and the columns padded."""
    n = w.shape[1]
    return fit(w.view(heads, size, n), heads, padded(size), padded(n)).reshape(-1, padded(n))


def fit_columns(w, heads, size):
    """An output projection (n, heads * size) that reads per-head padded rows, its own rows padded too."""
    n = w.shape[0]
    return fit(w.view(n, heads, size), padded(n), heads, padded(size)).reshape(padded(n), -1)


class Weights(nn.Module):
    """Frozen tensors by attribute name."""

    def put(self, name, value, dtype, device):
        self.register_parameter(name, nn.Parameter(value.to(dtype).to(device).contiguous(), requires_grad=False))


def under(take, prefix):
    return lambda name, *shape: take(prefix + name, *shape)


class ServedModel(nn.Module):
    @torch.no_grad()
    def load_tensors(self, tensors, device):
        """Take the named tensors (any float type) into the layouts of the kernels. A missing tensor, a wrong shape and a
        tensor without a place are errors."""
        left = set(tensors)

        def take(name, *shape):
            if name not in tensors:
                raise KeyError(f"tensor {name!r} is missing")
            t = tensors[name]
            if tuple(t.shape) != shape:
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration says {shape}")
            left.discard(name)
            return t

        self.pack(take, device)
        if left:
            raise ValueError(f"tensors the configuration has no place for: {sorted(left)[:8]}")
        return self

    def init_tensor(self, name, shape, normal):
        """A random tensor of a plausible scale; `normal(shape)` draws standard normals."""
        return normal(shape) * (1.0 if name == "embed" else shape[1] ** -0.5) if len(shape) == 2 else torch.zeros(shape)

    def init_weights(self, device, seed=0):
        """Random weights of a plausible scale (benchmarks, demonstrations)."""
        g = torch.Generator(device=device).manual_seed(seed)
        normal = lambda shape: torch.randn(shape, generator=g, device=device)
        return self.load_tensors({n: self.init_tensor(n, s, normal).to(torch.bfloat16) for n, s in self.tensor_shapes().items()}, device)

    def get_device(self):
        return self.embed.device


def load_folder(path, device, config_from_dict, build, dtype=None, **serving):
    """A model from a folder of config.json and model.safetensors."""
    from nanochat_b200.utils.safetensors import read_safetensors
    with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as f:
        config = config_from_dict(json.load(f), **serving)
    return build(config, dtype).load_tensors(read_safetensors(os.path.join(path, "model.safetensors")), device)
