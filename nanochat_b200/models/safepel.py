"""
Safepel: a decoder whose layers mix tokens with a gated delta rule or with window attention and fixed-decay linear
attention side by side, served by the framework's engine (it is not trained here). The module composes mechanisms of
`nanochat_b200.ops`; what belongs to the design is the order of things (N: layer norm with a weight, no bias):

  x = N(embed[token])                                    float32 residual stream
  per layer:  x += N(mixer(N(x)));  x += N(ff(N(x)))     the second line only where the layer has a feed-forward
  logits = head N(x) * logit_scale

  delta     short convolutions + silu on q, k, v; unit q and k; S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q;
            per-head RMS norm, silu gate
  parallel  left: window attention with soft-capped scores whose values are the unrotated keys
            right: S <- decay S + k v^T, o = S^T q on silu'd projections; RMS norm over all heads, sigmoid gate
            left_scale * left + right_scale * right, one output product for both

Everything that reads a mixer's input is one matrix (`w_in`) and one product; the delta rule's beta and decay inputs are the
rows behind it (`w_ba`), whose product keeps the accumulator's precision.
"""

import math
from dataclasses import dataclass, field
from typing import Optional

import torch
import torch.nn as nn

from nanochat_b200 import common, ops
from nanochat_b200.models import served
from nanochat_b200.models.sampling import NaiveSampler
from nanochat_b200.models.served import ServedModel, Weights, fit, fit_columns, fit_heads, padded, under


# ------------------------------------------------------------------------------ config

def _grouped(heads, kv_heads):
    if kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"{heads} heads do not share {kv_heads} key heads evenly")


@dataclass
class DeltaSpec:
    heads: int
    kv_heads: int                  # query / key heads, each shared by heads / kv_heads value heads
    dim: int
    vdim: int
    conv: int                      # taps of the short convolutions, the current token's included

    @classmethod
    def from_dict(cls, d):
        _grouped(d["heads"], d["kv_heads"])
        if d["conv"] < 1:
            raise ValueError(f"a convolution of {d['conv']} taps")
        return cls(**{k: d[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")})

    def to_dict(self):
        return dict(self.__dict__)


@dataclass
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int                       # of keys and, since the values are the keys, of values
    scale: float
    rot_base: float
    rot_dims: int                  # leading part of dim that turns
    softcap: Optional[float] = None
    window: Optional[int] = None   # keys a query sees, itself included

    @classmethod
    def from_dict(cls, d):
        rot, mask = d["rot"], d.get("mask") or {}
        _grouped(d["heads"], d["kv_heads"])
        if d.get("vdim", d["dim"]) != d["dim"]:
            raise ValueError(f"values of {d['vdim']} dimensions: they are the keys, which have {d['dim']}")
        out = cls(heads=d["heads"], kv_heads=d["kv_heads"], dim=d["dim"], scale=d["scale"], rot_base=rot["base"],
                  rot_dims=rot.get("dims", d["dim"]), softcap=d.get("softcap"), window=mask.get("size"))
        if out.rot_dims > out.dim or out.rot_dims % 2:
            raise ValueError(f"{out.rot_dims} rotated dimensions do not fit a head of {out.dim}")
        if out.window is not None and out.window < 1:
            raise ValueError(f"a window of {out.window} tokens")
        return out

    def to_dict(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "scale": self.scale,
               "rot": {"base": self.rot_base, "dims": self.rot_dims}}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass
class DecaySpec:
    heads: int
    dim: int
    vdim: int
    decay: list                    # one factor per head

    @classmethod
    def from_dict(cls, d):
        if len(d["decay"]) != d["heads"] or not all(0 <= x <= 1 for x in d["decay"]):
            raise ValueError(f"{d['heads']} heads need as many decays between 0 and 1, not {d['decay']}")
        return cls(d["heads"], d["dim"], d["vdim"], list(d["decay"]))

    def to_dict(self):
        return dict(self.__dict__)


@dataclass
class ParallelSpec:
    left: WindowSpec
    right: DecaySpec
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d):
        return cls(WindowSpec.from_dict(d["left"]), DecaySpec.from_dict(d["right"]), d["left_scale"], d["right_scale"])

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


@dataclass
class ReluGluSpec:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


MIXERS = {"delta": DeltaSpec, "parallel": ParallelSpec}
FEED_FORWARDS = {"dense": lambda d: ReluGluSpec(d["ff"])}


@dataclass
class LayerSpec:
    mixer: object
    mlp: Optional[ReluGluSpec] = None

    @classmethod
    def from_dict(cls, d):
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown layer type {d['type']!r}; known: {sorted(MIXERS)}")
        f = d.get("mlp")
        if f is not None and f["kind"] not in FEED_FORWARDS:
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}; known: {sorted(FEED_FORWARDS)}")
        return cls(MIXERS[d["type"]].from_dict(d["mixer"]), None if f is None else FEED_FORWARDS[f["kind"]](f))

    def to_dict(self):
        name = next(k for k, v in MIXERS.items() if isinstance(self.mixer, v))
        return {"type": name, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass
class SafepelConfig:
    vocab_size: int
    n_embd: int
    layers: list = field(default_factory=list)
    eps: float = 1e-5
    logit_scale: float = 1.0
    sequence_len: int = 32768              # tokens a request may hold (serving limit; the design has none)

    @classmethod
    def from_dict(cls, d, **serving):
        return cls(vocab_size=d["vocab"], n_embd=d["width"], layers=[LayerSpec.from_dict(x) for x in d["layers"]],
                   eps=d["norm"]["eps"], logit_scale=d.get("logit_scale", 1.0), **serving)

    def to_dict(self):
        return {"architecture": "Safepel", "vocab": self.vocab_size, "width": self.n_embd, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale, "layers": [x.to_dict() for x in self.layers]}

    @property
    def n_layer(self):
        return len(self.layers)


# ------------------------------------------------------------------------------ weights

class GatedDelta(Weights):
    """z = [q | k | v | gate logits], heads padded; channels of the convolutions are z's first columns. ba = [beta logits |
    decay inputs], each padded to hp."""

    entry = 0                                       # nothing in the paged store

    def __init__(self, spec, eps):
        super().__init__()
        s = self.spec = spec
        self.heads, self.kv_heads, self.taps, self.eps = s.heads, s.kv_heads, s.conv, eps
        self.dim, self.vdim, self.dp, self.vp, self.hp = s.dim, s.vdim, padded(s.dim), padded(s.vdim), padded(s.heads)
        self.channels = 2 * s.kv_heads * self.dp + s.heads * self.vp
        self.gate_off, self.y_width = self.channels, s.heads * self.vp
        self.sizes = [s.heads, s.kv_heads, s.dim, self.dp, s.vdim, self.vp, s.conv, self.hp]

    def states(self):
        """Per sequence: the state and the inputs of the last taps, token t in slot t % taps."""
        return {"S": (self.heads, self.dp, self.vp), "ring": (self.taps, self.channels)}

    def load(self, take, C, dtype, device):
        s, rows, conv = self.spec, [], []
        for name, heads, size in (("q", s.kv_heads, s.dim), ("k", s.kv_heads, s.dim), ("v", s.heads, s.vdim)):
            rows.append(fit_heads(take(name, heads * size, C), heads, size))
            w = take(name + ".conv", heads * size, s.conv).view(heads, size, s.conv)
            conv.append(fit(w, heads, padded(size), s.conv).reshape(-1, s.conv))
        rows.append(fit_heads(take("g", s.heads * s.vdim, C), s.heads, s.vdim))
        f32 = lambda name, w: self.put(name, w, torch.float32, device)
        f32("conv", torch.cat(conv).float().t())
        f32("norm", fit(take("norm", s.vdim).float(), self.vp))
        f32("neg_a", fit(-torch.exp(take("A_log", s.heads).double()), self.hp))
        f32("dt_bias", fit(take("dt_bias", s.heads).float(), self.hp))
        ba = [fit(take(n, s.heads, C), self.hp, padded(C)) for n in ("b", "a")]
        self.put("w_all", torch.cat(rows + ba), dtype, device)
        self.put("w_o", fit_columns(take("o", C, s.heads * s.vdim), s.heads, s.vdim), dtype, device)

    @property
    def w_in(self):
        return self.w_all[:self.channels + self.y_width]

    @property
    def w_ba(self):
        return self.w_all[self.channels + self.y_width:]

    def forward(self, h, cache, run, T):
        z, ba = ops.linear_rows(h, self.w_in), ops.linear_rows(h, self.w_ba, torch.float32)
        return ops.linear_rows(ops.gated_delta(self, z, ba, cache, run, T), self.w_o)

    # ------------------------------------------------------------------ cost accounting
    def flops_per_token(self, seen):
        return 6 * self.heads * self.spec.dim * self.spec.vdim

    def state_bytes(self):
        return 4 * sum(math.prod(s) for s in self.states().values())


class WindowAttention(Weights):
    """Segments of the layer's z: queries at q_off, keys at k_off. A store entry is [rotated keys | keys]."""

    def __init__(self, spec, out_scale, off):
        super().__init__()
        s = self.spec = spec
        self.heads, self.kv_heads, self.dp, self.window = s.heads, s.kv_heads, padded(s.dim), s.window
        self.q_off, self.k_off = off, off + s.heads * self.dp
        self.end = self.k_off + s.kv_heads * self.dp
        self.entry, self.y_width = 2 * s.kv_heads * self.dp, s.heads * self.dp
        self.scale, self.softcap, self.out_scale = s.scale, s.softcap or 0.0, out_scale
        self.sizes = [s.heads, s.kv_heads, self.dp, self.q_off, self.k_off, s.window or 0]
        self.reals = [self.scale, self.softcap, out_scale]

    def load(self, take, C, dtype, device):
        s = self.spec
        i = torch.arange(s.rot_dims // 2, dtype=torch.float64)
        f = s.rot_base ** (-2.0 * i / max(s.rot_dims, 1))
        self.register_buffer("freq", torch.stack([f.float(), (f - f.float().double()).float()]).to(device), persistent=False)
        return ([fit_heads(take("q", s.heads * s.dim, C), s.heads, s.dim), fit_heads(take("k", s.kv_heads * s.dim, C), s.kv_heads, s.dim)],
                fit_columns(take("o", C, s.heads * s.dim), s.heads, s.dim))


class DecayAttention(Weights):
    """Segments of the layer's z: q, k, v, gate logits from `off` on."""

    def __init__(self, spec, eps, out_scale, off):
        super().__init__()
        s = self.spec = spec
        self.heads, self.dim, self.vdim, self.dp, self.vp = s.heads, s.dim, s.vdim, padded(s.dim), padded(s.vdim)
        self.q_off, self.k_off, self.v_off = off, off + s.heads * self.dp, off + 2 * s.heads * self.dp
        self.gate_off = self.v_off + s.heads * self.vp
        self.end = self.gate_off + s.heads * self.vp
        self.y_width, self.eps, self.out_scale = s.heads * self.vp, eps, out_scale
        self.sizes = [s.heads, self.dp, s.vdim, self.vp, self.q_off, self.k_off, self.v_off, self.gate_off]
        self.reals = [eps, out_scale]

    def states(self):
        return {"S": (self.heads, self.dp, self.vp)}

    def load(self, take, C, dtype, device):
        s = self.spec
        log_decay = [math.log(x) if x > 0 else -math.inf for x in s.decay]
        # one token at exp(-1e4) = 0 already; multiples of it stay finite
        self.put("log_decay", torch.tensor(log_decay, dtype=torch.float64).clamp_min(-1e4), torch.float32, device)
        self.put("norm", fit(take("norm", s.heads * s.vdim).float().view(s.heads, s.vdim), s.heads, self.vp).reshape(-1), torch.float32, device)
        rows = [fit_heads(take(n, s.heads * size, C), s.heads, size) for n, size in (("q", s.dim), ("k", s.dim), ("v", s.vdim), ("g", s.vdim))]
        return rows, fit_columns(take("o", C, s.heads * s.vdim), s.heads, s.vdim)


class Parallel(Weights):
    """Both read one z and write one y, whose output product adds them."""

    def __init__(self, spec, eps):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.left = WindowAttention(spec.left, spec.left_scale, 0)
        self.right = DecayAttention(spec.right, eps, spec.right_scale, self.left.end)
        self.entry, self.y_width = self.left.entry, self.left.y_width + self.right.y_width

    def states(self):
        return self.right.states()

    def load(self, take, C, dtype, device):
        left, w_left = self.left.load(under(take, "left."), C, dtype, device)
        right, w_right = self.right.load(under(take, "right."), C, dtype, device)
        self.put("w_all", torch.cat(left + right), dtype, device)
        self.put("w_o", torch.cat([w_left, w_right], 1), dtype, device)

    def forward(self, h, cache, run, T):
        z = ops.linear_rows(h, self.w_all)
        return ops.linear_rows(ops.window_and_decay(self.left, self.right, z, cache, run, T), self.w_o)

    # ------------------------------------------------------------------ cost accounting
    def flops_per_token(self, seen):
        a, b = self.spec.left, self.spec.right
        return 4 * a.heads * a.dim * seen + 4 * b.heads * b.dim * b.vdim

    def state_bytes(self):
        return 4 * sum(math.prod(s) for s in self.states().values())


class ReluGlu(Weights):
    """W_down (relu(W_gate h) * (W_up h)); w_gate_up holds the gate rows, then the up rows."""

    def __init__(self, spec):
        super().__init__()
        self.spec, self.ff, self.fp = spec, spec.ff, padded(spec.ff)

    def load(self, take, C, dtype, device):
        gate, up, down = take("gate", self.ff, C), take("up", self.ff, C), take("down", C, self.ff)
        self.put("w_gate_up", torch.cat([fit(gate, self.fp, padded(C)), fit(up, self.fp, padded(C))]), dtype, device)
        self.put("w_down", fit(down, padded(C), self.fp), dtype, device)

    def forward(self, h):
        return ops.linear_rows(ops.relu_glu(h, self.w_gate_up), self.w_down)


class Layer(Weights):
    def __init__(self, spec, eps):
        super().__init__()
        self.spec = spec
        self.mix = (GatedDelta if isinstance(spec.mixer, DeltaSpec) else Parallel)(spec.mixer, eps)
        self.mlp = None if spec.mlp is None else ReluGlu(spec.mlp)

    def load(self, take, C, dtype, device):
        for name in ("norm1", "norm1b") + (() if self.mlp is None else ("norm2", "norm2b")):
            self.put(name, fit(take(name, C).float(), padded(C)), torch.float32, device)
        self.mix.load(under(take, "mix."), C, dtype, device)
        if self.mlp is not None:
            self.mlp.load(under(take, "mlp."), C, dtype, device)


class Safepel(ServedModel, NaiveSampler):
    step_graph = "RecurrentDecodeGraph"

    def __init__(self, config, dtype=None):
        super().__init__()
        self.config = config
        self.dtype = dtype or common.COMPUTE_DTYPE
        self.width = padded(config.n_embd)
        self.layers = nn.ModuleList([Layer(x, config.eps) for x in config.layers])
        self.embed = self.embed_norm = self.final_norm = self.head = None

    # ------------------------------------------------------------------------- weights
    def pack(self, take, device):
        C, V = self.config.n_embd, self.config.vocab_size
        for i, layer in enumerate(self.layers):
            layer.load(under(take, f"l{i}."), C, self.dtype, device)
        put = lambda w, dtype: nn.Parameter(w.to(dtype).to(device), requires_grad=False)
        self.embed = put(fit(take("embed", V, C), padded(V), self.width), self.dtype)
        self.head = put(fit(take("head", V, C), padded(V), self.width), self.dtype)
        self.embed_norm = put(fit(take("embed.norm", C).float(), self.width), torch.float32)
        # the logits' factor rides on the norm in front of the head
        self.final_norm = put(fit(take("final.norm", C).double() * self.config.logit_scale, self.width), torch.float32)

    def tensor_shapes(self):
        """Names and shapes of the stored tensors."""
        C, V = self.config.n_embd, self.config.vocab_size
        out = {"embed": (V, C), "embed.norm": (C,), "final.norm": (C,), "head": (V, C)}
        for i, layer in enumerate(self.layers):
            s, l, m = layer.spec.mixer, f"l{i}.", f"l{i}.mix."
            out.update({l + "norm1": (C,), l + "norm1b": (C,)})
            if isinstance(s, DeltaSpec):
                for name, n in (("q", s.kv_heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.heads * s.vdim)):
                    out.update({m + name: (n, C), m + name + ".conv": (n, s.conv)})
                out.update({m + "b": (s.heads, C), m + "a": (s.heads, C), m + "A_log": (s.heads,), m + "dt_bias": (s.heads,),
                            m + "norm": (s.vdim,), m + "g": (s.heads * s.vdim, C), m + "o": (C, s.heads * s.vdim)})
            else:
                a, b = s.left, s.right
                out.update({m + "left.q": (a.heads * a.dim, C), m + "left.k": (a.kv_heads * a.dim, C), m + "left.o": (C, a.heads * a.dim),
                            m + "right.q": (b.heads * b.dim, C), m + "right.k": (b.heads * b.dim, C), m + "right.v": (b.heads * b.vdim, C),
                            m + "right.g": (b.heads * b.vdim, C), m + "right.o": (C, b.heads * b.vdim), m + "right.norm": (b.heads * b.vdim,)})
            if layer.mlp is not None:
                ff = layer.mlp.ff
                out.update({l + "norm2": (C,), l + "norm2b": (C,), l + "mlp.gate": (ff, C), l + "mlp.up": (ff, C), l + "mlp.down": (C, ff)})
        return out

    def init_tensor(self, name, shape, normal):
        if "norm" in name:
            return torch.ones(shape)
        if name.endswith("dt_bias"):
            return torch.full(shape, -3.0)
        return super().init_tensor(name, shape, normal)

    # --------------------------------------------------------------------------- cache
    def make_cache(self, rows, sequence_len=None):
        """An empty cache: a paged store for the layers with attention, states for those with a recurrence."""
        from nanochat_b200.engine import RecurrentCache
        return RecurrentCache(rows, [layer.mix.entry for layer in self.layers], [layer.mix.states() for layer in self.layers],
                              sequence_len or self.config.sequence_len, self.get_device(), self.dtype)

    # ------------------------------------------------------------------------- forward
    def sublayers(self):
        """(sublayer, post-norm, the next sublayer's norm, layer index or None for a feed-forward), in order."""
        flat = []
        for i, layer in enumerate(self.layers):
            flat.append((layer.mix, layer.norm1, layer.norm1b, i))
            if layer.mlp is not None:
                flat.append((layer.mlp, layer.norm2, layer.norm2b, None))
        following = [norm for _, norm, _, _ in flat[1:]] + [self.final_norm]
        return [(sub, post, after, i) for (sub, _, post, i), after in zip(flat, following)]

    @property
    def first_norm(self):
        return self.layers[0].norm1 if len(self.layers) else self.final_norm

    @torch.inference_mode()
    def forward(self, idx, targets=None, kv_cache=None, want=None, residuals=None):
        """Logits (B, T, vocab), or (len(want), vocab) for the `want`ed rows of the flattened (B * T), None for none. The
        tokens continue what `kv_cache` holds. `residuals`, a list, collects the stream after every layer."""
        if targets is not None:
            raise NotImplementedError("Safepel is served, not trained: no loss")
        B, T = idx.shape
        if kv_cache is None:
            kv_cache = self.make_cache(B, T)
            kv_cache.reserve(0, T)
            kv_cache.begin_rows()
        cfg, eps, C = self.config, self.config.eps, self.config.n_embd
        x, h = ops.embed_layer_norm(idx.reshape(-1), self.embed, cfg.vocab_size, self.embed_norm, self.first_norm, eps, C)
        for sub, post, after, i in self.sublayers():
            if residuals is not None and i is not None and i > 0:
                residuals.append(x[:, :C].clone())
            y = sub(h) if i is None else sub(h, kv_cache, i, T)
            h = ops.layer_norm_residual(x, y, post, after, eps, C, self.dtype)
        if residuals is not None and len(self.layers):
            residuals.append(x[:, :C].clone())
        kv_cache.advance(T)
        if want is not None:
            if len(want) == 0:
                return None
            h = h[torch.as_tensor(want, dtype=torch.long, device=h.device)]
        logits = ops.linear_rows(h, self.head, torch.float32)[:, :cfg.vocab_size]
        return logits if want is not None else logits.reshape(B, T, -1)

    # ----------------------------------------------------------------- cost accounting
    def matmul_params_per_token(self):
        total = self.config.vocab_size * self.config.n_embd
        for layer in self.layers:
            total += layer.mix.w_all.numel() + layer.mix.w_o.numel()
            if layer.mlp is not None:
                total += layer.mlp.w_gate_up.numel() + layer.mlp.w_down.numel()
        return total

    def _seen(self, layer, context_len):
        w = layer.mix.left.window if isinstance(layer.mix, Parallel) else None
        return context_len if w is None else min(context_len, w)

    def estimate_decode_flops(self, context_len):
        return 2 * self.matmul_params_per_token() + sum(l.mix.flops_per_token(self._seen(l, context_len)) for l in self.layers)

    def estimate_prefill_flops(self, num_tokens):
        total = 2 * self.matmul_params_per_token() * num_tokens
        for layer in self.layers:
            w = self._seen(layer, num_tokens)
            mean = (w * (w + 1) / 2 + (num_tokens - w) * w) / num_tokens
            total += layer.mix.flops_per_token(mean) * num_tokens
        return total

    def kv_bytes_per_token(self):
        return sum(layer.mix.entry for layer in self.layers) * self.dtype.itemsize

    def kv_read_bytes(self, context_len):
        """Bytes of store and state a decode step reads per row."""
        return sum(self._seen(l, context_len) * l.mix.entry * self.dtype.itemsize + l.mix.state_bytes() for l in self.layers)

    def decode_weight_bytes(self):
        """Bytes of weights one decode row reads."""
        return self.matmul_params_per_token() * self.dtype.itemsize


def load_folder(path, device, dtype=None, **serving):
    return served.load_folder(path, device, SafepelConfig.from_dict, Safepel, dtype, **serving)
