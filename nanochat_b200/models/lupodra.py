"""
Lupodra: a decoder of latent-attention layers with dense or mixture-of-experts feed-forwards, served by the framework's
engine (it is not trained here). The module composes mechanisms of `nanochat_b200.ops`; what belongs to the design is
the order of things:

  x = embed[token] (float32 residual stream; kept as x0)
  for every layer run (the layers start .. stop-1 of a loop run `times` times with the same weights, each run with its
  own cache entries; a repeated pass begins with x += x0):
      h = norm(x)                                       RMS norm, weight stored as deviation from one
      x += m * (sigmoid(G1 h + b1) * attention(h) + sigmoid(G2 h + b2) * ff(h))      both sublayers read h
  logits = norm(x) embed^T

Everything that reads h (query and key-value down-projections, both gates, a dense feed-forward's up-projection) is one
matrix (`w_in`) and one product. Router logits and logits keep the accumulator's precision.
"""

from dataclasses import dataclass, field
from typing import Optional

import torch
import torch.nn as nn

from nanochat_b200 import common, ops
from nanochat_b200.models import served
from nanochat_b200.models.sampling import NaiveSampler
from nanochat_b200.models.served import ServedModel, Weights, fit, padded, under


# ------------------------------------------------------------------------------ config

@dataclass
class LatentAttentionSpec:
    heads: int
    dim: int                       # unrotated query / key dimensions per head
    rot_dim: int                   # rotated ones; the key's are shared by all heads
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_base: float
    rot_dims: int                  # leading part of rot_dim that turns
    window: Optional[int] = None   # keys a query sees, itself included

    @classmethod
    def from_dict(cls, d):
        rot, mask = d["rot"], d.get("mask") or {}
        return cls(heads=d["heads"], dim=d["dim"], rot_dim=d["rot_dim"], vdim=d["vdim"], kv_rank=d["kv_rank"], q_rank=d["q_rank"],
                   scale=d["scale"], rot_base=rot["base"], rot_dims=rot.get("dims", d["rot_dim"]), window=mask.get("size"))

    def to_dict(self):
        out = {k: getattr(self, k) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")}
        out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass
class DenseSpec:
    ff: int

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass
class MixtureSpec:
    ff: int
    experts: int
    top: int

    def to_dict(self):
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


MIXERS = {"latent_attention": LatentAttentionSpec.from_dict}
FEED_FORWARDS = {"dense": lambda d: DenseSpec(d["ff"]),
                 "moe": lambda d: MixtureSpec(d["expert"]["ff"], d["router"]["experts"], d["router"]["top"])}


@dataclass
class LayerSpec:
    mixer: LatentAttentionSpec
    mlp: object = None             # DenseSpec, MixtureSpec or None

    @classmethod
    def from_dict(cls, d):
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown layer type {d['type']!r}; known: {sorted(MIXERS)}")
        f = d.get("mlp")
        if f is not None and f["kind"] not in FEED_FORWARDS:
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}; known: {sorted(FEED_FORWARDS)}")
        return cls(MIXERS[d["type"]](d["mixer"]), None if f is None else FEED_FORWARDS[f["kind"]](f))

    def to_dict(self):
        return {"type": "latent_attention", "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass
class LupodraConfig:
    vocab_size: int
    n_embd: int
    layers: list = field(default_factory=list)
    loop: Optional[tuple] = None           # (start, stop, times)
    eps: float = 1e-6
    residual_mult: float = 1.0
    sequence_len: int = 32768              # tokens a request may hold (serving limit; the design has none)

    @classmethod
    def from_dict(cls, d, **serving):
        loop = d.get("loop")
        if loop is not None:
            loop = (loop["start"], loop["stop"], loop["times"])
            if not 0 <= loop[0] < loop[1] <= len(d["layers"]) or loop[2] < 1:
                raise ValueError(f"loop {loop} does not fit {len(d['layers'])} layers")
        return cls(vocab_size=d["vocab"], n_embd=d["width"], layers=[LayerSpec.from_dict(x) for x in d["layers"]], loop=loop,
                   eps=d["norm"]["eps"], residual_mult=d.get("residual_mult", 1.0), **serving)

    def to_dict(self):
        return {"architecture": "Lupodra", "vocab": self.vocab_size, "width": self.n_embd, "norm": {"eps": self.eps},
                "residual_mult": self.residual_mult, "layers": [x.to_dict() for x in self.layers],
                "loop": None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop))}

    def runs(self):
        """(layer index, whether the run opens a repeated pass), in order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        body = [(i, k > 0 and i == start) for k in range(times) for i in range(start, stop)]
        return [(i, False) for i in range(start)] + body + [(i, False) for i in range(stop, n)]

    @property
    def n_layer(self):
        return len(self.runs())


# ------------------------------------------------------------------------------ weights

class LatentAttention(Weights):
    """Padded sizes: dp / vp head dimensions, qp query latent, kvp + rp one store entry."""

    def __init__(self, spec, eps):
        super().__init__()
        s = self.spec = spec
        self.heads, self.rot_dim, self.kv_rank, self.q_rank = s.heads, s.rot_dim, s.kv_rank, s.q_rank
        self.window, self.scale, self.eps = s.window, s.scale, eps
        if s.rot_dims > s.rot_dim or s.rot_dims % 2:
            raise ValueError(f"{s.rot_dims} rotated dimensions do not fit a rotated part of {s.rot_dim}")
        self.dp, self.vp, self.qp = padded(s.dim), padded(s.vdim), padded(s.q_rank)
        self.kvp, self.rp = padded(s.kv_rank, 16), padded(s.rot_dim, 16)
        self.c_off, self.rot_off = self.qp, self.qp + self.kvp          # segments of w_in's output

    @property
    def entry(self):
        return self.kvp + self.rp

    def load(self, take, C, dtype, device):
        """Own matrices; returns the rows of w_in that the mixer reads."""
        s, H = self.spec, self.heads
        put = lambda name, w, dt=dtype: self.put(name, w, dt, device)
        dq, dkv = take("dq", s.q_rank, C), take("dkv", s.kv_rank + s.rot_dim, C)
        put("q_norm", fit(take("dq.norm", s.q_rank).float(), self.qp), torch.float32)
        put("kv_norm", fit(take("dkv.norm", s.kv_rank).float(), self.kvp), torch.float32)
        uq = take("uq", H * (s.dim + s.rot_dim), s.q_rank).view(H, s.dim + s.rot_dim, s.q_rank)
        w_q = torch.cat([fit(uq[:, :s.dim], H, self.dp, self.qp), fit(uq[:, s.dim:], H, self.rp, self.qp)], 1)
        put("w_q", w_q.reshape(-1, self.qp))
        uk = fit(take("uk", H * s.dim, s.kv_rank).view(H, s.dim, s.kv_rank), H, self.dp, self.kvp).reshape(-1, self.kvp)
        uv = fit(take("uv", H * s.vdim, s.kv_rank).view(H, s.vdim, s.kv_rank), H, self.vp, self.kvp).reshape(-1, self.kvp)
        put("w_kv", torch.cat([uk, uv]))
        o = take("o", C, H * s.vdim).view(C, H, s.vdim)
        put("w_o", fit(o, padded(C), H, self.vp).reshape(padded(C), -1))
        i = torch.arange(s.rot_dims // 2, dtype=torch.float64)
        self.register_buffer("freq", (s.rot_base ** (-2.0 * i / s.rot_dims)).float().to(device), persistent=False)
        return [fit(dq, self.qp, C), fit(dkv[:s.kv_rank], self.kvp, C), fit(dkv[s.kv_rank:], self.rp, C)]

    @property
    def w_uk(self):
        return self.w_kv[:self.heads * self.dp]

    @property
    def w_uv(self):
        return self.w_kv[self.heads * self.dp:]

    def forward(self, z, cache, run, T):
        return ops.latent_attention(self, z, cache, run, T)


class DenseFF(Weights):
    """W_down act(z), z = W_up h being a segment of the layer's fused input product."""

    def __init__(self, spec, eps):
        super().__init__()
        self.spec, self.eps, self.ff, self.fp = spec, eps, spec.ff, padded(spec.ff)

    def load(self, take, C, dtype, device):
        up, down = take("up", self.ff, C), take("down", C, self.ff)
        self.put("w_down", fit(down, padded(C), self.fp), dtype, device)
        self.put("act", take("act", 4).float(), torch.float32, device)
        return [fit(up, self.fp, C)], []

    def forward(self, h, z):
        return (ops.linear_rows(ops.poly_norm(z, self.act, self.eps, self.ff), self.w_down),)


class MixtureFF(Weights):
    """Expert matrices stacked: w_gate_up (experts, gate rows then up rows, width), w_down (experts, width, fp)."""

    def __init__(self, spec, eps):
        super().__init__()
        self.spec, self.ff, self.fp = spec, spec.ff, padded(spec.ff)
        self.experts, self.top = spec.experts, spec.top
        if not 1 <= self.top <= self.experts:
            raise ValueError(f"top {self.top} of {self.experts} experts")

    def load(self, take, C, dtype, device):
        gu, down = [], []
        for e in range(self.experts):
            gate, up = take(f"e{e}.gate", self.ff, C), take(f"e{e}.up", self.ff, C)
            gu.append(torch.cat([fit(gate, self.fp, padded(C)), fit(up, self.fp, padded(C))]))
            down.append(fit(take(f"e{e}.down", C, self.ff), padded(C), self.fp))
        self.put("w_gate_up", torch.stack(gu), dtype, device)
        self.put("w_down", torch.stack(down), dtype, device)
        return [], [fit(take("router", self.experts, C), padded(self.experts), C)]

    def forward(self, h, z):
        return ops.mixture(h, self)


class Layer(Weights):
    def __init__(self, spec, eps):
        super().__init__()
        self.spec = spec
        self.attn = LatentAttention(spec.mixer, eps)
        self.mlp = None if spec.mlp is None else (DenseFF if isinstance(spec.mlp, DenseSpec) else MixtureFF)(spec.mlp, eps)

    def load(self, take, C, dtype, device):
        Cp = padded(C)
        self.put("norm", fit(1 + take("norm1", C).float(), Cp), torch.float32, device)
        rows = self.attn.load(under(take, "mix."), C, dtype, device)
        self.gates = []                                       # where the gates' segments of w_in's output begin
        for name in ("rg1", "rg2") if self.mlp is not None else ("rg1",):
            self.gates.append(sum(r.shape[0] for r in rows))
            rows.append(fit(take(name, C, C), Cp, C))
            self.put(name + "_bias", fit(take(name + ".b", C).float(), Cp), torch.float32, device)
        extra, router = self.mlp.load(under(take, "mlp."), C, dtype, device) if self.mlp is not None else ([], [])
        self.up_off = sum(r.shape[0] for r in rows)
        rows += extra
        self.n_in = sum(r.shape[0] for r in rows)
        self.put("w_all", fit(torch.cat(rows + router), self.n_in + sum(r.shape[0] for r in router), Cp), dtype, device)
        if router:
            self.mlp.router = self.w_all[self.n_in:]

    @property
    def w_in(self):
        return self.w_all[:self.n_in]


class Lupodra(ServedModel, NaiveSampler):
    step_graph = "LatentDecodeGraph"

    def __init__(self, config, dtype=None):
        super().__init__()
        self.config = config
        self.dtype = dtype or common.COMPUTE_DTYPE
        self.width = padded(config.n_embd)
        self.layers = nn.ModuleList([Layer(x, config.eps) for x in config.layers])
        self.runs = [(self.layers[i], again) for i, again in config.runs()]
        self.keep_x0 = any(again for _, again in self.runs)
        self.embed = self.final_norm = None

    # ------------------------------------------------------------------------- weights
    def pack(self, take, device):
        C = self.config.n_embd
        for i, layer in enumerate(self.layers):
            layer.load(under(take, f"l{i}."), C, self.dtype, device)
        embed = fit(take("embed", self.config.vocab_size, C), padded(self.config.vocab_size), self.width)
        self.embed = nn.Parameter(embed.to(self.dtype).to(device), requires_grad=False)
        norm = fit(1 + take("final.norm", C).float(), self.width)
        self.final_norm = nn.Parameter(norm.to(device), requires_grad=False)

    def tensor_shapes(self):
        """Names and shapes of the stored tensors."""
        C, out = self.config.n_embd, {"embed": (self.config.vocab_size, self.config.n_embd), "final.norm": (self.config.n_embd,)}
        for i, layer in enumerate(self.layers):
            m, f, l = layer.spec.mixer, layer.spec.mlp, f"l{i}."
            out.update({l + "norm1": (C,), l + "rg1": (C, C), l + "rg1.b": (C,),
                        l + "mix.dq": (m.q_rank, C), l + "mix.dq.norm": (m.q_rank,), l + "mix.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                        l + "mix.dkv": (m.kv_rank + m.rot_dim, C), l + "mix.dkv.norm": (m.kv_rank,), l + "mix.uk": (m.heads * m.dim, m.kv_rank),
                        l + "mix.uv": (m.heads * m.vdim, m.kv_rank), l + "mix.o": (C, m.heads * m.vdim)})
            if f is not None:
                out.update({l + "rg2": (C, C), l + "rg2.b": (C,)})
            if isinstance(f, DenseSpec):
                out.update({l + "mlp.up": (f.ff, C), l + "mlp.down": (C, f.ff), l + "mlp.act": (4,)})
            elif f is not None:
                out[l + "mlp.router"] = (f.experts, C)
                for e in range(f.experts):
                    out.update({f"{l}mlp.e{e}.gate": (f.ff, C), f"{l}mlp.e{e}.up": (f.ff, C), f"{l}mlp.e{e}.down": (C, f.ff)})
        return out

    def init_tensor(self, name, shape, normal):
        if name.endswith((".dq.norm", ".dkv.norm")):
            return torch.ones(shape)
        if name.endswith(".act"):
            return torch.tensor([0.7, 0.3, 0.1, 0.0])
        return super().init_tensor(name, shape, normal)

    # --------------------------------------------------------------------------- cache
    def make_cache(self, rows, sequence_len=None):
        """An empty paged store with one pool per layer run."""
        from nanochat_b200.engine import PagedLatentCache
        return PagedLatentCache(rows, [layer.attn.entry for layer, _ in self.runs], sequence_len or self.config.sequence_len,
                                self.get_device(), self.dtype)

    # ------------------------------------------------------------------------- forward
    @torch.inference_mode()
    def forward(self, idx, targets=None, kv_cache=None, want=None, residuals=None):
        """Logits (B, T, vocab), or (len(want), vocab) for the `want`ed rows of the flattened (B * T), None for none. The tokens continue
        what `kv_cache` holds and are appended to it. `residuals`, a list, collects the stream after every layer run."""
        if targets is not None:
            raise NotImplementedError("Lupodra is served, not trained: no loss")
        B, T = idx.shape
        if kv_cache is None:
            kv_cache = self.make_cache(B, T)
            kv_cache.reserve(0, T)
            kv_cache.begin_rows()
        cfg, eps, C = self.config, self.config.eps, self.config.n_embd
        first = self.runs[0][0].norm if self.runs else self.final_norm
        x, x0, h = ops.embed_norm(idx.reshape(-1), self.embed, cfg.vocab_size, first, eps, C, self.keep_x0)
        for run, (layer, _) in enumerate(self.runs):
            last = run + 1 == len(self.runs)
            norm = self.final_norm if last else self.runs[run + 1][0].norm
            extra = x0 if not last and self.runs[run + 1][1] else None
            z = ops.linear_rows(h, layer.w_in)
            gate = lambda k: z[:, layer.gates[k]:layer.gates[k] + self.width]
            terms = [(gate(0), layer.rg1_bias, layer.attn(z, kv_cache, run, T))]
            if layer.mlp is not None:
                terms.append((gate(1), layer.rg2_bias, *layer.mlp(h, z[:, layer.up_off:layer.n_in])))
            h = ops.gated_residual_norm(x, terms, cfg.residual_mult, extra, norm, eps, C, self.dtype)
            if residuals is not None:
                residuals.append((x if extra is None else x - extra)[:, :C].clone())
        kv_cache.advance(T)
        if want is not None:
            if len(want) == 0:
                return None
            h = h[torch.as_tensor(want, dtype=torch.long, device=h.device)]
        logits = ops.linear_rows(h, self.embed, torch.float32)[:, :cfg.vocab_size]
        return logits if want is not None else logits.reshape(B, T, -1)

    # ----------------------------------------------------------------- cost accounting
    def matmul_params_per_token(self):
        """Weights a token multiplies with: its chosen experts only."""
        total = self.config.vocab_size * self.config.n_embd
        for layer, _ in self.runs:
            total += layer.w_all.numel() + layer.attn.w_q.numel() + layer.attn.w_kv.numel() + layer.attn.w_o.numel()
            if isinstance(layer.mlp, DenseFF):
                total += layer.mlp.w_down.numel()
            elif layer.mlp is not None:
                total += layer.mlp.top * (layer.mlp.w_gate_up[0].numel() + layer.mlp.w_down[0].numel())
        return total

    def estimate_decode_flops(self, context_len):
        attn = 0
        for layer, _ in self.runs:
            a = layer.attn
            seen = context_len if a.window is None else min(context_len, a.window)
            attn += 2 * a.heads * seen * (2 * a.kv_rank + a.rot_dim)
        return 2 * self.matmul_params_per_token() + attn

    def estimate_prefill_flops(self, num_tokens):
        attn = 0
        for layer, _ in self.runs:
            a = layer.attn
            w = num_tokens if a.window is None else min(num_tokens, a.window)
            pairs = w * (w + 1) // 2 + (num_tokens - w) * w
            attn += 2 * a.heads * pairs * (a.spec.dim + a.rot_dim + a.spec.vdim)
        return 2 * self.matmul_params_per_token() * num_tokens + attn

    def kv_bytes_per_token(self):
        return sum(layer.attn.entry for layer, _ in self.runs) * self.dtype.itemsize

    def kv_read_bytes(self, context_len):
        total = 0
        for layer, _ in self.runs:
            seen = context_len if layer.attn.window is None else min(context_len, layer.attn.window)
            total += seen * layer.attn.entry * self.dtype.itemsize
        return total

    def decode_weight_bytes(self):
        """Bytes of weights one decode row reads."""
        return self.matmul_params_per_token() * self.dtype.itemsize


def load_folder(path, device, dtype=None, **serving):
    return served.load_folder(path, device, LupodraConfig.from_dict, Lupodra, dtype, **serving)
