"""
Plain, slow restatement of the Safepel decoder for tests: one function per mechanism, whole sequences only, no cache, no
batching, token by token where the mechanism is a recurrence, nothing imported from the package. Works on a dict of
name -> tensor and the parsed configuration, in the floating-point type of the weights it is given (tests use float64).

Shapes: a sequence is (T, width); positions count from 0.
"""

import math

import torch

UNIT_EPS = 1e-6


# ------------------------------------------------------------------------------ norms

def layer_norm(x, w, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def silu(x):
    return x * torch.sigmoid(x)


# --------------------------------------------------------------------------- gated delta rule

def short_conv(x, w):
    """x (T, channels), w (channels, taps): the last tap meets the current token, zeros stand before the first."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for i in range(taps):
            if t - i >= 0:
                out[t] += w[:, taps - 1 - i] * x[t - i]
    return out


def delta_rule(q, k, v, beta, g):
    """q, k (T, H, d), v (T, H, e), beta and g (T, H) -> (T, H, e). The state is written before it is read."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out


def delta_mixer(h, p, cfg, eps):
    """p: the mixer's tensors by their short name ('q', 'q.conv', ...)."""
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ p[n].T, p[n + ".conv"])) for n in ("q", "k", "v"))
    per = lambda x: unit(x.reshape(T, G, d)).repeat_interleave(H // G, dim=1)
    q, k, v = per(q) * d ** -0.5, per(k), v.reshape(T, H, e)
    beta = torch.sigmoid(h @ p["b"].T)
    g = torch.exp(-torch.exp(p["A_log"]) * torch.nn.functional.softplus(h @ p["a"].T + p["dt_bias"], threshold=40.0))
    o = rms_norm(delta_rule(q, k, v, beta, g), p["norm"], eps)
    return (o.reshape(T, H * e) * silu(h @ p["g"].T)) @ p["o"].T


# ------------------------------------------------------------ window attention, keys as values

def rotate_pairs(x, positions, base, dims):
    """x (T, ..., n): entries 2i and 2i + 1 of the first `dims` turn by the angle position * base^(-2i / dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    angle = angle.reshape(angle.shape[0], *([1] * (x.dim() - 2)), dims // 2)
    c, s = angle.cos().to(x.dtype), angle.sin().to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(T, window):
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window)


def window_attention(h, p, cfg):
    H, G, d = cfg["heads"], cfg["kv_heads"], cfg["dim"]
    T = h.shape[0]
    pos = torch.arange(T)
    turn = lambda x: rotate_pairs(x, pos, cfg["rot"]["base"], cfg["rot"]["dims"])
    q = (h @ p["q"].T).reshape(T, H, d)
    k = (h @ p["k"].T).reshape(T, G, d)
    wide = lambda x: x.repeat_interleave(H // G, dim=1)
    score = torch.einsum("ihd,jhd->hij", turn(q), wide(turn(k))) * cfg["scale"]
    score = cfg["softcap"] * torch.tanh(score / cfg["softcap"])
    w = torch.softmax(score.masked_fill(~visible(T, cfg["mask"]["size"]), -math.inf), dim=-1)
    y = torch.einsum("hij,jhd->ihd", w, wide(k)).reshape(T, H * d)
    return y @ p["o"].T


# -------------------------------------------------------------- linear attention with fixed decay

def decay_attention(h, p, cfg, eps):
    H, d, e = cfg["heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q, k = (silu(h @ p[n].T).reshape(T, H, d) for n in ("q", "k"))
    v = silu(h @ p["v"].T).reshape(T, H, e)
    decay = torch.tensor(cfg["decay"], dtype=torch.float64).to(h.dtype)[:, None, None]
    S = torch.zeros(H, d, e, dtype=h.dtype)
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    y = rms_norm(out.reshape(T, H * e), p["norm"], eps) * torch.sigmoid(h @ p["g"].T)
    return y @ p["o"].T


def parallel_mixer(h, p, cfg, eps):
    left = window_attention(h, under(p, "left."), cfg["left"])
    right = decay_attention(h, under(p, "right."), cfg["right"], eps)
    return cfg["left_scale"] * left + cfg["right_scale"] * right


# -------------------------------------------------------------------------- layers

def dense_ff(h, p):
    return (torch.relu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def under(params, prefix):
    return {k[len(prefix):]: v for k, v in params.items() if k.startswith(prefix)}


def mix(h, p, spec, eps):
    return (delta_mixer if spec["type"] == "delta" else parallel_mixer)(h, p, spec["mixer"], eps)


def layer(x, params, i, cfg):
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    p = under(params, f"l{i}.")
    x = x + layer_norm(mix(layer_norm(x, p["norm1"], eps), under(p, "mix."), spec, eps), p["norm1b"], eps)
    if spec.get("mlp") is not None:
        x = x + layer_norm(dense_ff(layer_norm(x, p["norm2"], eps), under(p, "mlp.")), p["norm2b"], eps)
    return x


def forward(params, cfg, tokens, layers=None):
    """(T, vocab) logits. `layers`, when a list, collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = layer_norm(params["embed"][torch.as_tensor(tokens)], params["embed.norm"], eps)
    for i in range(len(cfg["layers"])):
        x = layer(x, params, i, cfg)
        if layers is not None:
            layers.append(x)
    return layer_norm(x, params["final.norm"], eps) @ params["head"].T * cfg["logit_scale"]


# ------------------------------------------------------------------- small random models

def tensor_shapes(cfg):
    C = cfg["width"]
    out = {"embed": (cfg["vocab"], C), "embed.norm": (C,), "final.norm": (C,), "head": (cfg["vocab"], C)}
    for i, spec in enumerate(cfg["layers"]):
        m, l = spec["mixer"], f"l{i}."
        out[l + "norm1"] = out[l + "norm1b"] = (C,)
        if spec["type"] == "delta":
            H, G, d, e, t = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                out[f"{l}mix.{n}"], out[f"{l}mix.{n}.conv"] = (rows, C), (rows, t)
            out.update({l + "mix.b": (H, C), l + "mix.a": (H, C), l + "mix.A_log": (H,), l + "mix.dt_bias": (H,), l + "mix.norm": (e,),
                        l + "mix.g": (H * e, C), l + "mix.o": (C, H * e)})
        else:
            a, b = m["left"], m["right"]
            out.update({l + "mix.left.q": (a["heads"] * a["dim"], C), l + "mix.left.k": (a["kv_heads"] * a["dim"], C),
                        l + "mix.left.o": (C, a["heads"] * a["dim"])})
            H, d, e = b["heads"], b["dim"], b["vdim"]
            out.update({l + "mix.right.q": (H * d, C), l + "mix.right.k": (H * d, C), l + "mix.right.v": (H * e, C),
                        l + "mix.right.g": (H * e, C), l + "mix.right.o": (C, H * e), l + "mix.right.norm": (H * e,)})
        if spec.get("mlp") is not None:
            f = spec["mlp"]["ff"]
            out[l + "norm2"] = out[l + "norm2b"] = (C,)
            out.update({l + "mlp.gate": (f, C), l + "mlp.up": (f, C), l + "mlp.down": (C, f)})
    return out


def random_params(cfg, seed=0, sharp=1.0):
    """bf16-representable float32 weights. `sharp` scales the attention's query and key projections: larger values make
    single keys stand out."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith("A_log"):
            w = -1.5 + 1.5 * r
        elif name.endswith("dt_bias"):
            w = -2.0 + r
        elif len(shape) == 1:
            w = 1 + 0.2 * r
        elif name.endswith(".conv"):
            w = r / math.sqrt(shape[1])
        elif name == "embed":
            w = 0.7 * r
        else:
            w = r * (1.2 / math.sqrt(shape[1]))
            if name.endswith(("left.q", "left.k")):
                w = w * sharp
        out[name] = w.to(torch.bfloat16).float()
    return out
