"""
Plain, slow restatement of the Lupodra decoder for tests: one function per mechanism, whole sequences only, no cache,
no batching, nothing imported from the package. Works on a dict of name -> tensor and the parsed configuration, in
the floating-point type of the weights it is given (tests use float64 or float32).

Shapes: a sequence is (T, width); positions count from 0.
"""

import math

import torch


# ------------------------------------------------------------------------------ norms

def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return x / root_mean_square(x, eps) * (1 + w)


def plain_norm(x, w, eps):
    return x / root_mean_square(x, eps) * w


# --------------------------------------------------------------------------- rotation

def rotate_half(x, positions, base, dims):
    """x (T, ..., n): the first `dims` entries of the last axis turn by position-dependent angles, entry i with entry
    i + dims / 2."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    freq = base ** (-2.0 * i / dims)
    angle = positions.to(torch.float64)[:, None] * freq[None, :]
    angle = angle.reshape(angle.shape[0], *([1] * (x.dim() - 2)), half)
    c, s = angle.cos().to(x.dtype), angle.sin().to(x.dtype)
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


# -------------------------------------------------------------------- latent attention

def visible(T, window):
    """(T, T) mask: query i sees key j when 0 <= i - j < window."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = d >= 0
    return seen if window is None else seen & (d < window)


def latent_attention(h, p, cfg, eps):
    """p: the mixer's tensors by their short name ('dq', 'dq.norm', ...)."""
    H, dn, dr, dv, rank = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    T = h.shape[0]
    pos = torch.arange(T)
    cq = plain_norm(h @ p["dq"].T, p["dq.norm"], eps)
    q = (cq @ p["uq"].T).reshape(T, H, dn + dr)
    q_flat, q_turn = q[..., :dn], rotate_half(q[..., dn:], pos, cfg["rot"]["base"], cfg["rot"]["dims"])
    down = h @ p["dkv"].T
    c = plain_norm(down[:, :rank], p["dkv.norm"], eps)
    k_turn = rotate_half(down[:, rank:], pos, cfg["rot"]["base"], cfg["rot"]["dims"])
    k_flat = (c @ p["uk"].T).reshape(T, H, dn)
    v = (c @ p["uv"].T).reshape(T, H, dv)
    score = torch.einsum("ihd,jhd->hij", q_flat, k_flat) + torch.einsum("ihd,jd->hij", q_turn, k_turn)
    score = score * cfg["scale"]
    mask = cfg.get("mask") or {}
    score = score.masked_fill(~visible(T, mask.get("size")), -math.inf)
    w = torch.softmax(score, dim=-1)
    y = torch.einsum("hij,jhd->ihd", w, v).reshape(T, H * dv)
    return y @ p["o"].T


# -------------------------------------------------------------------------- feed-forward

def poly_norm(z, coef, eps):
    a, b, c, e = coef.unbind()
    n = lambda t: t / root_mean_square(t, eps)
    return a * n(z) + b * n(z * z) + c * n(z * z * z) + e


def dense_ff(h, p, eps):
    return poly_norm(h @ p["up"].T, p["act"], eps) @ p["down"].T


def route(h, router, top):
    """Chosen experts (T, top) and their weights."""
    z = h @ router.T
    best, who = torch.topk(z, top, dim=-1)
    return who, torch.softmax(best, dim=-1)


def expert_ff(h, p, n):
    z = h @ p[f"e{n}.gate"].T
    return (z * torch.sigmoid(z) * (h @ p[f"e{n}.up"].T)) @ p[f"e{n}.down"].T


def mixture_ff(h, p, cfg):
    who, weight = route(h, p["router"], cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(who[t].tolist(), weight[t]):
            out[t] += w * expert_ff(h[t:t + 1], p, e)[0]
    return out


# --------------------------------------------------------------------------------- layers

def under(params, prefix):
    return {k[len(prefix):]: v for k, v in params.items() if k.startswith(prefix)}


def gate(h, w, b):
    return torch.sigmoid(h @ w.T + b)


def layer(x, params, i, cfg):
    spec, eps, m = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"]
    p = under(params, f"l{i}.")
    h = model_norm(x, p["norm1"], eps)
    change = gate(h, p["rg1"], p["rg1.b"]) * latent_attention(h, under(p, "mix."), spec["mixer"], eps)
    if spec.get("mlp") is not None:
        q = under(p, "mlp.")
        ff = dense_ff(h, q, eps) if spec["mlp"]["kind"] == "dense" else mixture_ff(h, q, spec["mlp"])
        change = change + gate(h, p["rg2"], p["rg2.b"]) * ff
    return x + m * change


def run_order(cfg):
    """(layer, opens a repeated pass) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for k in range(loop["times"]):
        order += [(i, k > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(params, cfg, tokens, layers=None):
    """(T, vocab) logits. `layers`, when a list, collects the residual stream after every layer run."""
    emb = params["embed"][torch.as_tensor(tokens)]
    x = emb
    for i, again in run_order(cfg):
        if again:
            x = x + emb
        x = layer(x, params, i, cfg)
        if layers is not None:
            layers.append(x)
    return model_norm(x, params["final.norm"], cfg["norm"]["eps"]) @ params["embed"].T


# ------------------------------------------------------------------- small random models

def tensor_shapes(cfg):
    C = cfg["width"]
    out = {"embed": (cfg["vocab"], C), "final.norm": (C,)}
    for i, spec in enumerate(cfg["layers"]):
        m, l = spec["mixer"], f"l{i}."
        H = m["heads"]
        out[l + "norm1"] = (C,)
        out[l + "mix.dq"] = (m["q_rank"], C)
        out[l + "mix.dq.norm"] = (m["q_rank"],)
        out[l + "mix.uq"] = (H * (m["dim"] + m["rot_dim"]), m["q_rank"])
        out[l + "mix.dkv"] = (m["kv_rank"] + m["rot_dim"], C)
        out[l + "mix.dkv.norm"] = (m["kv_rank"],)
        out[l + "mix.uk"] = (H * m["dim"], m["kv_rank"])
        out[l + "mix.uv"] = (H * m["vdim"], m["kv_rank"])
        out[l + "mix.o"] = (C, H * m["vdim"])
        out[l + "rg1"], out[l + "rg1.b"] = (C, C), (C,)
        f = spec.get("mlp")
        if f is None:
            continue
        out[l + "rg2"], out[l + "rg2.b"] = (C, C), (C,)
        if f["kind"] == "dense":
            out[l + "mlp.up"], out[l + "mlp.down"], out[l + "mlp.act"] = (f["ff"], C), (C, f["ff"]), (4,)
        else:
            n = f["expert"]["ff"]
            out[l + "mlp.router"] = (f["router"]["experts"], C)
            for e in range(f["router"]["experts"]):
                q = f"{l}mlp.e{e}."
                out[q + "gate"], out[q + "up"], out[q + "down"] = (n, C), (n, C), (C, n)
    return out


def random_params(cfg, seed=0, sharp=1.0):
    """bf16-representable float32 weights. `sharp` scales the query and key projections: larger values make single
    keys stand out."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith("mlp.act"):
            w = 0.5 + 0.3 * r
        elif name.endswith("q.norm") or name.endswith("kv.norm"):
            w = 1 + 0.2 * r
        elif len(shape) == 1:
            w = 0.2 * r
        elif name == "embed":
            w = 0.7 * r
        else:
            w = r * (1.2 / math.sqrt(shape[1]))
            if name.endswith(".uq"):
                w = w * sharp
        out[name] = w.to(torch.bfloat16).float()
    return out
