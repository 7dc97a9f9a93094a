"""
Native bodies of the inference mechanisms (`nanochat_b200._S`): latent attention over a paged store, gated residual
updates, the normed-powers activation, mixtures of experts; layer-normed residual updates, the gated delta rule, window
attention whose values are its keys, linear attention with a fixed decay; and the row linear they share. Every function has
a plain PyTorch body of the same name in `reference.py`; `ops.__init__` picks one per call.

Rows: a step brings B sequences x T tokens, flattened to B * T rows (row r is token r % T of sequence r // T). Weight
holders (`p`) are the modules of `nanochat_b200.models` (lupodra, safepel): sizes padded to multiples of 8 (16 for what the store
holds) with zeros, so that every kernel reads whole 16-byte vectors.

bf16: products on the tcgen05 GEMM. float: the same kernels in float, products by the library in true float32.
"""

import torch

from nanochat_b200.utils.build import load_serving_extension

_S = load_serving_extension()

BF16 = torch.bfloat16
ABSORB_ROWS = 8          # portions up to this many tokens run on absorbed queries (weights dominate), longer ones expand
CHUNK_ROWS = 16          # portions above this many tokens run their recurrences in chunks, shorter ones token by token
FEW_OUTPUTS = 64         # products with up to this many outputs leave most SMs without a GEMM tile: eight rows at a time instead
SPLIT_KEYS = 64          # keys per tile of the tensor-core attention over stored entries


def check_status(like=None):
    """Raise if a serving kernel recorded a failed wait or a token without a page. Synchronises."""
    dev = like if like is not None else torch.empty(0, device="cuda")
    with torch.inference_mode():
        st = _S.read_status(dev)
    if st[0] != 0:
        code, detail = st[0] >> 24, st[0] & 0xFFFFFF
        raise RuntimeError(f"nanochat_b200 serving kernel reported an error: code={code} detail={detail:#x}")


def launch_count():
    return _S.launch_count()


def linear_rows(h, w, out_dtype=None):
    """h (R, K) @ w (N, K)^T; `out_dtype` float32 keeps the accumulator's precision."""
    if h.dtype == BF16:
        out = torch.empty(h.shape[0], w.shape[0], dtype=out_dtype or BF16, device=h.device)
        if w.shape[0] <= FEW_OUTPUTS:
            _S.gemv_plain(h, w, out)
        else:
            _S.gemm(h, w, out)
        return out
    before = torch.get_float32_matmul_precision()
    if before == "highest":
        return torch.mm(h, w.t())
    torch.set_float32_matmul_precision("highest")
    try:
        return torch.mm(h, w.t())
    finally:
        torch.set_float32_matmul_precision(before)


def embed_norm(ids, table, vocab, w, eps, n, keep_x0=False):
    """(x, x0, h) of the token embeddings: float residual stream, a copy of it when asked, and its norm."""
    shape = (ids.numel(), table.shape[1])
    x = torch.empty(shape, dtype=torch.float32, device=table.device)
    x0 = torch.empty_like(x) if keep_x0 else None
    h = torch.empty(shape, dtype=table.dtype, device=table.device)
    _S.embed_norm(ids, table, vocab, w, eps, n, x, x0, h)
    return x, x0, h


def gated_residual_norm(x, terms, mult, extra, w, eps, n, dtype):
    """x += mult * sum over terms of sigmoid(gate + bias) * y (+ extra), in place; returns norm(x) * w. A term is
    (gate, bias, y) or (gate, bias, expert rows, slot, weight)."""
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    _S.gated_residual_norm(x, [list(t) for t in terms], mult, extra, w, eps, n, h)
    return h


def poly_norm(z, coef, eps, n):
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    _S.poly_norm(z, coef, eps, n, out)
    return out


# ------------------------------------------------------------------------ latent attention

def attention_splits(p, rows, keys, tensor_cores):
    """CTAs that share one query's keys: enough to fill the SMs, at most one per key tile."""
    if tensor_cores:
        tiles, per_split = -(-keys // SPLIT_KEYS), rows * -(-p.heads // 16)
    else:
        tiles, per_split = -(-keys // 128), rows * p.heads
    return max(1, min(tiles, 296 // per_split, 32))


def latent_attention(p, z, cache, run, T):
    """The mixer's output (R, width) from the fused input projection z; appends the step's entries to the store."""
    R, pool = z.shape[0], cache.pools[run]
    dt = pool.dtype
    table, lens = cache.table, cache.cache_seqlens
    cq = torch.empty(R, p.qp, dtype=dt, device=z.device)
    expand = (dt == BF16 and R == T and T > ABSORB_ROWS and _S.attention_split_supported(p.dp, p.rp, p.vp))
    kv = None
    if expand:
        before = cache.get_pos()
        seen = before if p.window is None else min(before, p.window - 1)
        entries = torch.empty(seen + T, p.kvp + p.rp, dtype=dt, device=z.device)
        kv = entries[seen:]
    _S.latent_post(z, p.q_rank, p.q_norm, cq, p.c_off, p.kv_rank, p.kvp, p.kv_norm, p.eps, p.rot_off, p.rot_dim, p.freq,
                   pool, table, lens, T, kv)
    q = linear_rows(cq, p.w_q)
    if not expand:
        return linear_rows(latent_attention_absorbed(p, q, cache, run, T), p.w_o)
    if seen:
        _S.latent_gather(pool, table, 0, before - seen, entries[:seen])
    _S.rotate_heads(q, p.heads, p.dp, p.freq, table, lens, T)
    k_v = linear_rows(entries[:, :p.kvp], p.w_kv)                    # unrotated keys of all heads, then values
    q3 = q.view(T, p.heads, p.dp + p.rp)
    k3 = k_v[:, :p.heads * p.dp].unflatten(1, (p.heads, p.dp))
    v3 = k_v[:, p.heads * p.dp:].unflatten(1, (p.heads, p.vp))
    y = torch.empty(T, p.heads, p.vp, dtype=dt, device=z.device)
    window_left = -1 if p.window is None else p.window - 1
    _S.attention_split(q3[..., :p.dp], q3[..., p.dp:], k3, entries[:, p.kvp:], v3, y, window_left, p.scale)
    return linear_rows(y.view(T, -1), p.w_o)


def latent_attention_absorbed(p, q, cache, run, T):
    """Heads' values (R, heads * vp) by dot products with the stored entries themselves."""
    R, pool = q.shape[0], cache.pools[run]
    keys = cache.max_seq_len if p.window is None else min(p.window, cache.max_seq_len)
    splits = attention_splits(p, R, keys, pool.dtype == BF16)
    e = lambda *s, dtype=torch.float32: torch.empty(*s, dtype=dtype, device=q.device)
    qa, y = e(R, p.heads, p.kvp, dtype=pool.dtype), e(R, p.heads * p.vp, dtype=pool.dtype)
    ml, acc = e(R, p.heads, splits, 2), e(R, p.heads, splits, p.kvp)
    _S.absorb_query(q, p.heads, p.w_uk, qa, False)
    _S.latent_attention(qa, q, p.heads, p.dp, p.rot_dim, p.freq, p.kvp, pool, cache.table, cache.cache_seqlens, T,
                        p.window or 0, p.scale, splits, ml, acc, False)
    _S.latent_values(ml, acc, R, p.heads, splits, p.w_uv, y, False)
    return y


# ---------------------------------------------------------------------- mixture of experts

def route(h, p):
    """(expert ids, weights), each (R, top)."""
    logits = linear_rows(h, p.router, torch.float32)
    idx = torch.empty(h.shape[0], p.top, dtype=torch.int32, device=h.device)
    wt = torch.empty(h.shape[0], p.top, dtype=torch.float32, device=h.device)
    _S.route_topk(logits, p.experts, idx, wt)
    return idx, wt


def mixture(h, p):
    """The feed-forward's part of a residual term: (rows,) or (expert rows, slot, weight)."""
    R = h.shape[0]
    if h.dtype != BF16 or R * p.top <= ABSORB_ROWS * 4:
        idx, wt = route(h, p)
        act = torch.empty(R * p.top, p.fp, dtype=h.dtype, device=h.device)
        y = torch.empty(R, h.shape[1], dtype=h.dtype, device=h.device)
        _S.expert_gate_up(h, p.w_gate_up, idx, wt, act)
        _S.expert_down(act, p.w_down, idx, wt, y)
        return (y,)
    logits = linear_rows(h, p.router, torch.float32)
    ints = lambda *s: torch.empty(*s, dtype=torch.int32, device=h.device)
    idx, rank, slot, offsets = ints(R, p.top), ints(R, p.top), ints(R, p.top), ints(p.experts)
    wt = torch.empty(R, p.top, dtype=torch.float32, device=h.device)
    counts = torch.zeros(p.experts, dtype=torch.int32, device=h.device)
    _S.route_topk(logits, p.experts, idx, wt, counts, rank)
    tiles = -(-(R * p.top + p.experts * 127) // 128)
    tile_group = ints(tiles)
    rows = lambda n: torch.empty(tiles * 128, n, dtype=BF16, device=h.device)
    xg, gu, act, y = rows(h.shape[1]), rows(2 * p.fp), rows(p.fp), rows(h.shape[1])
    _S.group_rows(h, idx, rank, counts, offsets, tile_group, slot, xg)
    _S.gemm(xg, p.w_gate_up, gu, tile_group)
    _S.silu_mul(gu, tile_group, act)
    _S.gemm(act, p.w_down, y, tile_group)
    return (y, slot, wt)


# ----------------------------------------------------------- layer-normed residual, feed-forward

def embed_layer_norm(ids, table, vocab, w_embed, w, eps, n):
    """(x, h): the normed token embeddings as float residual stream, and the first sublayer's norm of it."""
    x = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    h = torch.empty(x.shape, dtype=table.dtype, device=table.device)
    _S.layer_norm_residual(ids, table, vocab, w_embed, x, w, eps, n, h)
    return x, h


def layer_norm_residual(x, y, w_post, w, eps, n, dtype):
    """x += norm(y) * w_post in place; returns norm(x) * w."""
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    _S.layer_norm_residual(None, y, 0, w_post, x, w, eps, n, h)
    return h


def relu_glu(h, w_gate_up):
    """relu(h Wg^T) * (h Wu^T): the activation and the product ride on the two products' epilogues."""
    fp = w_gate_up.shape[0] // 2
    if h.dtype == BF16:
        out = torch.empty(h.shape[0], fp, dtype=BF16, device=h.device)
        _S.gemm(h, w_gate_up[:fp], out, epi=1)
        _S.gemm(h, w_gate_up[fp:], out, epi=2, aux=out)
        return out
    return torch.relu(linear_rows(h, w_gate_up[:fp])) * linear_rows(h, w_gate_up[fp:])


# -------------------------------------------------------------------------------- recurrences

def _prepared(z, T, heads, kv_heads, dp, vp):
    """Where a prepare kernel puts its outputs: tiles of the chunk kernels, or rows for the token-by-token kernel."""
    R = z.shape[0]
    if z.dtype == BF16 and T > CHUNK_ROWS and _S.recurrence_chunks_supported(dp):
        return torch.empty(_S.recurrence_tiles(R // T, T, heads, kv_heads, dp, vp), dtype=torch.uint8, device=z.device)
    return torch.empty(R, 2 * kv_heads * dp + heads * vp, dtype=z.dtype, device=z.device)


def _recurrence(act, z, heads, kv_heads, dp, vp, state, cache, T, norms=None, beta_g=None, log_decay=None):
    R = z.shape[0]
    o, scratch = torch.empty(R, heads * vp, dtype=z.dtype, device=z.device), None
    if act.dtype == torch.uint8:
        scratch = torch.empty(_S.recurrence_scratch(R // T, T, heads, beta_g is not None), dtype=torch.uint8, device=z.device)
    _S.recurrence(act, [heads, kv_heads, dp, vp], norms, beta_g, log_decay, state, cache.cache_seqlens, T, o, scratch)
    return o


def gated_delta(p, z, ba, cache, run, T):
    """What the mixer's output product reads (R, heads * vp); state and convolution inputs move on by T tokens."""
    R, S, ring = z.shape[0], cache.states[run]["S"], cache.states[run]["ring"]
    y = torch.empty(R, p.y_width, dtype=z.dtype, device=z.device)
    if T == 1 and _S.delta_step_supported(p.dp, p.vp):
        _S.delta_step(z, p.sizes, p.conv, ba, p.neg_a, p.dt_bias, ring, S, cache.cache_seqlens, p.norm, p.eps, p.gate_off, y)
        return y
    act = _prepared(z, T, p.heads, p.kv_heads, p.dp, p.vp)
    norms = torch.empty(R, 2 * p.kv_heads, device=z.device)
    beta_g = torch.empty(R, 2 * p.heads, device=z.device)
    _S.delta_prepare(z, p.sizes, p.conv, ba, p.neg_a, p.dt_bias, ring, cache.cache_seqlens, T, act, norms, beta_g)
    o = _recurrence(act, z, p.heads, p.kv_heads, p.dp, p.vp, S, cache, T, norms, beta_g)
    _S.delta_finish(o, z[:, p.gate_off:p.gate_off + p.y_width], p.norm, p.eps, y, z, p.sizes, p.conv, p.neg_a, p.dt_bias, ring, cache.cache_seqlens, T)
    return y


def decay_attention(p, z, cache, run, T, y):
    """y (R, heads * vp) from p's segments of z; the state moves on by T tokens."""
    R, S = z.shape[0], cache.states[run]["S"]
    if T == 1 and _S.decay_step_supported(p.dp, p.vp):
        o = torch.empty(R, p.y_width, device=z.device)
        _S.decay_step(z, p.sizes, p.reals, p.log_decay, S, cache.cache_seqlens, p.norm, o, cache.done, y)
        return y
    act = _prepared(z, T, p.heads, p.heads, p.dp, p.vp)
    _S.decay_prepare(z[:, p.q_off:p.gate_off], p.heads, p.dp, p.vp, T, act)
    o = _recurrence(act, z, p.heads, p.heads, p.dp, p.vp, S, cache, T, log_decay=p.log_decay)
    _S.norm_gate(o, z[:, p.gate_off:p.end], p.norm, p.eps, 1, p.heads * p.vdim, True, p.out_scale, y)
    return y


# ----------------------------------------------------------------- window attention, keys as values

def window_attention(p, z, cache, run, T, y):
    """y (R, heads * dp) from p's segments of z (the queries' is overwritten); appends the step's entries to the store."""
    R, pool, table, lens = z.shape[0], cache.pools[run], cache.table, cache.cache_seqlens
    if T == 1 and _S.window_step_supported(pool.dtype != BF16, p.dp):
        _S.window_step(z, p.sizes, p.reals, p.freq, pool, table, lens, y)
        return y
    tiles = pool.dtype == BF16 and R == T and _S.attention_capped_supported(p.dp, p.dp)
    entries = None
    if tiles:
        before = cache.get_pos()
        seen = before if p.window is None else min(before, p.window - 1)
        entries = torch.empty(seen + T, p.entry, dtype=pool.dtype, device=z.device)
    _S.window_post(z, p.sizes, p.reals, p.freq, pool, table, lens, T, entries[seen:] if tiles else None)
    if not tiles:
        _S.window_attention(z, p.sizes, p.reals, p.freq, pool, table, lens, T, y)
        return y
    if seen:
        _S.latent_gather(pool, table, 0, before - seen, entries[:seen])
    kv = entries.view(-1, 2, p.kv_heads, p.dp)
    _S.attention_capped(z[:, p.q_off:p.k_off].unflatten(1, (p.heads, p.dp)), kv[:, 0], kv[:, 1], y.unflatten(1, (p.heads, p.dp)),
                        -1 if p.window is None else p.window - 1, p.scale, p.softcap, p.out_scale)
    return y


def window_and_decay(left, right, z, cache, run, T):
    """Both mechanisms on one z into one y: [left | right]."""
    y = torch.empty(z.shape[0], left.y_width + right.y_width, dtype=z.dtype, device=z.device)
    y_left, y_right = y[:, :left.y_width], y[:, left.y_width:]
    if T == 1 and _S.window_step_supported(z.dtype != BF16, left.dp) and _S.decay_step_supported(right.dp, right.vp):
        o = torch.empty(z.shape[0], right.y_width, device=z.device)
        _S.parallel_step(z, left.sizes, left.reals, left.freq, cache.pools[run], cache.table, cache.cache_seqlens, y_left,
                         right.sizes, right.reals, right.log_decay, cache.states[run]["S"], right.norm, o, cache.done, y_right)
        return y
    window_attention(left, z, cache, run, T, y_left)
    decay_attention(right, z, cache, run, T, y_right)
    return y
