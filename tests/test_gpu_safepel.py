"""The Safepel model on the serving kernels: every mechanism, cut, batch and edge against the float64 oracle, in float32
(sharp) and bf16 (the serving precision)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import safepel_cases as cases
import safepel_oracle as oracle

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def randn(*shape, seed=0, dtype=BF16):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


def kernels():
    from nanochat_b200 import ops
    return ops.serving_module()


@DTYPES
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_cut_of_a_prompt_gives_the_oracles_logits(name, dtype):
    cases.check_cuts(name, "cuda", dtype, 150, [[10 ** 6], [1], [2], [100, 1], [70, 2, 5, 1, 1, 30, 9], [17, 65, 1]])


@DTYPES
@pytest.mark.parametrize("spec", [dict(heads=4, kv_heads=2, dim=24, vdim=40, conv=4), dict(heads=2, kv_heads=1, dim=128, vdim=72, conv=2),
                                  dict(heads=3, kv_heads=3, dim=13, vdim=19, conv=1), dict(heads=6, kv_heads=1, dim=64, vdim=64, conv=9),
                                  dict(heads=1, kv_heads=1, dim=200, vdim=264, conv=4)])
def test_delta_rule(spec, dtype):
    """Chunk borders at multiples of 64 from a portion's start, short portions below the chunked path, single tokens."""
    for strength in ({}, {"memory": True}, {"forget": True}, {"write": True, "memory": True}):
        cases.check_delta("cuda", dtype, spec, 140, [[10 ** 6], [64, 1], [65, 2, 3, 1, 40], [2], [63, 17, 1, 1, 20]], **strength)


@DTYPES
@pytest.mark.parametrize("spec", [cases.right((1.0, 0.3), 8, 12), cases.right((0.0, 0.999, 0.9), 5, 3), cases.right((1.0, 0.97), 128, 136),
                                  cases.right((1.0,), 200, 600)])
def test_decay_attention(spec, dtype):
    cases.check_decay("cuda", dtype, spec, 140, [[10 ** 6], [64, 1], [65, 2, 3, 1, 40], [2], [63, 17, 1, 1, 20]])


@DTYPES
@pytest.mark.parametrize("window,sizes", [(11, dict(heads=4, kv_heads=2, dim=32, rot_dims=8)), (130, dict(heads=4, kv_heads=1, dim=64, rot_dims=32)),
                                          (64, dict(heads=2, kv_heads=2, dim=128, rot_dims=64)), (1, dict(heads=2, kv_heads=1, dim=16, rot_dims=4)),
                                          (65, dict(heads=20, kv_heads=1, dim=40, rot_dims=16)), (90, dict(heads=1, kv_heads=1, dim=160, rot_dims=32))])
def test_window_edges(window, sizes, dtype):
    m = cases.left(window=window, softcap=12.0, scale=sizes["dim"] ** -0.5, **sizes)
    T = window + 140
    keys = [k for k in (0, 1, 63, 64, 127, 128) if k + window < T]
    cases.check_window_edges("cuda", dtype, m, 192, T, keys, lambda key, w: [[10 ** 6], [key + 1, 1], [max(key + w - 1, 1), 1, 2, 7], [key + w, 20, 1]])


@DTYPES
def test_pages_and_states_are_reused(dtype):
    cases.check_reuse("cuda", dtype)


@DTYPES
@pytest.mark.parametrize("rows", [1, 2, 5, 8, 9, 20])
def test_rows_of_a_batch_are_independent(rows, dtype):
    for name in ("mixed", "wide", "heads"):
        cases.check_rows("cuda", dtype, rows, name)


@DTYPES
def test_unequal_sequences_side_by_side(dtype):
    cases.check_unequal_sequences("cuda", dtype)


@DTYPES
def test_several_sequences_in_one_pass(dtype):
    """Prompts of equal length in one forward, without and with what earlier tokens left."""
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=14)
    model = cases.model_of(cfg, params, "cuda", dtype)
    tokens = [cases.tokens_of(cfg, 110, 70 + r) for r in range(3)]
    cache = model.make_cache(3, 110)
    cache.reserve(0, 110)
    cache.begin_rows()
    ids = torch.tensor(tokens, device="cuda")
    got = torch.cat([model.forward(ids[:, a:b], kv_cache=cache) for a, b in ((0, 80), (80, 83), (83, 110))], 1)
    cases.assert_close(got, torch.stack([oracle.forward(cases.double(params), cfg, t) for t in tokens]), dtype)


@DTYPES
@pytest.mark.parametrize("samples", [1, 3, 12])
def test_greedy_generation(samples, dtype):
    cases.check_greedy("cuda", dtype, samples)


@DTYPES
def test_long_decoding(dtype):
    cfg = cases.config([(cases.delta(heads=2, kv_heads=1, dim=8, vdim=8), 24), (cases.parallel(cases.left(heads=2, kv_heads=1, dim=8, rot_dims=8, window=6),
                                                                                                cases.right((1.0, 0.99), 8, 8)), 24)], width=48)
    params = oracle.random_params(cfg, seed=11)
    tokens = cases.tokens_of(cfg, 600)
    engine = cases.Engine(cases.model_of(cfg, params, "cuda", dtype), None)
    cases.assert_close(cases.feed(engine, tokens, [2, 1]), oracle.forward(cases.double(params), cfg, tokens), dtype)


@DTYPES
def test_far_positions_turn_by_the_right_angle(dtype):
    """The rotation at position 20,000: a window's scores depend on differences of positions only."""
    m = cases.left(heads=2, kv_heads=1, dim=32, rot_dims=32, window=16, base=100.0, softcap=20.0, scale=0.4)
    one = cases.window_mixer("cuda", dtype, m, 64)
    h = one.inputs(40)
    want = one.expected(h)
    cache = one.model.make_cache(1, 20100)
    cache.reserve(0, 20100)
    cache.begin_rows()
    start = 20000
    cache.cache_seqlens.fill_(start)
    cache._pos = start
    got = []
    for a, b in ((0, 20), (20, 39), (39, 40)):
        got.append(one.model.layers[0].mix(h[a:b].to(dtype).cuda(), cache, 0, b - a).float().cpu())
        cache.advance(b - a)
    cases.assert_close(torch.cat(got)[16:], want[16:], dtype, tol=cases.MIXER_TOL)      # from there on the window holds these tokens only


# ------------------------------------------------------------------------------ kernels

@pytest.mark.parametrize("T,S", [(1, 1), (9, 9), (128, 128), (129, 300), (300, 300), (40, 1000)])
@pytest.mark.parametrize("H,G,D", [(2, 1, 64), (4, 2, 128), (3, 3, 8), (5, 1, 72), (6, 2, 40)])
def test_capped_attention(T, S, H, G, D):
    """The tensor-core prompt kernel with grouped keys, a soft cap and an output factor, windows around tile edges."""
    K = kernels()._S
    q, kv = randn(T, H, D, seed=1), randn(S, 2, G, D, seed=2)
    scale = 2.0 * D ** -0.5
    raw = torch.einsum("thd,shd->hts", q.double(), kv[:, 0].double().repeat_interleave(H // G, 1)) * scale
    gap = torch.arange(S - T, S)[:, None] - torch.arange(S)
    dq, dkv = q.cuda(), kv.cuda()
    for window in (None, 1, 2, 64, 127, 128, 129, 200):
        for cap in (0.0, 1.5, 30.0):
            o = torch.full((T, H, D), float("nan"), dtype=BF16, device="cuda")
            K.attention_capped(dq, dkv[:, 0], dkv[:, 1], o, -1 if window is None else window - 1, scale, cap, 0.6)
            s = cap * torch.tanh(raw / cap) if cap else raw
            w = torch.softmax(s.masked_fill((gap < 0) | (gap >= (window or 10 ** 9)), -float("inf")), -1)
            want = 0.6 * torch.einsum("hts,shd->thd", w, kv[:, 1].double().repeat_interleave(H // G, 1))
            assert cases.row_errors(o, want).max() < 1.5e-2, (window, cap, cases.row_errors(o, want).max())
    kernels().check_status()


def recurrence_inputs(seqs, T, H, G, dp, vp, seed=0):
    R = seqs * T
    act = randn(R, 2 * G * dp + H * vp, seed=seed)
    q, k = (act[:, i * G * dp:(i + 1) * G * dp].double().view(R, G, dp) for i in range(2))
    norms = torch.cat([1 / q.norm(dim=-1) * dp ** -0.5, 1 / k.norm(dim=-1)], 1).float()
    g = torch.Generator().manual_seed(seed + 1)
    log_g = -torch.exp(4 * torch.randn(R, H, generator=g) - 3)                  # from next to nothing to e^-400 a token
    beta_g = torch.cat([torch.sigmoid(2 * torch.randn(R, H, generator=g)), log_g], 1)
    return act, norms, beta_g, torch.randn(seqs, H, dp, vp, generator=g)


def as_tiles(act, seqs, H, G, dp, vp):
    """Rows of q, k, v as the chunk kernels' tiles: 64 tokens of a head, heads padded to 64 or 128 columns, pitch 8 more;
    then v in slices of 16 columns, pitch 24. Padding that no one may read is NaN."""
    K = kernels()._S
    T = act.shape[0] // seqs
    chunks, D, slices = -(-T // 64), 64 if dp <= 64 else 128, -(-vp // 16)
    full = torch.zeros(seqs, chunks * 64, act.shape[1], dtype=BF16)
    full[:, :T] = act.view(seqs, T, -1)
    full = full.view(seqs, chunks, 64, -1)
    qk = torch.full((seqs, chunks, G, 2, 64, D + 8), float("nan"), dtype=BF16)
    qk[..., :D] = 0
    qk[..., :dp] = full[..., :2 * G * dp].view(seqs, chunks, 64, 2, G, dp).permute(0, 1, 4, 3, 2, 5)
    wide = torch.zeros(seqs, chunks, 64, H, slices * 16, dtype=BF16)
    wide[..., :vp] = full[..., 2 * G * dp:].view(seqs, chunks, 64, H, vp)
    v = torch.full((seqs, chunks, H, slices, 64, 24), float("nan"), dtype=BF16)
    v[..., :16] = wide.view(seqs, chunks, 64, H, slices, 16).permute(0, 1, 3, 4, 2, 5)
    out = torch.cat([qk.flatten(), v.flatten()]).view(torch.uint8).cuda()
    assert out.numel() == K.recurrence_tiles(seqs, T, H, G, dp, vp)
    return out


def recurrence_expected(act, seqs, H, G, dp, vp, state, norms=None, beta_g=None, log_decay=None):
    R = act.shape[0]
    T, out, states = R // seqs, [], []
    for b in range(seqs):
        rows = slice(b * T, (b + 1) * T)
        a, S = act[rows].double(), state[b].double()
        q, k = (a[:, i * G * dp:(i + 1) * G * dp].view(T, G, dp) for i in range(2))
        v = a[:, 2 * G * dp:].view(T, H, vp)
        if beta_g is not None:
            q, k = q * norms[rows, :G, None].double(), k * norms[rows, G:, None].double()
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        for t in range(T):
            if beta_g is not None:
                S = S * torch.exp(beta_g[b * T + t, H:].double())[:, None, None]
                u = beta_g[b * T + t, :H].double()[:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
            else:
                S, u = S * torch.exp(log_decay.double())[:, None, None], v[t]
            S = S + k[t][:, :, None] * u[:, None, :]
            out.append(torch.einsum("hde,hd->he", S, q[t]).reshape(-1))
        states.append(S)
    return torch.stack(out), torch.stack(states)


@pytest.mark.parametrize("seqs,T,H,G,dp,vp", [(1, 64, 2, 1, 64, 64), (1, 1, 1, 1, 8, 8), (2, 63, 3, 3, 24, 40), (1, 200, 4, 2, 128, 128), (1, 65, 2, 2, 72, 24), (3, 130, 2, 1, 16, 16)])
@pytest.mark.parametrize("delta", [True, False])
@pytest.mark.parametrize("fresh", [True, False])
def test_recurrence_in_chunks_and_token_by_token(seqs, T, H, G, dp, vp, delta, fresh):
    """Both kernels in bf16 against float64, and the state they leave: float, so far closer than a bf16 state could be."""
    K = kernels()._S
    if not delta:
        G = H
    act, norms, beta_g, state = recurrence_inputs(seqs, T, H, G, dp, vp)
    log_decay = torch.linspace(-3.0, 0.0, H) if H > 1 else torch.tensor([-0.01])
    log_decay[0] = -1e4
    extra = dict(norms=norms, beta_g=beta_g) if delta else dict(log_decay=log_decay)
    want, want_state = recurrence_expected(act, seqs, H, G, dp, vp, torch.zeros_like(state) if fresh else state, **extra)
    lens = torch.full((seqs,), 0 if fresh else 5, dtype=torch.int32, device="cuda")
    dev = {k: v.cuda().contiguous() for k, v in extra.items()}
    if not delta:
        dev["log_decay"] = torch.cat([dev["log_decay"], torch.zeros(4, device="cuda")])
    for chunks in (True, False):
        memory = torch.full((seqs, H * dp * vp + 32), float("nan"), device="cuda")
        S = memory[:, :H * dp * vp].unflatten(1, (H, dp, vp))
        S.copy_(state if not fresh else torch.full_like(state, float("nan")))
        o = torch.full((seqs * T, H * vp), float("nan"), dtype=BF16, device="cuda")
        scratch = torch.empty(K.recurrence_scratch(seqs, T, H, delta), dtype=torch.uint8, device="cuda") if chunks else None
        put = as_tiles(act, seqs, H, G, dp, vp) if chunks else act.cuda()
        K.recurrence(put, [H, G, dp, vp], dev.get("norms"), dev.get("beta_g"), dev.get("log_decay"), S, lens, T, o, scratch)
        assert cases.row_errors(o, want).max() < 8e-3, chunks
        assert cases.row_errors(S.flatten(2), want_state.flatten(2)).max() < 2e-5, chunks
    kernels().check_status()


def test_state_is_kept_in_floats_over_many_chunks():
    """A state that neither decays nor is corrected: 2,000 tokens later its error is still a float's."""
    K = kernels()._S
    T, dp, vp = 2000, 64, 16
    act = randn(T, 2 * dp + vp, seed=3)
    act[:, 2 * dp:] = act[:, 2 * dp:].abs()
    act[:, dp:2 * dp] = act[:, dp:2 * dp].abs()
    log_decay = torch.zeros(1)
    _, want = recurrence_expected(act, 1, 1, 1, dp, vp, torch.zeros(1, 1, dp, vp), log_decay=log_decay)
    S = torch.empty(1, 1, dp, vp, device="cuda")
    o = torch.empty(T, vp, dtype=BF16, device="cuda")
    scratch = torch.empty(K.recurrence_scratch(1, T, 1, False), dtype=torch.uint8, device="cuda")
    K.recurrence(as_tiles(act, 1, 1, 1, dp, vp), [1, 1, dp, vp], None, None, log_decay.cuda(), S, torch.zeros(1, dtype=torch.int32, device="cuda"), T, o, scratch)
    assert ((S.cpu().double() - want).abs() / want.abs()).max() < 2e-5


@DTYPES
@pytest.mark.parametrize("n,np_", [(1, 8), (37, 40), (192, 192), (2500, 2504), (8192, 8192)])
def test_layer_norm_residual(n, np_, dtype):
    from nanochat_b200 import ops
    x, y, w1, w2 = torch.randn(5, np_), randn(5, np_, seed=3).float() + 30, torch.randn(np_), torch.randn(np_)
    for t in (x, y):
        t[:, n:] = 0
    for w in (w1, w2):
        w[n:] = 0
    y = y.to(dtype)
    want = x.double()[:, :n] + oracle.layer_norm(y.double()[:, :n], w1.double()[:n], 1e-3)
    got = x.cuda()
    h = ops.layer_norm_residual(got, y.cuda(), w1.cuda(), w2.cuda(), 1e-3, n, dtype)
    assert cases.row_errors(got[:, :n], want).max() < 3e-6                      # the residual stream is float in either precision
    assert (got[:, n:] == 0).all() and (h[:, n:] == 0).all()
    want_h = oracle.layer_norm(want, w2.double()[:n], 1e-3)
    assert (h[:, :n].cpu().double() - want_h).abs().max() < (1e-4 if dtype == F32 else 5e-2)
    table = randn(9, np_, seed=4, dtype=dtype)
    table[:, n:] = 0
    ids = torch.tensor([8, 0, 3, 3, 100])
    x2, _ = ops.embed_layer_norm(ids.cuda(), table.cuda(), 9, w1.cuda(), w2.cuda(), 1e-3, n)
    assert (x2[:, :n].cpu().double() - oracle.layer_norm(table[ids.clamp_max(8)].double()[:, :n], w1.double()[:n], 1e-3)).abs().max() < 1e-4


@DTYPES
@pytest.mark.parametrize("rows,ff,width", [(1, 24, 40), (8, 72, 96), (130, 8, 16), (300, 264, 200)])
def test_relu_glu(rows, ff, width, dtype):
    from nanochat_b200 import ops
    h, w = randn(rows, width, seed=1, dtype=dtype), randn(2 * ff, width, seed=2, dtype=dtype)
    want = torch.relu(h.double() @ w[:ff].double().t()) * (h.double() @ w[ff:].double().t())
    got = [ops.relu_glu(h.cuda(), w.cuda())]
    if dtype == BF16 and rows <= 8:
        got.append(torch.full((rows, ff), float("nan"), dtype=BF16, device="cuda"))
        kernels()._S.gemv_relu_glu(h.cuda(), w.cuda(), got[1])
    for g in got:
        assert cases.row_errors(g, want).max() < (1e-5 if dtype == F32 else 1e-2)


def test_a_token_without_a_page_is_reported_and_goes_nowhere():
    S = kernels()
    one = cases.window_mixer("cuda", BF16, cases.left(), 96)
    mix = one.model.layers[0].mix
    cache = one.model.make_cache(1, 64)
    cache.reserve(0, 64)
    cache.begin_rows()
    before = cache.pools[0].clone()
    for T in (1, 3):
        cache.cache_seqlens.fill_(64)             # the table has one page
        mix(torch.randn(T, 96, device="cuda").to(BF16), cache, 0, T)
        with pytest.raises(RuntimeError, match="code=6"):
            S.check_status()
        assert torch.equal(cache.pools[0], before)
    S.check_status()


@pytest.mark.parametrize("name", ["mixed", "wide", "heads"])
def test_fused_decode_step_matches_the_forward_pass(name):
    """The chained decode kernels against the general forward on the same cache contents, and its replay against itself."""
    from nanochat_b200.runtime import RecurrentDecodeGraph
    cfg = cases.CONFIGS[name]
    params = oracle.random_params(cfg, seed=12)
    model = cases.model_of(cfg, params, "cuda", BF16)
    engine = cases.Engine(model, None)
    cache = engine._pooled_cache(4, 50, 80)
    view = cache.begin_prompt(50)
    engine._prompt_logits(torch.tensor([cases.tokens_of(cfg, 50)], device="cuda"), view, [49])
    cache.fork(view)
    for step in range(5):
        ids = torch.tensor([[7 * r + step] for r in range(4)], device="cuda")
        kept = cache.memory.clone()
        want = model.forward(ids, kv_cache=cache)[:, 0]
        cache.cache_seqlens -= 1
        cache._pos -= 1
        cache.memory.copy_(kept)
        got = engine._decode_step(ids, cache)
        assert isinstance(engine._decode_graphs[id(cache)], RecurrentDecodeGraph) and engine._decode_graphs[id(cache)].fused
        cases.assert_close(got.cpu(), want.cpu(), BF16)
    assert engine._decode_graphs[id(cache)].graph is not None
    assert (cache.done == 0).all()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_replay_runner(tmp_path, dtype):
    from test_lupodra import write_folder
    cfg = cases.CONFIGS["wide"]
    params = oracle.random_params(cfg)
    write_folder(tmp_path / "m", cfg, params)
    tokens = cases.tokens_of(cfg, 40)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:31], "want": [30, 2]}], "end": []}]
    steps += [{"step": 1 + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(tokens[31:])]
    out = tmp_path / "out"
    out.mkdir()
    runner = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, runner, "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    want = oracle.forward(cases.double(params), cfg, tokens)
    got = [torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for i in range(10)]
    cases.assert_close(torch.cat(got), want[[30, 2, *range(31, 40)]], getattr(torch, dtype))
