"""The Lupodra model on the serving kernels: every mechanism, cut, batch and edge against the float64 oracle, in float32
(sharp) and bf16 (the serving precision)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lupodra_cases as cases
import lupodra_oracle as oracle

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def randn(*shape, seed=0, dtype=BF16):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


@DTYPES
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_cut_of_a_prompt_gives_the_oracles_logits(name, dtype):
    cases.check_cuts(name, "cuda", dtype, 150, [[10 ** 6], [1], [2], [100, 1], [70, 2, 5, 1, 1, 30, 9]])


@DTYPES
@pytest.mark.parametrize("window,sizes", [(11, dict(dim=32, rot_dim=8, kv_rank=40)), (130, dict(dim=64, rot_dim=32, kv_rank=96, vdim=64)),
                                          (64, dict(dim=128, rot_dim=64, kv_rank=144, vdim=128)), (1, dict(dim=32, rot_dim=16, kv_rank=64))])
def test_window_edges(window, sizes, dtype):
    m = cases.mixer(heads=2, window=window, **sizes)
    T = window + 140
    keys = [k for k in (0, 1, 63, 64, 127, 128) if k + window < T]
    cases.check_window_edges("cuda", dtype, m, 160, T, keys,
                             lambda key, w: [[10 ** 6], [key + 1, 1], [max(key + w - 1, 1), 1, 2, 7], [key + w, 20, 1]])


@DTYPES
def test_far_and_first_keys(dtype):
    m = cases.mixer(heads=3, dim=64, rot_dim=16, kv_rank=96, window=None)
    for key in (0, 1, 64, 255):
        cases.check_far_and_first("cuda", dtype, m, 128, 700, key, [[10 ** 6], [600, 1], [33, 2, 500, 60]])


@DTYPES
def test_pages_are_reused(dtype):
    cases.check_reuse("cuda", dtype)


@DTYPES
@pytest.mark.parametrize("rows", [1, 2, 3, 5, 8, 9, 20])
def test_rows_of_a_batch_are_independent(rows, dtype):
    for name in ("all_experts", "wide", "mixed"):
        cases.check_rows("cuda", dtype, rows, name)


@DTYPES
@pytest.mark.parametrize("samples", [1, 3, 12])
def test_greedy_generation(samples, dtype):
    cases.check_greedy("cuda", dtype, samples)


@DTYPES
def test_long_decoding(dtype):
    cfg = cases.config([(cases.mixer(window=6), cases.dense(24))], width=48, loop={"start": 0, "stop": 1, "times": 2})
    params = oracle.random_params(cfg, seed=11)
    tokens = cases.tokens_of(cfg, 600)
    engine = cases.Engine(cases.model_of(cfg, params, "cuda", dtype), None)
    cases.assert_close(cases.feed(engine, tokens, [2, 1]), oracle.forward(cases.double(params), cfg, tokens), dtype)


# ------------------------------------------------------------------------------ mechanisms

@pytest.mark.parametrize("T,S", [(1, 1), (9, 9), (128, 128), (129, 300), (300, 300), (40, 1000)])
@pytest.mark.parametrize("H,D,D2,Dv", [(2, 64, 32, 64), (3, 128, 64, 128), (1, 8, 16, 8), (2, 40, 48, 72), (2, 72, 16, 40)])
def test_split_attention(T, S, H, D, D2, Dv):
    """The tensor-core prompt kernel on two-part keys, for full and partial 64-column boxes and windows around tile edges."""
    from nanochat_b200 import ops
    K = ops.serving_module()._S
    q, k = randn(T, H, D + D2, seed=1), randn(S, H, D, seed=2)
    k2, v = randn(S, D2, seed=3), randn(S, H, Dv, seed=4)
    scale = (D + D2) ** -0.5
    for window in (None, 1, 2, 64, 127, 128, 129, 200):
        dev = [t.cuda() for t in (q, k, k2, v)]
        o = torch.full((T, H, Dv), float("nan"), dtype=BF16, device="cuda")
        K.attention_split(dev[0][..., :D], dev[0][..., D:], dev[1], dev[2], dev[3], o, -1 if window is None else window - 1, scale)
        s = torch.einsum("thd,shd->hts", q[..., :D].double(), k.double()) + torch.einsum("thd,sd->hts", q[..., D:].double(), k2.double())
        gap = torch.arange(S - T, S)[:, None] - torch.arange(S)
        hidden = (gap < 0) | (gap >= (window or 10 ** 9))
        w = torch.softmax((s * scale).masked_fill(hidden, -float("inf")), -1)
        want = torch.einsum("hts,shd->thd", w, v.double())
        assert cases.row_errors(o, want).max() < 1.5e-2, (window, cases.row_errors(o, want).max())
    ops.serving_module().check_status()


@DTYPES
@pytest.mark.parametrize("rows", [1, 3, 40, 300])
@pytest.mark.parametrize("experts,top,ff,width", [(1, 1, 16, 64), (7, 1, 24, 40), (9, 4, 40, 96), (70, 6, 8, 32)])
def test_mixture(rows, experts, top, ff, width, dtype):
    from nanochat_b200 import ops
    cfg = cases.config([(cases.mixer(), cases.moe(experts=experts, top=top, ff=ff))], width=width)
    params = oracle.random_params(cfg, seed=1)
    model = cases.model_of(cfg, params, "cuda", dtype)
    h = randn(rows, width, seed=5)
    y, *chosen = ops.mixture(h.to(dtype).cuda(), model.layers[0].mlp)
    if chosen:
        slot, wt = chosen
        y = (y[slot.long()].double() * wt[..., None]).sum(1)
    want = oracle.mixture_ff(h.double(), oracle.under(cases.double(params), "l0.mlp."), cfg["layers"][0]["mlp"])
    cases.assert_close(y, want, dtype)


def test_routing_prefers_the_lower_index_among_equals():
    from nanochat_b200 import ops
    K = ops.serving_module()._S
    logits = torch.tensor([[1.0, 3.0, 3.0, 2.0, 3.0, 0.0, 0.0, 0.0], [0.0] * 8, [-5.0, -1.0, -2.0, -1.0, -9.0, -1.0, -3.0, -4.0]], device="cuda")
    idx, wt = torch.empty(3, 3, dtype=torch.int32, device="cuda"), torch.empty(3, 3, device="cuda")
    K.route_topk(logits, 6, idx, wt)
    assert idx.tolist() == [[1, 2, 4], [0, 1, 2], [1, 3, 5]]
    assert torch.allclose(wt, torch.full((3, 3), 1 / 3, device="cuda"))


@DTYPES
@pytest.mark.parametrize("n,np_", [(1, 8), (37, 40), (96, 96), (4096, 4096)])
def test_poly_norm(n, np_, dtype):
    from nanochat_b200 import ops
    z = torch.zeros(5, np_)
    z[:, :n] = randn(5, n, seed=7)
    coef = torch.tensor([0.5, -0.3, 0.2, 0.1])
    got = ops.poly_norm(z.to(dtype).cuda(), coef.cuda(), 1e-4, n).cpu()
    want = oracle.poly_norm(z[:, :n].double(), coef.double(), 1e-4)
    assert cases.row_errors(got[:, :n], want).max() < (1e-6 if dtype == F32 else 4e-3)
    assert (got[:, n:] == 0).all()


@DTYPES
def test_gated_residual_norm(dtype):
    from nanochat_b200 import ops
    n, np_ = 61, 64
    x, extra = torch.randn(6, np_), torch.randn(6, np_)
    x[:, n:], extra[:, n:] = 0, 0
    bias, w = torch.randn(np_), torch.randn(np_)
    gate, y, rows = (randn(k, np_, seed=s) for k, s in ((6, 1), (6, 2), (11, 3)))
    for t in (gate, y, rows):
        t[:, n:] = 0
    slot = torch.randint(0, 11, (6, 3), dtype=torch.int32)
    wt = torch.rand(6, 3)
    g = torch.sigmoid(gate.double() + bias.double())
    want = x.double() + 0.7 * g * (y.double() + (rows.double()[slot.long()] * wt[..., None].double()).sum(1)) + extra.double()
    got, d = x.cuda(), lambda t: t.to(dtype).cuda()
    h = ops.gated_residual_norm(got, [(d(gate), bias.cuda(), d(y)), (d(gate), bias.cuda(), d(rows), slot.cuda(), wt.cuda())], 0.7, extra.cuda(),
                                w.cuda(), 1e-3, n, dtype)
    assert cases.row_errors(got[:, :n], want[:, :n]).max() < 1e-6          # the residual stream is float in either precision
    assert cases.row_errors(h[:, :n], oracle.plain_norm(want[:, :n], w[:n].double(), 1e-3)).max() < (1e-6 if dtype == F32 else 4e-3)


def test_a_token_without_a_page_is_reported_and_goes_nowhere():
    """The append finds no room in the page table: nothing is written and the status word says so."""
    from nanochat_b200 import ops
    S = ops.serving_module()
    one = cases.OneMixer(cases.mixer(), 96, "cuda", BF16)
    cache = one.model.make_cache(1, 64)
    cache.reserve(0, 64)
    cache.begin_rows()
    before = cache.pools[0].clone()
    cache.cache_seqlens.fill_(64)                 # the table has one page
    z = ops.linear_rows(torch.randn(1, 96, device="cuda").to(BF16), one.model.layers[0].w_in)
    a = one.model.layers[0].attn
    S._S.latent_post(z, a.q_rank, a.q_norm, None, a.c_off, a.kv_rank, a.kvp, a.kv_norm, a.eps, a.rot_off, a.rot_dim, a.freq, cache.pools[0],
                     cache.table, cache.cache_seqlens, 1, None)
    with pytest.raises(RuntimeError, match="code=6"):
        S.check_status()
    assert torch.equal(cache.pools[0], before)
    S.check_status()


def test_fused_decode_step_matches_the_forward_pass():
    """The chained decode kernels against the general forward on the same cache contents, and its replay against itself."""
    from nanochat_b200.runtime import LatentDecodeGraph
    cfg = cases.CONFIGS["all_experts"]
    params = oracle.random_params(cfg, seed=12)
    model = cases.model_of(cfg, params, "cuda", BF16)
    engine = cases.Engine(model, None)
    cache = engine._pooled_cache(4, 50, 80)
    view = cache.begin_prompt(50)
    engine._prompt_logits(torch.tensor([cases.tokens_of(cfg, 50)], device="cuda"), view, [49])
    cache.fork(view)
    for step in range(5):
        ids = torch.tensor([[7 * r + step] for r in range(4)], device="cuda")
        want = model.forward(ids, kv_cache=cache)[:, 0]
        cache.cache_seqlens -= 1
        cache._pos -= 1
        got = engine._decode_step(ids, cache)
        assert isinstance(engine._decode_graphs[id(cache)], LatentDecodeGraph) and engine._decode_graphs[id(cache)].fused
        cases.assert_close(got.cpu(), want.cpu(), BF16)
    assert engine._decode_graphs[id(cache)].graph is not None


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
