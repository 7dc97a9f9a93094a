"""The Lupodra model on the CPU bodies: mechanisms, cuts of a prompt, batches, page reuse, the engine, loading, replay."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lupodra_cases as cases
import lupodra_oracle as oracle
from nanochat_b200 import ops
from nanochat_b200.engine import Engine, PagedLatentCache
from nanochat_b200.models.lupodra import Lupodra, LupodraConfig
from nanochat_b200.models.registry import architectures, get_architecture, load_model_folder
from nanochat_b200.utils.safetensors import SafetensorsError, read_safetensors, write_safetensors

F32, BF16 = torch.float32, torch.bfloat16
CUTS = [[10 ** 6], [1], [2], [17, 2, 5, 1, 1, 30, 2]]


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_cut_of_a_prompt_gives_the_oracles_logits(name):
    cases.check_cuts(name, "cpu", F32, 75, CUTS)


def test_bf16_bodies():
    cases.check_cuts("wide", "cpu", BF16, 40, [[10 ** 6], [13, 1]])


def test_residual_stream_after_every_layer_run():
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=2)
    tokens = cases.tokens_of(cfg, 20)
    want, got = [], []
    oracle.forward(cases.double(params), cfg, tokens, want)
    cases.model_of(cfg, params, "cpu", F32).forward(torch.tensor([tokens]), residuals=got)
    assert len(got) == len(want) == 1 + 2 * 3 + 1
    for a, b in zip(got, want):
        assert cases.row_errors(a, b).max() < 2e-5


def test_oracle_order_of_a_loop():
    cfg = {"layers": [{}] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert oracle.run_order(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    mine = LupodraConfig.from_dict(cases.CONFIGS["mixed"]).runs()
    assert mine == oracle.run_order(cases.CONFIGS["mixed"])


# ------------------------------------------------------------------------------ mechanisms

def test_oracle_rotation_against_complex_numbers():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    pos = torch.tensor([0, 1, 7, 100, 3000])
    y = oracle.rotate_half(x, pos, 50.0, 8)
    z = torch.complex(x[..., :4], x[..., 4:8])
    turn = torch.exp(1j * pos[:, None, None].double() * 50.0 ** (-torch.arange(4).double() / 4))
    assert torch.allclose(torch.cat([(z * turn).real, (z * turn).imag, x[..., 8:]], -1), y)


def test_poly_norm():
    z = torch.randn(6, 40)
    z[:, 37:] = 0
    coef = torch.tensor([0.5, -0.3, 0.2, 0.1])
    got = ops.poly_norm(z, coef, 1e-4, 37)
    assert torch.allclose(got[:, :37].double(), oracle.poly_norm(z[:, :37].double(), coef.double(), 1e-4), atol=1e-5)
    assert (got[:, 37:] == 0).all()


def test_gated_residual_norm_with_expert_rows():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g)
    x, w, bias, gate = r(4, 16), r(16), r(16), r(4, 16)
    rows, slot, wt = r(9, 16), torch.tensor([[3, 1], [8, 0], [2, 2], [5, 7]]), torch.rand(4, 2, generator=g)
    extra = r(4, 16)
    want = x + 0.5 * (torch.sigmoid(gate + bias) * (rows[slot] * wt[..., None]).sum(1) + torch.sigmoid(-gate) * 2.0) + extra
    got = x.clone()
    h = ops.gated_residual_norm(got, [(gate, bias, rows, slot.int(), wt), (-gate, torch.zeros(16), torch.full((4, 16), 2.0))], 0.5, extra, w,
                                1e-3, 16, F32)
    assert torch.allclose(got, want, atol=1e-6)
    assert torch.allclose(h, oracle.plain_norm(want, w, 1e-3), atol=1e-5)


@pytest.mark.parametrize("top", [1, 2, 5])
def test_mixture(top):
    cfg = cases.config([(cases.mixer(), cases.moe(experts=5, top=top, ff=12))], width=40)
    params = oracle.random_params(cfg, seed=1)
    model = cases.model_of(cfg, params, "cpu", F32)
    h = torch.randn(7, 40)
    (got,) = ops.mixture(h, model.layers[0].mlp)
    want = oracle.mixture_ff(h.double(), oracle.under(cases.double(params), "l0.mlp."), cfg["layers"][0]["mlp"])
    assert cases.row_errors(got, want).max() < 1e-5


@pytest.mark.parametrize("portions", [[10 ** 6], [1], [2], [7, 30, 1, 2]])
def test_window_edges(portions):
    m = cases.mixer(heads=2, dim=32, rot_dim=8, kv_rank=40, window=11)
    cases.check_window_edges("cpu", F32, m, 64, 90, [0, 3, 52, 63, 64], lambda key, w: [portions, [key + 1, 1], [key + w, 5]])


def test_far_and_first_keys():
    m = cases.mixer(heads=2, dim=32, rot_dim=8, kv_rank=40, window=None)
    for key in (0, 5, 64):
        cases.check_far_and_first("cpu", F32, m, 64, 200, key, [[10 ** 6], [150, 1], [3, 60]])


# ---------------------------------------------------------------------- cache, batch, engine

def test_pages_are_reused():
    cases.check_reuse("cpu", F32)


@pytest.mark.parametrize("rows", [1, 3])
def test_rows_of_a_batch_are_independent(rows):
    cases.check_rows("cpu", F32, rows)


@pytest.mark.parametrize("samples", [1, 3])
def test_greedy_generation(samples):
    cases.check_greedy("cpu", F32, samples)


def test_long_decoding():
    cfg = cases.config([(cases.mixer(window=6), cases.dense(24))], width=48, loop={"start": 0, "stop": 1, "times": 2})
    params = oracle.random_params(cfg, seed=11)
    tokens = cases.tokens_of(cfg, 300)
    engine = Engine(cases.model_of(cfg, params, "cpu", F32), None)
    cases.assert_close(cases.feed(engine, tokens, [2, 1]), oracle.forward(cases.double(params), cfg, tokens), F32)


def test_sampled_rows_are_reproducible_and_end_at_the_limit():
    cfg = cases.CONFIGS["mixed"]
    engine = Engine(cases.model_of(cfg, oracle.random_params(cfg), "cpu", F32), None)
    prompt = cases.tokens_of(cfg, 10)
    runs = [engine.generate_batch(prompt, num_samples=2, max_tokens=6, temperature=0.8, top_k=20, seed=5)[0] for _ in range(2)]
    assert runs[0] == runs[1] and all(len(r) == 16 for r in runs[0])


def test_nested_generations_do_not_share_pages():
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=9)
    engine = Engine(cases.model_of(cfg, params, "cpu", F32), None)
    a, b = cases.tokens_of(cfg, 20, 1), cases.tokens_of(cfg, 30, 2)
    ga, gb = (engine.generate(t, max_tokens=5, temperature=0.0) for t in (a, b))
    got = [(next(ga)[0][0], next(gb)[0][0]) for _ in range(5)]
    assert [x for x, _ in got] == cases.greedy_expected(params, cfg, a, 5)
    assert [y for _, y in got] == cases.greedy_expected(params, cfg, b, 5)


def test_a_full_sequence_is_refused():
    cfg = cases.CONFIGS["mixed"]
    engine = Engine(cases.model_of(cfg, oracle.random_params(cfg), "cpu", F32), None)
    seq = engine.open_sequence(10)
    seq.extend(cases.tokens_of(cfg, 10))
    with pytest.raises(ValueError):
        seq.extend([1])
    seq.close()
    with pytest.raises(ValueError):
        next(engine.generate([1, 2], max_tokens=4000))


def test_latent_cache_fork_shares_full_pages_and_copies_the_rest():
    cache = PagedLatentCache(2, [16, 32], 256, "cpu", F32, page_tokens=8)
    cache.reserve(19, 10)
    view = cache.begin_prompt(19)
    for run, pool in enumerate(view.pools):
        flat = pool.view(-1, pool.shape[2])
        flat[:19] = torch.arange(19.)[:, None] + 100 * run
    view.advance(19)
    cache.fork(view)
    assert cache.get_pos() == 19 and (cache.table[0, :2] == cache.table[1, :2]).all() and cache.table[0, 2] != cache.table[1, 2]
    for run in range(2):
        for row in range(2):
            assert torch.equal(cache.gather_row(run, row)[:, 0], torch.arange(19.) + 100 * run)
    assert cache.row_capacity() == 16 + 8 * cache.private_pages


# -------------------------------------------------------------------- folder, registry, replay

def write_folder(path, cfg, params):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.to(BF16) for k, v in params.items()})


def test_safetensors_round_trip_and_errors(tmp_path):
    t = {"a": torch.randn(3, 4).to(BF16), "b": torch.arange(5, dtype=torch.int32), "c": torch.randn(2), "s": torch.tensor(1.5)}
    path = str(tmp_path / "x.safetensors")
    write_safetensors(path, t)
    got = read_safetensors(path)
    assert all(torch.equal(got[k], t[k]) and got[k].dtype == t[k].dtype for k in t)
    data = open(path, "rb").read()
    open(path, "wb").write(data[:-4])
    with pytest.raises(SafetensorsError):
        read_safetensors(path)
    open(path, "wb").write(data[:4])
    with pytest.raises(SafetensorsError):
        read_safetensors(path)


def test_registry_and_folder(tmp_path):
    assert {"GPT", "Lupodra"} <= set(architectures())
    with pytest.raises(ValueError):
        get_architecture("Nothing")
    cfg = cases.CONFIGS["odd"]
    params = oracle.random_params(cfg)
    write_folder(tmp_path, cfg, params)
    model = load_model_folder(str(tmp_path), "cpu", dtype=F32)
    assert isinstance(model, Lupodra)
    tokens = cases.tokens_of(cfg, 9)
    cases.assert_close(model.forward(torch.tensor([tokens]))[0], oracle.forward(cases.double(params), cfg, tokens), F32)
    again = LupodraConfig.from_dict(model.config.to_dict())
    assert again.layers == model.config.layers and again.loop == model.config.loop


def test_gpt_folder(tmp_path):
    from nanochat_b200.models.gpt import GPT, GPTConfig
    kw = dict(sequence_len=32, vocab_size=64, n_layer=2, n_head=2, n_kv_head=2, n_embd=32)
    torch.manual_seed(0)
    gpt = GPT(GPTConfig(**kw))
    gpt.init_weights()
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "GPT", **kw}))
    write_safetensors(str(tmp_path / "model.safetensors"), gpt.state_dict())
    model = load_model_folder(str(tmp_path), "cpu")
    ids = torch.tensor([[3, 5, 9, 2]])
    assert torch.allclose(model(ids), gpt(ids))
    seq = Engine(model, None).open_sequence(8)
    first = seq.extend([3, 5], [1])
    rest = seq.extend([9, 2], [0, 1])
    assert torch.allclose(torch.cat([first, rest]), gpt(ids)[0, 1:], atol=1e-4)


def test_wrong_folders_are_refused(tmp_path):
    cfg = cases.CONFIGS["odd"]
    params = oracle.random_params(cfg)
    for name, change in (("missing", lambda p: p.pop("l0.mix.uk")), ("extra", lambda p: p.update({"l7.norm1": torch.zeros(3)})),
                         ("shape", lambda p: p.update({"l0.mix.uv": torch.zeros(4, 4)}))):
        bad = dict(params)
        change(bad)
        write_folder(tmp_path / name, cfg, bad)
        with pytest.raises((KeyError, ValueError)):
            load_model_folder(str(tmp_path / name), "cpu", dtype=F32)
    for change in ({"loop": {"start": 1, "stop": 1, "times": 2}}, {"loop": {"start": 0, "stop": 3, "times": 2}},
                   {"layers": [dict(cfg["layers"][0], type="other")]}):
        with pytest.raises(ValueError):
            LupodraConfig.from_dict({**cfg, **change})


def test_replay_runner(tmp_path):
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg)
    write_folder(tmp_path / "m", cfg, params)
    a, b = cases.tokens_of(cfg, 30, 1), cases.tokens_of(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [3, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:29], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[29:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [11]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    runner = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, runner, "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(out), "--max-tokens", "32",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
    wa, wb = (oracle.forward(cases.double(params), cfg, t) for t in (a, b))
    for name, want in (("0", wa[[3, 0]]), ("2", wa[[29]]), ("3", wb[[11]])):
        got = torch.from_numpy(np.fromfile(out / f"{name}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        cases.assert_close(got, want, F32)
