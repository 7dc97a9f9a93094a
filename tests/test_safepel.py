"""The Safepel model on the CPU bodies: mechanisms, cuts of a prompt, batches, state and page reuse, the engine, loading,
replay."""

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import safepel_cases as cases
import safepel_oracle as oracle
from nanochat_b200 import ops
from nanochat_b200.engine import Engine, RecurrentCache
from nanochat_b200.models.registry import architectures, load_model_folder
from nanochat_b200.models.safepel import Safepel, SafepelConfig
from test_lupodra import write_folder

F32, BF16 = torch.float32, torch.bfloat16
CUTS = [[10 ** 6], [1], [2], [17, 2, 5, 1, 1, 30, 2]]


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_cut_of_a_prompt_gives_the_oracles_logits(name):
    cases.check_cuts(name, "cpu", F32, 60, CUTS)


def test_bf16_bodies():
    cases.check_cuts("mixed", "cpu", BF16, 40, [[10 ** 6], [13, 1]])


def test_residual_stream_after_every_layer():
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=2)
    tokens = cases.tokens_of(cfg, 20)
    want, got = [], []
    oracle.forward(cases.double(params), cfg, tokens, want)
    cases.model_of(cfg, params, "cpu", F32).forward(torch.tensor([tokens]), residuals=got)
    assert len(got) == len(want) == 4
    for a, b in zip(got, want):
        assert cases.row_errors(a, b).max() < 3e-5


# ------------------------------------------------------------------------------ the oracle's mechanisms

def test_oracle_rotation_against_complex_numbers():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    pos = torch.tensor([0, 1, 7, 100, 3000])
    y = oracle.rotate_pairs(x, pos, 50.0, 8)
    z = torch.view_as_complex(x[..., :8].reshape(5, 2, 4, 2).contiguous())
    turn = torch.exp(1j * pos[:, None, None].double() * 50.0 ** (-torch.arange(4).double() / 4))
    assert torch.allclose(torch.cat([torch.view_as_real(z * turn).reshape(5, 2, 8), x[..., 8:]], -1), y)


def test_oracle_convolution_against_conv1d():
    x, w = torch.randn(9, 6, dtype=torch.float64), torch.randn(6, 4, dtype=torch.float64)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(x.t()[None], (3, 0)), w[:, None], groups=6)[0].t()
    assert torch.allclose(oracle.short_conv(x, w), want)


def test_oracle_delta_rule_solves_for_the_last_key():
    """With step size one and no decay, reading with the key just written returns its value."""
    q = k = oracle.unit(torch.randn(12, 2, 8, dtype=torch.float64) * 100)
    v = torch.randn(12, 2, 5, dtype=torch.float64)
    one = torch.ones(12, 2, dtype=torch.float64)
    assert torch.allclose(oracle.delta_rule(q, k, v, one, one), v, atol=1e-6)


def test_oracle_layer_norm():
    x, w = torch.randn(3, 20, dtype=torch.float64), torch.randn(20, dtype=torch.float64)
    assert torch.allclose(oracle.layer_norm(x, w, 1e-3), torch.nn.functional.layer_norm(x, (20,), w, eps=1e-3))


# ------------------------------------------------------------------------------ mechanisms

@pytest.mark.parametrize("portions", [[10 ** 6], [1], [2], [7, 30, 1, 2]])
@pytest.mark.parametrize("spec", [dict(heads=4, kv_heads=2, dim=8, vdim=12, conv=4), dict(heads=2, kv_heads=2, dim=5, vdim=3, conv=1),
                                  dict(heads=3, kv_heads=1, dim=16, vdim=8, conv=7)])
def test_delta_rule(spec, portions):
    for strength in ({}, {"memory": True}, {"forget": True}, {"write": True, "memory": True}):
        cases.check_delta("cpu", F32, spec, 45, [portions], **strength)


@pytest.mark.parametrize("portions", [[10 ** 6], [1], [2], [7, 30, 1, 2]])
def test_decay_attention(portions):
    for spec in (cases.right((1.0, 0.3), 8, 12), cases.right((0.0, 0.999, 0.9), 5, 3)):
        cases.check_decay("cpu", F32, spec, 45, [portions])


@pytest.mark.parametrize("portions", [[10 ** 6], [1], [2], [7, 30, 1, 2]])
def test_window_edges(portions):
    m = cases.left(heads=4, kv_heads=2, dim=24, rot_dims=8, window=11, softcap=9.0)
    cases.check_window_edges("cpu", F32, m, 64, 90, [0, 3, 52, 63, 64], lambda key, w: [portions, [key + 1, 1], [key + w, 5]])


def test_soft_cap_and_scale_matter_and_agree():
    """Scores well above the cap: the capped softmax differs from the plain one, and the product follows the oracle."""
    one = cases.window_mixer("cpu", F32, cases.left(heads=2, kv_heads=1, dim=16, rot_dims=4, window=30, scale=2.0, softcap=3.0), 48)
    h = one.inputs(40)
    want = one.expected(h)
    plain = {**one.spec, "mixer": {**one.spec["mixer"], "left": {**one.spec["mixer"]["left"], "softcap": 1e6}}}
    assert cases.row_errors(one.expected(h, plain), want)[5:].median() > 0.05
    cases.assert_close(one.run(h, [11, 1]), want, F32)


def test_relu_glu():
    h, w = torch.randn(5, 16), torch.randn(24, 16)
    want = torch.relu(h.double() @ w[:12].double().t()) * (h.double() @ w[12:].double().t())
    assert cases.row_errors(ops.relu_glu(h, w), want).max() < 1e-5


def test_layer_norm_residual_ignores_padding():
    x, y, w1, w2 = torch.randn(4, 16), torch.randn(4, 16), torch.randn(16), torch.randn(16)
    for t in (x, y):
        t[:, 13:] = 0
    for w in (w1, w2):
        w[13:] = 0
    want = x.double()[:, :13] + oracle.layer_norm(y.double()[:, :13], w1.double()[:13], 1e-3)
    h = ops.layer_norm_residual(x, y, w1, w2, 1e-3, 13, F32)
    assert cases.row_errors(x[:, :13], want).max() < 1e-6 and (x[:, 13:] == 0).all() and (h[:, 13:] == 0).all()
    assert cases.row_errors(h[:, :13], oracle.layer_norm(want, w2.double()[:13], 1e-3)).max() < 1e-6


# ---------------------------------------------------------------------- cache, batch, engine

def test_pages_and_states_are_reused():
    cases.check_reuse("cpu", F32)


@pytest.mark.parametrize("rows", [1, 3])
def test_rows_of_a_batch_are_independent(rows):
    cases.check_rows("cpu", F32, rows)


def test_unequal_sequences_side_by_side():
    cases.check_unequal_sequences("cpu", F32)


@pytest.mark.parametrize("samples", [1, 3])
def test_greedy_generation(samples):
    cases.check_greedy("cpu", F32, samples)


def test_long_decoding():
    cfg = cases.config([(cases.delta(heads=2, kv_heads=1, dim=8, vdim=8), 24), (cases.parallel(cases.left(heads=2, kv_heads=1, dim=8, rot_dims=8, window=6),
                                                                                                cases.right((1.0, 0.99), 8, 8)), 24)], width=48)
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


def test_nested_generations_do_not_share_pages_or_states():
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


def test_recurrent_cache_forks_pages_and_states():
    cache = RecurrentCache(2, [16, 0], [{}, {"S": (2, 8, 4), "ring": (3, 40)}], 256, "cpu", F32, page_tokens=8)
    cache.reserve(19, 10)
    view = cache.begin_prompt(19)
    view.pools[0].view(-1, 16)[:19] = torch.arange(19.)[:, None]
    view.states[1]["S"].fill_(3.0)
    view.states[1]["ring"].copy_(torch.arange(120.).view(1, 3, 40))
    cache.states[1]["S"].fill_(-1.0)
    view.advance(19)
    cache.fork(view)
    for row in range(2):
        assert torch.equal(cache.gather_row(0, row)[:, 0], torch.arange(19.))
        assert (cache.states[1]["S"][row] == 3).all() and torch.equal(cache.states[1]["ring"][row].flatten(), torch.arange(120.))
    cache.states[1]["S"][0] = 7.0
    assert (cache.states[1]["S"][1] == 3).all()
    assert cache.states[1]["S"].stride(0) == cache.memory.shape[1] and cache.states[0] == {}


# -------------------------------------------------------------------- folder, registry, replay

def test_registry_and_folder(tmp_path):
    assert {"GPT", "Lupodra", "Safepel"} <= set(architectures())
    cfg = cases.CONFIGS["odd"]
    params = oracle.random_params(cfg)
    write_folder(tmp_path, cfg, params)
    model = load_model_folder(str(tmp_path), "cpu", dtype=F32)
    assert isinstance(model, Safepel)
    assert model.tensor_shapes() == oracle.tensor_shapes(cfg)
    tokens = cases.tokens_of(cfg, 9)
    cases.assert_close(model.forward(torch.tensor([tokens]))[0], oracle.forward(cases.double(params), cfg, tokens), F32)
    assert SafepelConfig.from_dict(model.config.to_dict()).layers == model.config.layers
    assert math.isfinite(Safepel(model.config, F32).init_weights("cpu").forward(torch.tensor([tokens])).sum())


def test_wrong_folders_are_refused(tmp_path):
    cfg = cases.CONFIGS["odd"]
    params = oracle.random_params(cfg)
    for name, change in (("missing", lambda p: p.pop("l0.mix.k.conv")), ("extra", lambda p: p.update({"l7.norm1": torch.zeros(3)})),
                         ("shape", lambda p: p.update({"l1.mix.right.v": torch.zeros(4, 4)}))):
        bad = dict(params)
        change(bad)
        write_folder(tmp_path / name, cfg, bad)
        with pytest.raises((KeyError, ValueError)):
            load_model_folder(str(tmp_path / name), "cpu", dtype=F32)
    layer = lambda kind, m, mlp=None: {"layers": [{"type": kind, "mixer": m, "mlp": mlp}]}
    p = cases.parallel()[1]
    for change in (layer("other", {}), layer(*cases.delta(heads=3, kv_heads=2)), layer(*cases.delta(conv=0)),
                   layer("parallel", {**p, "right": {**p["right"], "decay": [0.5]}}), layer("parallel", {**p, "left": {**p["left"], "vdim": 8}}),
                   layer("parallel", {**p, "left": cases.left(rot_dims=7)}), layer(*cases.delta(), {"kind": "sparse"})):
        with pytest.raises(ValueError):
            SafepelConfig.from_dict({**cfg, **change})


def test_command_line(tmp_path):
    """Greedy continuation of token ids through the chat command's model-folder path."""
    cfg = cases.CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=9)
    write_folder(tmp_path, cfg, params)
    prompt = cases.tokens_of(cfg, 12, 3)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "scripts.chat_cli", "--model-dir", str(tmp_path), "--token-ids", ",".join(map(str, prompt)), "--max-tokens", "4",
                        "-t", "0", "--device-type", "cpu"], cwd=root, capture_output=True, text=True, timeout=120, env={**os.environ, "NANOCHAT_DTYPE": "float32"})
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()[-4:]] == cases.greedy_expected(params, cfg, prompt, 4)


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
    wa, wb = (oracle.forward(cases.double(params), cfg, t) for t in (a, b))
    for name, want in (("0", wa[[3, 0]]), ("2", wa[[29]]), ("3", wb[[11]])):
        got = torch.from_numpy(np.fromfile(out / f"{name}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        cases.assert_close(got, want, F32)
