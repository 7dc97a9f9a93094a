"""
Configurations, inputs and checks shared by the CPU and GPU tests of the Safepel model. Expected values come from
`safepel_oracle` in float64.
"""

import torch

import safepel_oracle as oracle
from lupodra_cases import double, feed, row_errors, tokens_of
from nanochat_b200.engine import Engine
from nanochat_b200.models.safepel import Safepel, SafepelConfig

F32, BF16 = torch.float32, torch.bfloat16
# relative RMS error of a row of logits, and of a mixer's output, against the oracle: the largest (a norm over a few small
# entries can blow bf16 rounding up); the median is held to a fifth
TOL = {F32: 5e-5, BF16: 0.12}
MIXER_TOL = {F32: 5e-5, BF16: 0.06}


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=3):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def left(heads=6, kv_heads=2, dim=32, window=9, base=1000.0, rot_dims=16, scale=0.3, softcap=8.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": base, "dims": rot_dims}, "softcap": softcap,
         "mask": {"size": window}}
    return m


def right(decay=(0.5, 0.9, 1.0), dim=16, vdim=24):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(a=None, b=None, left_scale=0.7, right_scale=0.4):
    return "parallel", {"left": a or left(), "right": b or right(), "left_scale": left_scale, "right_scale": right_scale}


def config(layers, width=96, vocab=130, eps=1e-5, logit_scale=0.8):
    return {"architecture": "Safepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{"type": kind, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (kind, m), ff in layers]}


CONFIGS = {
    # every layer another shape, two without a feed-forward; a decay that forgets nothing
    "mixed": config([(delta(), 72), (parallel(), None), (delta(heads=2, dim=16, vdim=8, conv=1), None),
                     (parallel(left(heads=3, kv_heads=1, dim=16, rot_dims=16, window=20, softcap=30.0), right((0.97, 0.8), 24, 8), -0.5, 1.3), 40)]),
    # sizes that are multiples of nothing, more taps than a short portion has tokens, a decay that forgets everything
    "odd": config([(delta(heads=3, kv_heads=1, dim=13, vdim=11, conv=5), 37),
                   (parallel(left(heads=5, kv_heads=5, dim=11, window=7, rot_dims=6, softcap=2.0), right((0.0, 0.97), 9, 5)), 53)],
                  width=61, vocab=103, eps=1e-3, logit_scale=1.7),
    # more query heads on a key head than one tile holds, windows beyond one key tile, many value heads on one key
    "heads": config([(parallel(left(heads=34, kv_heads=2, dim=16, rot_dims=8, window=150, softcap=5.0), right((0.99,) * 5, 8, 16)), 96),
                     (delta(heads=6, kv_heads=1, dim=32, vdim=16, conv=2), 24)], width=160, vocab=200),
    # the largest heads the chunk kernels and the tensor-core prompt attention take
    "wide": config([(delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=4), 128),
                    (parallel(left(heads=2, kv_heads=1, dim=128, rot_dims=64, window=100, scale=0.09, softcap=20.0), right((0.9, 0.999), 128, 96)), 200)], width=128),
    # one of everything; a window of one token
    "single": config([(delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=4), 8),
                      (parallel(left(heads=1, kv_heads=1, dim=8, rot_dims=2, window=1), right((0.7,), 8, 8), 1.0, 1.0), 8)], width=16, vocab=17, logit_scale=1.0),
    # beyond what the tensor-core prompt kernels take, then beyond what the step kernels take
    "huge": config([(delta(heads=2, kv_heads=2, dim=136, vdim=264, conv=3), 64),
                    (parallel(left(heads=2, kv_heads=1, dim=144, window=40, rot_dims=144, scale=0.08), right((0.95, 0.6), 160, 72)), 48),
                    (parallel(left(heads=1, kv_heads=1, dim=264, window=70, rot_dims=20, scale=0.06), right((0.9,), 264, 520)), None)], width=104),
}


def model_of(cfg, params, device, dtype):
    return Safepel(SafepelConfig.from_dict(cfg, sequence_len=2048), dtype).load_tensors({k: v.to(BF16) for k, v in params.items()}, device)


def assert_close(got, want, dtype, tol=TOL):
    err = row_errors(got, want).flatten()
    assert err.max() < tol[dtype] and err.median() < tol[dtype] / 5, (err.max(), err.argmax(), err.median())


# -------------------------------------------------------------------------------- model

def check_cuts(name, device, dtype, n, cuts):
    """One prompt, cut in several ways, against the oracle."""
    cfg = CONFIGS[name]
    params = oracle.random_params(cfg, seed=3, sharp=1.5)
    tokens = tokens_of(cfg, n)
    want = oracle.forward(double(params), cfg, tokens)
    engine = Engine(model_of(cfg, params, device, dtype), None)
    for portions in cuts:
        assert_close(feed(engine, tokens, portions), want, dtype)
    engine.check()


def check_reuse(device, dtype):
    """Pages and state rows given back and used again, with whatever was left in them."""
    cfg = CONFIGS["heads"]
    params = oracle.random_params(cfg, seed=4)
    engine = Engine(model_of(cfg, params, device, dtype), None)
    long, short = tokens_of(cfg, 150, 5), tokens_of(cfg, 70, 6)
    first = {len(t): feed(engine, t, p, 200) for t, p in ((long, [90, 30, 1]), (short, [40, 1]))}
    cache = engine._cache_pool[1]
    for pool in cache.pools:
        pool.fill_(float("nan"))                # every page is rewritten before it is read, every state starts from zeros
    cache.memory.fill_(float("nan"))
    for t, p in ((short, [40, 1]), (long, [90, 30, 1]), (short, [40, 1])):
        again = feed(engine, t, p, 200)
        assert torch.equal(again, first[len(t)]) or row_errors(again, first[len(t)]).max() < TOL[dtype] / 4
    assert engine._cache_pool[1] is cache


def check_rows(device, dtype, rows, name="mixed"):
    """Rows of one batch that go different ways after a common prompt, each against the oracle and against itself alone."""
    cfg = CONFIGS[name]
    params = oracle.random_params(cfg, seed=7, sharp=1.5)
    model = model_of(cfg, params, device, dtype)
    engine = Engine(model, None)
    prompt, steps = tokens_of(cfg, 61, 8), 9                  # crosses a page border while decoding
    own = [tokens_of(cfg, steps, 100 + r) for r in range(rows)]
    cache = engine._pooled_cache(rows, len(prompt), len(prompt) + steps)
    view = cache.begin_prompt(len(prompt))
    engine._prompt_logits(torch.tensor([prompt], device=device), view, [len(prompt) - 1])
    cache.fork(view)
    engine._begin_decode(cache)
    got = torch.stack([engine._decode_step(torch.tensor([[own[r][s]] for r in range(rows)], device=device), cache).float().cpu().clone()
                       for s in range(steps)], 1)
    engine.check()
    want = torch.stack([oracle.forward(double(params), cfg, prompt + t)[len(prompt):] for t in own])
    assert_close(got, want, dtype)
    assert_close(got[-1], feed(Engine(model, None), prompt + own[-1], [len(prompt), 1])[len(prompt):], dtype)


def check_unequal_sequences(device, dtype, lengths=(3, 70, 129, 20)):
    """Sequences of different lengths decoded side by side in one batch (the rows' caches filled one by one), each against the
    oracle alone."""
    cfg = CONFIGS["mixed"]
    params = oracle.random_params(cfg, seed=13, sharp=1.5)
    model = model_of(cfg, params, device, dtype)
    rows, steps = len(lengths), 6
    tokens = [tokens_of(cfg, n + steps, 50 + r) for r, n in enumerate(lengths)]
    cache = model.make_cache(rows, max(lengths) + steps)
    cache.reserve(0, max(lengths) + steps)
    cache.begin_rows()
    for r, n in enumerate(lengths):
        one = RowView(cache, r)
        model.forward(torch.tensor([tokens[r][:n]], device=device), kv_cache=one, want=[])
    cache.cache_seqlens.copy_(torch.tensor(lengths, dtype=torch.int32))
    for s in range(steps):
        ids = torch.tensor([[tokens[r][n + s]] for r, n in enumerate(lengths)], device=device)
        got = model.forward(ids, kv_cache=cache)[:, 0]
        want = torch.stack([oracle.forward(double(params), cfg, tokens[r][:n + s + 1])[-1] for r, n in enumerate(lengths)])
        assert_close(got, want, dtype)


class RowView:
    """One row of a cache as a batch-1 cache."""

    def __init__(self, cache, row):
        self.pools, self.table, self.max_seq_len = cache.pools, cache.table[row:row + 1].contiguous(), cache.max_seq_len
        self.states = [{k: t[row:row + 1] for k, t in s.items()} for s in cache.states]
        self.done = torch.zeros(1, dtype=torch.int32, device=cache.device)
        self.cache_seqlens, self._pos = torch.zeros(1, dtype=torch.int32, device=cache.device), 0

    def get_pos(self):
        return self._pos

    def advance(self, n):
        self.cache_seqlens += n
        self._pos += n


def greedy_expected(params, cfg, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(oracle.forward(double(params), cfg, tokens)[-1].argmax()))
    return tokens[len(prompt):]


def check_greedy(device, dtype, samples=1):
    cfg = CONFIGS["mixed"] if dtype == F32 else CONFIGS["wide"]
    params = oracle.random_params(cfg, seed=9)
    prompt = tokens_of(cfg, 57, 10)
    want = greedy_expected(params, cfg, prompt, 10)
    model = model_of(cfg, params, device, dtype)
    got = list(Engine(model, None).generate(prompt, num_samples=samples, max_tokens=10, temperature=0.0))
    assert [c for c, _ in got] == [[t] * samples for t in want]
    assert list(model.generate(prompt, 10, temperature=0.0)) == want


# ----------------------------------------------------------------------------- one mixer

class OneMixer:
    """A single mixer on given inputs h, run through the product's operations over its cache."""

    def __init__(self, spec, width, device, dtype, seed=0, change=None):
        self.cfg = config([(spec, None)], width=width)
        self.params = oracle.random_params(self.cfg, seed=seed)
        if change:
            change(self.params)
            self.params = {k: v.to(BF16).float() for k, v in self.params.items()}
        self.mix = oracle.under(double(self.params), "l0.mix.")
        self.model = model_of(self.cfg, self.params, device, dtype)
        self.device, self.dtype, self.spec, self.eps = device, dtype, self.cfg["layers"][0], self.cfg["norm"]["eps"]

    def inputs(self, T, seed=2):
        return torch.randn(T, self.cfg["width"], generator=torch.Generator().manual_seed(seed)).to(BF16).double()

    def expected(self, h, spec=None):
        return oracle.mix(h.double(), self.mix, spec or self.spec, self.eps)

    def run(self, h, portions):
        cache = self.model.make_cache(1, h.shape[0])
        cache.reserve(0, h.shape[0])
        cache.begin_rows()
        cache.memory.fill_(float("nan"))
        full = torch.zeros(h.shape[0], self.model.width)
        full[:, :h.shape[1]] = h
        full = full.to(self.dtype).to(self.device)
        out, at, k = [], 0, 0
        while at < h.shape[0]:
            n = min(portions[min(k, len(portions) - 1)], h.shape[0] - at)
            out.append(self.model.layers[0].mix(full[at:at + n], cache, 0, n)[:, :h.shape[1]].float().cpu())
            cache.advance(n)
            at, k = at + n, k + 1
        return torch.cat(out)


def check_delta(device, dtype, spec, T, portions, **strength):
    """The delta rule alone; `memory`: decays so slow that the first tokens still count at the end."""
    def change(p):
        if strength.get("memory"):
            p["l0.mix.A_log"].fill_(-9.0)
        if strength.get("forget"):                       # decays down to e^-60 a token next to ones near 1
            p["l0.mix.A_log"].copy_(torch.linspace(-6.0, 2.0, p["l0.mix.A_log"].numel()))
            p["l0.mix.dt_bias"].fill_(8.0)
        if strength.get("write"):                        # full step sizes
            p["l0.mix.b"].mul_(6.0)
    one = OneMixer(("delta", spec), 48, device, dtype, change=change)
    h = one.inputs(T)
    if strength.get("memory"):
        h[:6] *= 8.0
    want = one.expected(h)
    if strength.get("memory"):
        other = h.clone()
        other[:6] = 8.0 * one.inputs(6, seed=9)
        assert row_errors(one.expected(other), want)[-1] > 3 * MIXER_TOL[dtype]
    for p in portions:
        assert_close(one.run(h, p), want, dtype, tol=MIXER_TOL)


def check_decay(device, dtype, spec, T, portions):
    """Fixed-decay attention alone (the other side's factor is zero); the first token still counts at the end where a decay is one."""
    one = OneMixer(parallel(left(heads=1, kv_heads=1, dim=8, rot_dims=2), spec, 0.0, 0.9), 48, device, dtype)
    h = one.inputs(T)
    want = one.expected(h)
    if 1.0 in spec["decay"]:
        other = h.clone()
        other[:8] = 4.0 * one.inputs(8, seed=9)
        assert row_errors(one.expected(other), want)[-1] > 3 * MIXER_TOL[dtype]
    for p in portions:
        assert_close(one.run(h, p), want, dtype, tol=MIXER_TOL)


def standout(one, T, key, queries, seed=2):
    """Inputs in which the key of token `key` dominates head 0's scores of the tokens `queries`: the unrotated parts of both
    point the same way."""
    m, p = one.spec["mixer"]["left"], one.mix
    g = torch.Generator().manual_seed(seed)
    h = torch.randn(T, one.cfg["width"], generator=g).double()
    a = torch.randn(one.cfg["width"], generator=g).double()
    target = (p["left.q"] @ a)[:m["dim"]]
    target[:m["rot"]["dims"]] = 0
    b = torch.linalg.pinv(p["left.k"][:m["dim"]]) @ target
    h[queries] = a
    h[key] = b / b.norm() * a.norm()
    return h.to(BF16).double()


def window_mixer(device, dtype, m, width, out_scale=0.8):
    return OneMixer(parallel(m, right((0.5,), 8, 8), out_scale, 0.0), width, device, dtype)


def with_window(one, window):
    spec = {**one.spec, "mixer": {**one.spec["mixer"], "left": {**one.spec["mixer"]["left"], "mask": {"size": window}}}}
    return spec


def check_window_edges(device, dtype, m, width, T, keys, portions):
    """A key that stands out, asked for at the last place that sees it and at the first that does not."""
    one, w = window_mixer(device, dtype, m, width), m["mask"]["size"]
    for key in keys:
        inside, outside = key + w - 1, key + w
        h = standout(one, T, key, [i for i in {key + 1, inside, outside} if key < i < T])
        want = one.expected(h)
        # the inputs do show a window that is one key too small or too large
        for other, at in ((w + 1, outside), (w - 1, inside)):
            if key < at < T and other > 0:
                assert row_errors(one.expected(h, with_window(one, other)), want)[at] > 3 * MIXER_TOL[dtype]
        for p in portions(key, w):
            assert_close(one.run(h, p), want, dtype, tol=MIXER_TOL)
