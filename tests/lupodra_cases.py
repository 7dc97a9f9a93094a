"""
Configurations, inputs and checks shared by the CPU and GPU tests of the Lupodra model. Expected values come from
`lupodra_oracle` in float64.
"""

import torch

import lupodra_oracle as oracle
from nanochat_b200.engine import Engine
from nanochat_b200.models.lupodra import Lupodra, LupodraConfig

# relative RMS error of a row of logits, and of a mixer's output for scores that stand out, against the oracle
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
MIXER_TOL = {torch.float32: 2e-5, torch.bfloat16: 4e-2}


def mixer(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=40, window=9, base=1000.0, rot_dims=None, scale=0.2):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dims or rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=96, vocab=130, loop=None, eps=1e-5, mult=0.6):
    return {"architecture": "Lupodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "loop": loop,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


CONFIGS = {
    # every layer another shape, one without a feed-forward, a loop in the middle
    "mixed": config([(mixer(), dense()), (mixer(heads=2, dim=32, vdim=16, window=20), None),
                     (mixer(heads=4, dim=16, rot_dim=8, kv_rank=32), moe()), (mixer(window=5), dense(40))],
                    loop={"start": 1, "stop": 3, "times": 3}),
    # sizes that are multiples of nothing
    "odd": config([(mixer(heads=3, dim=13, rot_dim=6, vdim=11, kv_rank=27, q_rank=21, window=7), dense(37)),
                   (mixer(heads=1, dim=5, rot_dim=2, vdim=3, kv_rank=9, q_rank=7, window=12), moe(experts=3, top=3, ff=13))],
                  width=61, vocab=103, loop={"start": 0, "stop": 2, "times": 2}, eps=1e-3, mult=1.0),
    # more heads than one attention tile holds, unlimited keys, one expert per token
    "heads": config([(mixer(heads=17, dim=16, rot_dim=16, vdim=16, kv_rank=64, window=None), moe(experts=4, top=1, ff=32)),
                     (mixer(heads=17, dim=64, rot_dim=32, vdim=64, kv_rank=160, window=70, rot_dims=16), dense(96))], width=160, vocab=200),
    # experts without a decision to make: every one of them, every time
    "all_experts": config([(mixer(heads=18, dim=24, rot_dim=16, vdim=24, kv_rank=80, window=33), moe(experts=3, top=3, ff=40)),
                           (mixer(heads=2, window=None), dense(48))], width=104, loop={"start": 0, "stop": 1, "times": 2}),
    # the largest split the tensor-core prompt kernel takes; a window of one key; the loop runs once
    "wide": config([(mixer(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96, window=100, scale=0.07), dense(128)),
                    (mixer(heads=2, dim=96, rot_dim=48, vdim=64, kv_rank=272, q_rank=64, window=1, scale=0.07), None)],
                   width=128, loop={"start": 0, "stop": 2, "times": 1}),
    # beyond what either tensor-core kernel takes
    "huge": config([(mixer(heads=2, dim=136, rot_dim=80, vdim=144, kv_rank=544, q_rank=64, window=40, scale=0.05), dense(64))], width=128),
}


def model_of(cfg, params, device, dtype):
    return Lupodra(LupodraConfig.from_dict(cfg, sequence_len=2048), dtype).load_tensors(
        {k: v.to(torch.bfloat16) for k, v in params.items()}, device)


def double(params):
    return {k: v.double() for k, v in params.items()}


def tokens_of(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    got, want = got.detach().double().cpu(), want.double()
    return (got - want).square().mean(-1).sqrt() / want.square().mean(-1).sqrt()


def routes(cfg):
    """Whether some router has a choice."""
    return any(x["mlp"] is not None and x["mlp"]["kind"] == "moe" and x["mlp"]["router"]["top"] < x["mlp"]["router"]["experts"]
               for x in cfg["layers"])


def assert_close(got, want, dtype, close_calls=False, tol=TOL):
    """`close_calls`: bf16 rounding may turn a few routing decisions of random weights, so a small part of the rows may be
    off (never most of them, and none in float32)."""
    err = row_errors(got, want).flatten()
    if close_calls and dtype == torch.bfloat16:
        assert err.median() < tol[dtype], err
        assert (err > tol[dtype]).float().mean() <= 0.15, err
    else:
        assert err.max() < tol[dtype], (err.max(), err.argmax())


def feed(engine, tokens, portions, max_tokens=None):
    """Logits of every position, the tokens cut as `portions` says (the last size repeats)."""
    seq = engine.open_sequence(max_tokens or len(tokens))
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(portions[min(k, len(portions) - 1)], len(tokens) - at)
        out.append(seq.extend(tokens[at:at + n], range(n)).cpu())
        at, k = at + n, k + 1
    seq.close()
    return torch.cat(out)


# -------------------------------------------------------------------------------- model

def check_cuts(name, device, dtype, n, cuts):
    """One prompt, cut in several ways, against the oracle."""
    cfg = CONFIGS[name]
    params = oracle.random_params(cfg, seed=3, sharp=2.0)
    tokens = tokens_of(cfg, n)
    want = oracle.forward(double(params), cfg, tokens)
    engine = Engine(model_of(cfg, params, device, dtype), None)
    for portions in cuts:
        assert_close(feed(engine, tokens, portions), want, dtype, routes(cfg))
    engine.check()


def check_reuse(device, dtype):
    """Pages and slots given back and used again, with whatever was left in them."""
    cfg = CONFIGS["heads"]
    params = oracle.random_params(cfg, seed=4)
    engine = Engine(model_of(cfg, params, device, dtype), None)
    long, short = tokens_of(cfg, 150, 5), tokens_of(cfg, 70, 6)
    first = {len(t): feed(engine, t, p, 200) for t, p in ((long, [90, 30, 1]), (short, [40, 1]))}
    cache = engine._cache_pool[1]
    for pool in cache.pools:
        pool.fill_(float("nan"))                # every page is rewritten before it is read
    for t, p in ((short, [40, 1]), (long, [90, 30, 1]), (short, [40, 1])):
        again = feed(engine, t, p, 200)
        assert torch.equal(again, first[len(t)]) or row_errors(again, first[len(t)]).max() < TOL[dtype] / 4
    assert engine._cache_pool[1] is cache


def check_rows(device, dtype, rows, name="mixed"):
    """Rows of one batch that go different ways after a common prompt, each against the oracle and against itself alone."""
    cfg = CONFIGS[name]
    params = oracle.random_params(cfg, seed=7, sharp=2.0)
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
    assert_close(got, want, dtype, routes(cfg))
    if not routes(cfg):
        assert_close(got[-1], feed(Engine(model, None), prompt + own[-1], [len(prompt), 1])[len(prompt):], dtype)


def greedy_expected(params, cfg, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(oracle.forward(double(params), cfg, tokens)[-1].argmax()))
    return tokens[len(prompt):]


def check_greedy(device, dtype, samples=1):
    cfg = CONFIGS["mixed"] if dtype == torch.float32 else CONFIGS["wide"]
    params = oracle.random_params(cfg, seed=9)
    prompt = tokens_of(cfg, 57, 10)
    want = greedy_expected(params, cfg, prompt, 12)
    model = model_of(cfg, params, device, dtype)
    got = list(Engine(model, None).generate(prompt, num_samples=samples, max_tokens=12, temperature=0.0))
    assert [c for c, _ in got] == [[t] * samples for t in want]
    assert list(model.generate(prompt, 12, temperature=0.0)) == want


# ----------------------------------------------------------------------------- one mixer

class OneMixer:
    """A single latent-attention mixer on given inputs h, run through the product's operation over its paged store."""

    def __init__(self, m, width, device, dtype, seed=0):
        self.cfg = config([(m, None)], width=width)
        self.params = oracle.random_params(self.cfg, seed=seed)
        self.mix = oracle.under(double(self.params), "l0.mix.")
        self.model = model_of(self.cfg, self.params, device, dtype)
        self.device, self.dtype, self.m, self.eps = device, dtype, m, self.cfg["norm"]["eps"]

    def expected(self, h, window="own"):
        m = dict(self.m)
        if window != "own":
            m["mask"] = {"size": window}
        return oracle.latent_attention(h.double(), self.mix, m, self.eps)

    def run(self, h, portions):
        from nanochat_b200 import ops
        layer = self.model.layers[0]
        cache = self.model.make_cache(1, h.shape[0])
        cache.reserve(0, h.shape[0])
        cache.begin_rows()
        full = torch.zeros(h.shape[0], self.model.width)
        full[:, :h.shape[1]] = h
        full = full.to(self.dtype).to(self.device)
        out, at, k = [], 0, 0
        while at < h.shape[0]:
            n = min(portions[min(k, len(portions) - 1)], h.shape[0] - at)
            z = ops.linear_rows(full[at:at + n], layer.w_in)
            out.append(layer.attn(z, cache, 0, n)[:, :h.shape[1]].float().cpu())
            cache.advance(n)
            at, k = at + n, k + 1
        return torch.cat(out)

    def standout(self, T, key, queries, seed=2, gain=1.0):
        """Inputs in which the key of token `key` dominates the scores of the tokens `queries` in head 0: the key's latent
        points along the queries' absorbed vector."""
        g = torch.Generator().manual_seed(seed)
        h = torch.randn(T, self.cfg["width"], generator=g).double()
        a = torch.randn(self.cfg["width"], generator=g).double()
        p, m = self.mix, self.m
        cq = oracle.plain_norm(p["dq"] @ a, p["dq.norm"], self.eps)
        q = (p["uq"] @ cq)[:m["dim"]]
        target = (p["uk"][:m["dim"]].T @ q) / p["dkv.norm"]
        b = torch.linalg.pinv(p["dkv"][:m["kv_rank"]]) @ target
        h[queries] = gain * a
        h[key] = b / b.norm() * a.norm()
        return h.to(torch.bfloat16).double()


def check_window_edges(device, dtype, m, width, T, keys, portions):
    """A key that stands out, asked for at the last place that sees it and at the first that does not."""
    one, w = OneMixer(m, width, device, dtype), m["mask"]["size"]
    for key in keys:
        inside, outside = key + w - 1, key + w
        queries = [i for i in {key + 1, inside, outside} if key < i < T]
        h = one.standout(T, key, queries)
        want = one.expected(h)
        # the inputs do show a window that is one key too small or too large
        for other, at in ((w + 1, outside), (w - 1, inside)):
            if key < at < T and other > 0:
                assert row_errors(one.expected(h, other), want)[at] > 5 * MIXER_TOL[dtype]
        for p in portions(key, w):
            assert_close(one.run(h, p), want, dtype, tol=MIXER_TOL)


def check_far_and_first(device, dtype, m, width, T, key, portions):
    """Unlimited keys: one token far back (or the very first) among hundreds."""
    one = OneMixer(m, width, device, dtype)
    h = one.standout(T, key, [T - 1, T // 2], gain=1.0)
    want = one.expected(h)
    blind = h.clone()
    blind[key] = h[key + 1]
    assert row_errors(one.expected(blind), want)[T - 1] > 5 * MIXER_TOL[dtype]
    for p in portions:
        assert_close(one.run(h, p), want, dtype, tol=MIXER_TOL)
