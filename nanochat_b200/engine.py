"""
Inference engine: KV cache, batched sampling and the tool-use state machine.

Behavioural contract (reference: nanochat/engine.py):
  * `KVCache` holds (n_layers, B, T, H, D) key/value tensors plus per-row lengths
    (engine.py:82-137); `prefill(other)` copies a batch-1 prompt cache into every
    row of a wider cache.
  * `Engine.generate` prefills the prompt once at batch 1, forks the cache to
    `num_samples` rows, samples every row's first token independently, then decodes
    in lock-step, yielding `(token_column, token_masks)` per step (mask 1 = sampled,
    0 = forced). Rows finish on <|assistant_end|> or <|bos|> (engine.py:176-275).
  * Between <|python_start|> and <|python_end|> the row's tokens are collected,
    decoded and handed to `use_calculator`; a result is force-fed back as
    <|output_start|> result <|output_end|> (engine.py:252-267).

B200-native differences: the cache position is mirrored on the host so a decode
step never calls `.item()`; on CUDA the per-token forward of a `GPT` is replayed
from a captured CUDA graph whose positions live in device memory (see
`runtime.DecodeGraph`), and weights are consumed from bf16 shadows instead of
being re-cast from fp32 every token. On that path the cache is paged
(`PagedKVCache`): the prompt is prefilled straight into pages that every sample
row's page table points at, so forking N samples copies at most one partial page
per row instead of the whole prompt, and N samples hold the prompt once.
"""

import math
import signal
import warnings
from collections import deque
from contextlib import contextmanager

import torch

from nanochat_b200 import common
from nanochat_b200 import ops


# ----------------------------------------------------------------------------
# calculator tool

@contextmanager
def timeout(duration, formula):
    def on_alarm(signum, frame):
        raise Exception(f"'{formula}': timed out after {duration} seconds")
    signal.signal(signal.SIGALRM, on_alarm)
    signal.alarm(duration)
    try:
        yield
    finally:
        signal.alarm(0)


def eval_with_timeout(formula, max_time=3):
    try:
        with timeout(max_time, formula):
            with warnings.catch_warnings():
                warnings.simplefilter("ignore", SyntaxWarning)
                return eval(formula, {"__builtins__": {}}, {})
    except Exception:
        signal.alarm(0)
        return None


_MATH_CHARS = set("0123456789*+-/.() ")
_TEXT_CHARS = set("abcdefghijklmnopqrstuvwxyzABCDEFGHIJKLMNOPQRSTUVWXYZ0123456789'\"()._ ")
_BANNED = ("__", "import", "exec", "eval", "compile", "open", "file", "input", "raw_input",
           "globals", "locals", "vars", "dir", "getattr", "setattr", "delattr", "hasattr")


def use_calculator(expr):
    """Evaluate a model-written expression: plain arithmetic (no **) or `'..'.count('..')`.

    Anything else returns None (reference: engine.py:46-79).
    """
    expr = expr.replace(",", "")
    if all(ch in _MATH_CHARS for ch in expr):
        if "**" in expr:
            return None
        return eval_with_timeout(expr)
    if not all(ch in _TEXT_CHARS for ch in expr):
        return None
    lowered = expr.lower()
    if any(bad in lowered for bad in _BANNED):
        return None
    if ".count(" not in expr:
        return None
    return eval_with_timeout(expr)


# ----------------------------------------------------------------------------

class KVCache:
    """Per-layer K/V store in (B, T, H, D) layout with in-place append.

    `cache_seqlens` (int32, device) is what kernels read; `_pos` mirrors row 0 on the
    host so the engine never synchronises to learn the position.
    """

    def __init__(self, batch_size, num_heads, seq_len, head_dim, num_layers, device, dtype):
        self.batch_size = batch_size
        self.max_seq_len = seq_len
        self.n_layers = num_layers
        self.n_heads = num_heads
        self.head_dim = head_dim
        shape = (num_layers, batch_size, seq_len, num_heads, head_dim)
        self.k_cache = torch.zeros(shape, device=device, dtype=dtype)
        self.v_cache = torch.zeros(shape, device=device, dtype=dtype)
        self.cache_seqlens = torch.zeros(batch_size, dtype=torch.int32, device=device)
        self.prev_embedding = None
        self._pos = 0

    def reset(self):
        self.cache_seqlens.zero_()
        self.prev_embedding = None
        self._pos = 0

    def get_pos(self):
        return self._pos

    def get_layer_cache(self, layer_idx):
        return self.k_cache[layer_idx], self.v_cache[layer_idx]

    def advance(self, num_tokens):
        self.cache_seqlens += num_tokens
        self._pos += num_tokens

    def prefill(self, other):
        """Fork: copy `other`'s filled prefix (batch 1) into every row of this empty cache."""
        assert self.get_pos() == 0, "Cannot prefill a non-empty KV cache"
        assert (self.n_layers, self.n_heads, self.head_dim) == (other.n_layers, other.n_heads, other.head_dim)
        assert self.max_seq_len >= other.max_seq_len
        n = other.get_pos()
        self.k_cache[:, :, :n] = other.k_cache[:, :, :n]
        self.v_cache[:, :, :n] = other.v_cache[:, :, :n]
        self.cache_seqlens.fill_(n)
        self._pos = n
        if other.prev_embedding is not None:
            self.prev_embedding = other.prev_embedding.expand(self.batch_size, -1, -1).clone()


PAGE_TOKENS = 64


class _PromptView:
    """The shared prompt pages of a paged cache seen as a batch-1 cache: what the prefill writes into. `get_layer_cache`
    serves KVCache's surface; a latent cache's kernels use `pools` and `table` instead."""

    def __init__(self, owner, capacity):
        self.owner = owner
        self.batch_size = 1
        self.max_seq_len = capacity
        self.n_layers = owner.n_layers
        self.cache_seqlens = torch.zeros(1, dtype=torch.int32, device=owner.device)
        self.prev_embedding = None
        self._pos = 0

    def get_pos(self):
        return self._pos

    def get_layer_cache(self, layer_idx):
        o, n = self.owner, self.max_seq_len // self.owner.page_tokens
        shape = (1, self.max_seq_len, o.n_heads, o.head_dim)
        return o.k_pool[layer_idx, :n].view(shape), o.v_pool[layer_idx, :n].view(shape)

    @property
    def pools(self):
        return self.owner.pools

    @property
    def table(self):
        return self.owner.identity_table[:, :self.max_seq_len // self.owner.page_tokens].contiguous()

    def advance(self, num_tokens):
        self.cache_seqlens += num_tokens
        self._pos += num_tokens


class PagedCache:
    """Pages of PAGE_TOKENS tokens plus a per-row page table for `batch_size` sample rows; what a page holds is up to the
    subclass (`_allocate`, `_copy_tokens`).

    Pool pages [0, shared_pages) hold the prompt, written once by the batch-1 prefill through `begin_prompt()`;
    `fork()` points every row's table at the prompt's full pages and gives each row private pages for the prompt's
    partial last page (copied: rows append into it) and for what it decodes. The decode kernels address tokens
    through the table. The pool grows when a request needs more pages than any before it; `pool_version` then moves so
    that a captured decode graph is rebuilt on the new addresses.
    """

    paged = True

    def __init__(self, batch_size, num_layers, seq_len, device, dtype, page_tokens):
        assert page_tokens & (page_tokens - 1) == 0, "page size must be a power of two"
        self.batch_size = batch_size
        self.max_seq_len = seq_len                  # per-row capacity in tokens (what the page table can address)
        self.n_layers = num_layers
        self.page_tokens = page_tokens
        self.max_pages = -(-seq_len // page_tokens)
        self.device, self.dtype = device, dtype
        self.table = torch.zeros(batch_size, self.max_pages, dtype=torch.int32, device=device)
        self.cache_seqlens = torch.zeros(batch_size, dtype=torch.int32, device=device)
        self.shared_pages = self.private_pages = 0
        self.pool_version = 0
        self.prev_embedding = None
        self._pos = 0
        self._row_end = 0

    # ----------------------------------------------------------------------------- pool
    def reserve(self, prompt_tokens, new_tokens):
        """Make room for a prompt of `prompt_tokens` and `new_tokens` decoded tokens per row."""
        P = self.page_tokens
        assert prompt_tokens + new_tokens <= self.max_seq_len
        self._reserve_pages(-(-prompt_tokens // P), -(-(prompt_tokens % P + new_tokens) // P))

    def reserve_any_prompt(self, tokens):
        """Make room for `tokens` tokens per row, however many of them the prompt turns out to be."""
        P = self.page_tokens
        assert tokens <= self.max_seq_len
        self._reserve_pages(-(-tokens // P), -(-tokens // P))

    def _reserve_pages(self, shared, private):
        if self.pool_version and shared <= self.shared_pages and private <= self.private_pages:
            return
        self.shared_pages = max(shared, self.shared_pages)
        self.private_pages = max(private, self.private_pages)
        # one spare page at the end: table entries a row has no page for point at it, so a token appended past a row's
        # pages lands there instead of in a page that holds someone's keys
        total = self.shared_pages + self.batch_size * self.private_pages + 1
        self.spare_page = total - 1
        self._allocate(total)
        self.identity_table = torch.arange(total, dtype=torch.int32, device=self.device)[None]
        self.pool_version += 1

    def reset(self):
        self.cache_seqlens.zero_()
        self.prev_embedding = None
        self._pos = 0

    def get_pos(self):
        return self._pos

    def advance(self, num_tokens):
        self.cache_seqlens += num_tokens
        self._pos += num_tokens

    # --------------------------------------------------------------------- prompt, fork
    def begin_prompt(self, prompt_tokens):
        """A batch-1 view of the shared pages for the prefill of a `prompt_tokens`-token prompt."""
        assert self.pool_version and -(-prompt_tokens // self.page_tokens) <= self.shared_pages
        self.reset()
        return _PromptView(self, -(-prompt_tokens // self.page_tokens) * self.page_tokens)

    def begin_rows(self):
        """Every row starts empty on its private pages."""
        self.reset()
        self._point_rows(0)

    def _point_rows(self, full):
        """Tables: the first `full` prompt pages, then each row's private pages, then the spare page."""
        first_private = self.shared_pages + torch.arange(self.batch_size, dtype=torch.int32, device=self.device) * self.private_pages
        table = torch.full((self.batch_size, self.max_pages), self.spare_page, dtype=torch.int32, device=self.device)
        if full:
            table[:, :full] = torch.arange(full, dtype=torch.int32, device=self.device)
        own = min(self.private_pages, self.max_pages - full)
        table[:, full:full + own] = first_private[:, None] + torch.arange(own, dtype=torch.int32, device=self.device)
        self.table.copy_(table)
        self._row_end = min(self.max_seq_len, (full + own) * self.page_tokens)
        return first_private

    def fork(self, view):
        """Every row continues the prompt in `view`: full prompt pages are shared, the partial last one is copied."""
        P, B = self.page_tokens, self.batch_size
        n = view.get_pos()
        full, rem = n // P, n % P
        first_private = self._point_rows(full)
        if rem:
            self._copy_tokens(first_private.long(), full, rem)
        self.cache_seqlens.fill_(n)
        self._pos = n
        self.prev_embedding = None
        if view.prev_embedding is not None:
            self.prev_embedding = view.prev_embedding.expand(B, -1, -1).clone()

    def row_capacity(self):
        """Tokens a row can hold with the pages it has now."""
        return self._row_end

    def _row_pages(self, row):
        return self.table[row, :-(-self._pos // self.page_tokens)].long()


class PagedKVCache(PagedCache):
    """Keys and values of every head (reference behaviour: nanochat/engine.py:82-137, a contiguous cache per row and a
    copy at the fork)."""

    def __init__(self, batch_size, num_heads, seq_len, head_dim, num_layers, device, dtype, page_tokens=PAGE_TOKENS):
        super().__init__(batch_size, num_layers, seq_len, device, dtype, page_tokens)
        self.n_heads, self.head_dim = num_heads, head_dim
        self.k_pool = self.v_pool = None

    def _allocate(self, total):
        shape = (self.n_layers, total, self.page_tokens, self.n_heads, self.head_dim)
        self.k_pool = self.v_pool = None            # release before allocating the larger pool
        self.k_pool = torch.zeros(shape, device=self.device, dtype=self.dtype)
        self.v_pool = torch.zeros(shape, device=self.device, dtype=self.dtype)

    def _copy_tokens(self, pages, source, n):
        self.k_pool[:, pages, :n] = self.k_pool[:, source:source + 1, :n]
        self.v_pool[:, pages, :n] = self.v_pool[:, source:source + 1, :n]

    def pool_bytes(self):
        return 0 if self.k_pool is None else 2 * self.k_pool.numel() * self.k_pool.element_size()

    def get_layer_cache(self, layer_idx):
        """One layer's pools, (pages, PAGE_TOKENS, H, D): the paged decode kernels take them with `table`."""
        return self.k_pool[layer_idx], self.v_pool[layer_idx]

    def gather_row(self, layer_idx, row):
        """(T, H, D) keys and values of one row in position order (tests and debugging; copies)."""
        n, pages = self._pos, self._row_pages(row)
        k = self.k_pool[layer_idx, pages].reshape(-1, self.n_heads, self.head_dim)[:n]
        v = self.v_pool[layer_idx, pages].reshape(-1, self.n_heads, self.head_dim)[:n]
        return k, v


class PagedLatentCache(PagedCache):
    """One vector per token and layer run, `widths[run]` elements (latent attention: the latent and the shared rotated key
    part). Layers of a loop have one pool per pass."""

    def __init__(self, batch_size, widths, seq_len, device, dtype, page_tokens=PAGE_TOKENS):
        super().__init__(batch_size, len(widths), seq_len, device, dtype, page_tokens)
        self.widths = list(widths)
        self.pools = None

    def _allocate(self, total):
        self.pools = None
        self.pools = [torch.zeros(total, self.page_tokens, w, device=self.device, dtype=self.dtype) for w in self.widths]

    def _copy_tokens(self, pages, source, n):
        for pool in self.pools:
            if pool.shape[2]:
                pool[pages, :n] = pool[source:source + 1, :n]

    def pool_bytes(self):
        return 0 if self.pools is None else sum(p.numel() * p.element_size() for p in self.pools)

    def gather_row(self, run, row):
        """(T, width) entries of one row in position order (tests and debugging; copies)."""
        return self.pools[run][self._row_pages(row)].reshape(-1, self.widths[run])[:self._pos]


class RecurrentCache(PagedLatentCache):
    """A paged store for the layers that attend (`widths[run]` elements a token, 0: none) and, beside it, fixed-size float
    states for the layers with a recurrence: `shapes[run]` names a layer's states and their shapes. All states of one
    sequence are one row of memory; row `batch_size` belongs to the prompt, and `fork()` copies it to the others.

    Nothing is cleared: kernels start a sequence at position 0 from zeros whatever its row holds."""

    ALIGN = 32                                       # floats

    def __init__(self, batch_size, widths, shapes, seq_len, device, dtype, page_tokens=PAGE_TOKENS):
        super().__init__(batch_size, widths, seq_len, device, dtype, page_tokens)
        places, total = [], 0
        for names in shapes:
            places.append({})
            for name, shape in names.items():
                n = math.prod(shape)
                places[-1][name] = (total, n, shape)
                total += -(-n // self.ALIGN) * self.ALIGN
        self.memory = torch.zeros(batch_size + 1, max(total, self.ALIGN), device=device)
        self.all_states = [{name: self.memory[:, at:at + n].unflatten(1, shape) for name, (at, n, shape) in p.items()} for p in places]
        self.states = [{name: t[:batch_size] for name, t in p.items()} for p in self.all_states]
        self.prompt_states = [{name: t[batch_size:] for name, t in p.items()} for p in self.all_states]
        self.done = torch.zeros(batch_size, dtype=torch.int32, device=device)     # counters of the step kernels, zero between steps

    def begin_prompt(self, prompt_tokens):
        view = super().begin_prompt(prompt_tokens)
        view.states, view.done = self.prompt_states, self.done[:1]
        return view

    def fork(self, view):
        super().fork(view)
        self.memory[:-1] = self.memory[-1]

    def state_bytes(self):
        return self.memory.numel() * self.memory.element_size()


@torch.inference_mode()
def sample_next_token(logits, rng, temperature=1.0, top_k=None):
    """(B, V) logits -> (B, 1) ids; argmax at temperature 0, else top-k / full multinomial."""
    return ops.sample_next_token(logits, rng, temperature, top_k)


class RowState:
    """Decode-time bookkeeping of one sample row."""

    __slots__ = ("current_tokens", "forced_tokens", "in_python_block", "python_expr_tokens", "completed")

    def __init__(self, current_tokens=None):
        self.current_tokens = current_tokens or []
        self.forced_tokens = deque()
        self.in_python_block = False
        self.python_expr_tokens = []
        self.completed = False


def ids_on_cuda(device):
    return torch.device(device).type == "cuda"


class Sequence:
    """One request fed in portions of any size: `extend` runs a portion's tokens on top of what earlier ones left and
    returns logits where asked. The first portion, and later ones of several tokens where the model can continue a
    sequence that way, take the prefill path, single tokens the decode step, as in `Engine.generate`. `close()` gives
    the pages back."""

    def __init__(self, engine, max_tokens):
        self.engine, self.max_tokens, self.length = engine, max_tokens, 0
        self.cache = engine._row_cache(1) if engine.own_cache or engine._graph_applies(1, max_tokens) else None
        if self.cache is None:                      # no captured decode here: a contiguous cache of its own
            self.cache = KVCache(batch_size=1, seq_len=max_tokens, **engine._kv_geometry())
        else:
            self.cache.reset()
            self.cache.reserve_any_prompt(max_tokens)

    @torch.inference_mode()
    def extend(self, tokens, want=()):
        """(len(want), V) float logits at the places `want` among `tokens`, or None when nothing is wanted."""
        n, want = len(tokens), list(want)
        if n == 0:
            return None
        if self.length + n > self.max_tokens:
            raise ValueError(f"sequence of {self.length + n} tokens, room for {self.max_tokens}")
        engine, paged = self.engine, getattr(self.cache, "paged", False)
        ids = torch.tensor([tokens], dtype=torch.long, device=engine.model.get_device())
        if self.length == 0:
            view = self.cache.begin_prompt(n) if paged else self.cache
            logits = engine._prompt_logits(ids, view, want)
            if paged:
                self.cache.fork(view)
            engine._begin_decode(self.cache)
        elif n > 1 and engine.own_cache:
            logits = engine._prompt_logits(ids, self.cache, want)
        else:
            rows = {}
            for i in range(n):
                step = engine._decode_step(ids[:, i:i + 1], self.cache)
                if i in want:
                    rows[i] = step.float().clone()
            logits = torch.cat([rows[i] for i in want]) if want else None
        self.length += n
        return logits

    def close(self):
        self.cache.reset()
        self.cache.in_use = False


class Engine:
    """`tokenizer` may be None (models without one): prompts and results are token ids and no token is special."""

    def __init__(self, model, tokenizer):
        self.model = model
        self.tokenizer = tokenizer
        self._decode_graphs = {}
        self._cache_pool = {}      # rows -> full-length cache reused across generations (keeps its decode graph)
        self.own_cache = hasattr(model, "make_cache")      # the model brings its own paged store

    def open_sequence(self, max_tokens):
        """A request of up to `max_tokens` tokens to be fed in portions; see Sequence."""
        return Sequence(self, max_tokens)

    def _prompt_logits(self, ids, cache, want):
        """Run a portion of tokens; (len(want), V) logits at the places `want`, None when there are none."""
        if self.own_cache:
            return self.model.forward(ids, kv_cache=cache, want=list(want))
        logits = self.model.forward(ids, kv_cache=cache)[0]
        return logits[list(want)].float() if len(want) else None

    def _begin_decode(self, cache):
        """The cache has been filled by a prompt: let its captured decode step take over what the prompt left."""
        if ids_on_cuda(self.model.get_device()) and ops.get_kernel_mode() == "native":
            from nanochat_b200.runtime import decode_graph_for
            runner = decode_graph_for(self, cache)
            if runner is not None:
                runner.begin()

    def _decode_step(self, ids, kv_cache):
        """One lock-step decode forward; returns (B, V) logits for the new position."""
        runner = None
        if ids.is_cuda and ops.get_kernel_mode() == "native":
            from nanochat_b200.runtime import decode_graph_for
            runner = decode_graph_for(self, kv_cache)
        if runner is not None:
            return runner.step(ids)
        if getattr(kv_cache, "paged", False) and kv_cache.get_pos() >= kv_cache.row_capacity():
            raise ValueError(f"no room for token {kv_cache.get_pos()}: the rows' pages hold {kv_cache.row_capacity()}")
        return self.model.forward(ids, kv_cache=kv_cache)[:, -1, :]

    @torch.inference_mode()
    def generate(self, tokens, num_samples=1, max_tokens=None, temperature=1.0, top_k=None, seed=42):
        assert isinstance(tokens, list) and isinstance(tokens[0], int), "expecting list of ints"
        device = self.model.get_device()
        rng = torch.Generator(device=device)
        rng.manual_seed(seed)

        cfg = self.model.config
        ids = torch.tensor([tokens], dtype=torch.long, device=device)
        capacity = (len(tokens) + max_tokens) if max_tokens is not None else cfg.sequence_len
        cache = self._pooled_cache(num_samples, len(tokens), capacity)
        pooled = cache is not None
        if pooled:
            # 1) batch-1 prefill straight into the pages every row will share  2) fork = page tables + one partial page
            view = cache.begin_prompt(len(tokens))
            logits = self._prompt_logits(ids, view, [len(tokens) - 1])
            cache.fork(view)
            logits = logits.expand(num_samples, -1)
        else:
            # 1) batch-1 prefill of the prompt  2) fork: copy it into every sample row of a contiguous cache
            geometry = self._kv_geometry()
            prompt_cache = KVCache(batch_size=1, seq_len=len(tokens), **geometry)
            logits = self.model.forward(ids, kv_cache=prompt_cache)
            cache = KVCache(batch_size=num_samples, seq_len=capacity, **geometry)
            cache.prefill(prompt_cache)
            del prompt_cache
            logits = logits[:, -1, :].expand(num_samples, -1)
        try:
            yield from self._decode_loop(tokens, num_samples, max_tokens, temperature, top_k, rng, logits, cache,
                                         self._special_tokens())
        finally:
            if pooled:
                cache.in_use = False

    def _kv_geometry(self):
        cfg = self.model.config
        return dict(num_heads=cfg.n_kv_head, head_dim=cfg.n_embd // cfg.n_head, num_layers=cfg.n_layer,
                    device=self.model.get_device(), dtype=common.COMPUTE_DTYPE)

    def _graph_applies(self, rows, capacity):
        from nanochat_b200.runtime import graph_path_applies
        return capacity <= self.model.config.sequence_len and graph_path_applies(self.model, rows)

    def check(self):
        """Raise if a kernel behind this engine recorded an error (a failed wait, a token without a page)."""
        if ids_on_cuda(self.model.get_device()) and ops.get_kernel_mode() == "native":
            (ops.serving_module() if self.own_cache else ops.native_module()).check_status()

    def _special_tokens(self):
        tok = self.tokenizer
        if tok is None:
            return (None,) * 6
        names = ("<|python_start|>", "<|python_end|>", "<|output_start|>", "<|output_end|>", "<|assistant_end|>")
        return (*(tok.encode_special(n) for n in names), tok.get_bos_token_id())

    def _row_cache(self, rows):
        """The paged cache of this row count, marked in use. It lives as long as the engine, so its captured decode graph
        is reused; its page pool grows to the largest request seen. A model with its own store gets a second, unpooled
        cache when the pooled one is busy (nested generations); for the others None then."""
        cache = self._cache_pool.get(rows)
        if cache is None:
            if self.own_cache:
                cache = self.model.make_cache(rows)
            else:
                cache = PagedKVCache(batch_size=rows, seq_len=self.model.config.sequence_len, **self._kv_geometry())
            cache.pooled = True
            cache.in_use = False
            self._cache_pool[rows] = cache
        if cache.in_use:
            if not self.own_cache:
                return None
            cache = self.model.make_cache(rows)
        cache.in_use = True
        return cache

    def _pooled_cache(self, rows, prompt_tokens, capacity):
        """A paged cache with room for the request, or None when the model decodes without one here (no captured graph
        for it, or its cache is busy)."""
        if self.own_cache:
            if capacity > self.model.config.sequence_len:
                raise ValueError(f"request of {capacity} tokens; this server holds {self.model.config.sequence_len} per row")
        elif not self._graph_applies(rows, capacity):
            return None
        cache = self._row_cache(rows)
        if cache is None:
            return None
        cache.reset()
        cache.reserve(prompt_tokens, capacity - prompt_tokens)
        return cache

    def _decode_loop(self, tokens, num_samples, max_tokens, temperature, top_k, rng, logits, cache, specials):
        python_start, python_end, output_start, output_end, assistant_end, bos = specials
        tok = self.tokenizer
        device = self.model.get_device()
        self._begin_decode(cache)
        # 3) lock-step decode with the per-row state machine
        rows = [RowState(tokens.copy()) for _ in range(num_samples)]
        produced = 0
        while True:
            if max_tokens is not None and produced >= max_tokens:
                break
            if all(r.completed for r in rows):
                break
            sampled = sample_next_token(logits, rng, temperature, top_k)[:, 0].tolist()
            column, masks = [], []
            for i, row in enumerate(rows):
                forced = len(row.forced_tokens) > 0
                token = row.forced_tokens.popleft() if forced else sampled[i]
                masks.append(0 if forced else 1)
                column.append(token)
                row.current_tokens.append(token)
                if token == assistant_end or token == bos:
                    row.completed = True
                if token == python_start:
                    row.in_python_block = True
                    row.python_expr_tokens = []
                elif token == python_end and row.in_python_block:
                    row.in_python_block = False
                    if row.python_expr_tokens:
                        result = use_calculator(tok.decode(row.python_expr_tokens))
                        if result is not None:
                            row.forced_tokens.append(output_start)
                            row.forced_tokens.extend(tok.encode(str(result)))
                            row.forced_tokens.append(output_end)
                    row.python_expr_tokens = []
                elif row.in_python_block:
                    row.python_expr_tokens.append(token)
            yield column, masks
            produced += 1
            ids = torch.tensor(column, dtype=torch.long, device=device).unsqueeze(1)
            logits = self._decode_step(ids, cache)

    def generate_batch(self, tokens, num_samples=1, **kwargs):
        """Non-streaming: returns (sequences, masks) without the terminal token; prompt mask is 0."""
        *_, assistant_end, bos = self._special_tokens()
        results = [tokens.copy() for _ in range(num_samples)]
        masks = [[0] * len(tokens) for _ in range(num_samples)]
        done = [False] * num_samples
        for column, column_masks in self.generate(tokens, num_samples, **kwargs):
            for i, (t, m) in enumerate(zip(column, column_masks)):
                if done[i]:
                    continue
                if t == assistant_end or t == bos:
                    done[i] = True
                else:
                    results[i].append(t)
                    masks[i].append(m)
            if all(done):
                break
        return results, masks


if __name__ == "__main__":
    # Self-check: the naive full-recompute sampler and the Engine must agree at temperature 0.
    import time
    from nanochat_b200.checkpoint_manager import load_model
    device_type = common.autodetect_device_type()
    _, _, _, _, device = common.compute_init(device_type)
    model, tokenizer, meta = load_model("base", device, phase="eval")
    prompt = tokenizer.encode("The chemical formula of water is", prepend=tokenizer.get_bos_token_id())
    t0 = time.time()
    naive = list(model.generate(prompt, max_tokens=64, temperature=0.0))
    t1 = time.time()
    fast = [col[0] for col, _ in Engine(model, tokenizer).generate(prompt, num_samples=1, max_tokens=64, temperature=0.0)]
    t2 = time.time()
    print(tokenizer.decode(naive))
    print(f"naive {t1 - t0:.2f}s | engine {t2 - t1:.2f}s | Match: {naive == fast}")
