"""
Execution runtime: CUDA-graph replay of the single-token decode step.

A decode step of the reference engine is one `model.forward` on a (B, 1) batch: a few hundred
small library kernels whose launch cost, not their work, sets the token rate
(reference: nanochat/engine.py:186-190). Here the step is a fixed sequence of purpose-built
kernels (`ops/csrc/decode.cu`: weight-streaming GEMV with fused residual / relu^2, rotary +
QK-norm + value-embedding gate + cache append, split-key attention) over static buffers. Every
position-dependent quantity is read from device memory (`KVCache.cache_seqlens`), so the whole
step is captured once per (engine, cache) and replayed with a single launch per token.

`StepGraph` is the capture-and-replay shell; `DecodeGraph` is GPT's step, `LatentDecodeGraph` that of models over a
paged latent store, `RecurrentDecodeGraph` that of models with recurrent states. A model names its step in `step_graph`.

`decode_graph_for(engine, kv_cache)` returns the graph of a cache, or None when the
fast path does not apply (CPU, kernels disabled, more than 64 rows, GPT with a head dim != 128).
"""

import os

import torch

from nanochat_b200 import common, ops
from nanochat_b200.ops import reference as ref_ops

LM_HEAD_PREFETCH_ROWS = 16384     # rows of lm_head (54 MB at 1664 wide) the last layer prefetches: what L2 can hold
MAX_ROWS = 64          # rows of one decode graph; up to GEMV_ROWS of them use the weight-streaming GEMV
GEMV_ROWS = 8
# Up to this many rows the layer's mix + norm is folded into the QKV GEMV (one launch fewer per layer). Every CTA of
# that GEMV redoes the mix for its rows, which is free while the kernel waits on memory (few rows) and costs more
# than the launch it saves once the rows make it arithmetic-bound. Measured on d26: 1 row +4.8 %, 2 rows +2 %,
# 4 rows -5 %, 8 rows -4 % tokens per second.
FOLD_MIX_ROWS = int(os.environ.get("NANOCHAT_DECODE_FOLD_ROWS", "2"))
# every GEMV of the step prefetches the next kernel's weight matrix into L2 (NANOCHAT_DECODE_PREFETCH=0: off, A/B runs)
PREFETCH_NEXT = os.environ.get("NANOCHAT_DECODE_PREFETCH", "1") != "0"


class StepGraph:
    """A decode step over static buffers, run eagerly once (kernels get configured outside a capture), captured at the
    second call and replayed from then on. Subclasses define `_forward` (reads `self.ids`, leaves `self.logits`) and may
    refresh what it reads in `_prepare`."""

    def __init__(self, model, kv_cache):
        self.model, self.cache = model, kv_cache
        self.paged = getattr(kv_cache, "paged", False)
        self.pool_version = getattr(kv_cache, "pool_version", 0)
        self.B = kv_cache.batch_size
        self.ids = torch.zeros(self.B, 1, dtype=torch.long, device=kv_cache.cache_seqlens.device)
        self.graph = None
        self.warm = False

    def begin(self):
        """Start of a generation: the cache has just been filled by a prompt."""

    def _prepare(self):
        pass

    @torch.inference_mode()
    def step(self, ids):
        """ids: (B, 1) token ids of the new position; returns (B, V) fp32 logits (a static buffer, valid until
        the next step)."""
        if self.paged and self.cache.get_pos() >= self.cache.row_capacity():
            raise ValueError(f"no room for token {self.cache.get_pos()}: the rows' pages hold {self.cache.row_capacity()}")
        self.ids.copy_(ids)
        self._prepare()
        if self.graph is not None:
            self.graph.replay()
        elif not self.warm:
            self._forward()                      # first step runs eagerly: kernels get configured outside capture
            self.warm = True
        else:
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g):
                self._forward()
            self.graph = g
            g.replay()
        self.cache._pos += 1
        return self.logits


class DecodeGraph(StepGraph):
    """GPT's decode step."""

    def __init__(self, model, kv_cache):
        super().__init__(model, kv_cache)
        nat = ops.native_module()
        self.nat, self.C_ = nat, nat._C
        cfg = model.config
        dev = kv_cache.cache_seqlens.device
        B, C = kv_cache.batch_size, cfg.n_embd
        self.C = C
        self.H, self.Hkv = cfg.n_head, cfg.n_kv_head
        nq, nkv = self.H * 128, self.Hkv * 128
        bf16 = torch.bfloat16
        e = lambda *shape, dtype=bf16: torch.empty(*shape, dtype=dtype, device=dev)
        self.prev = torch.zeros(B, C, dtype=bf16, device=dev)
        self.xm, self.xn, self.xa, self.xn2 = e(B, C), e(B, C), e(B, C), e(B, C)
        self.xs = [e(B, C), e(B, C)]                       # residual stream ping-pong
        self.x_in = e(B, C)                                # embedding + smear: the stream's input and the x0 of every layer
        self.x_backout = e(B, C)
        self.qkv, self.y, self.h = e(B, nq + 2 * nkv), e(B, nq), e(B, 4 * C)
        self.logits_bf16 = e(B, model.lm_head.weight.shape[0])
        self.logits = e(B, cfg.vocab_size, dtype=torch.float32)
        self.scratch = torch.zeros(self.C_.decode_attn_scratch(B, self.H), dtype=torch.float32, device=dev)
        self.cos = model.cos.reshape(-1, 64).contiguous()
        self.sin = model.sin.reshape(-1, 64).contiguous()
        self.use_gemv = B <= GEMV_ROWS     # more rows: the tcgen05 GEMM (rows padded to a 128-row tile) inside the graph
        self.weights_epoch = None
        self.w = None

    # ------------------------------------------------------------------ weights
    def _refresh_weights(self):
        """bf16 operand copies laid out for the step (fused QKV); re-copied in place when the parameters moved,
        so a captured graph keeps pointing at valid buffers."""
        nat = self.nat
        m = self.model
        fresh = []
        for blk in m.transformer.h:
            a = blk.attn
            fresh.append(dict(
                qkv=[nat.shadow_of(a.c_q.weight), nat.shadow_of(a.c_k.weight), nat.shadow_of(a.c_v.weight)],
                o=nat.shadow_of(a.c_proj.weight), fc=nat.shadow_of(blk.mlp.c_fc.weight),
                pr=nat.shadow_of(blk.mlp.c_proj.weight),
                wg=a.ve_gate.weight if a.ve_gate is not None else None))
        lm_head = nat.shadow_of(m.lm_head.weight)
        epoch = nat._weights_epoch            # read after the shadows: a re-cast above moves it
        if self.w is not None and self.weights_epoch == epoch:
            return
        first = self.w is None
        if first:
            self.w = []
        for i, f in enumerate(fresh):
            if first:
                self.w.append(dict(qkv=torch.cat(f["qkv"]).contiguous(),
                                   wg=f["wg"].detach().float().contiguous() if f["wg"] is not None else None))
            else:
                torch.cat(f["qkv"], out=self.w[i]["qkv"])
                if f["wg"] is not None:
                    self.w[i]["wg"].copy_(f["wg"].detach().float())
            # the other matrices are used where they live (bf16 parameters or their persistent shadows)
            self.w[i].update(o=f["o"], fc=f["fc"], pr=f["pr"])
        self.lm_head = lm_head
        self.weights_epoch = epoch
        # tensors the step reads where they live: if any of them was re-homed since the capture (a parameter arena
        # built later, a checkpoint loaded with assign=True) the captured addresses are stale and the graph is dropped
        where = tuple(t.data_ptr() for w in self.w for t in (w["o"], w["fc"], w["pr"])) + (
            lm_head.data_ptr(), m.transformer.wte.weight.data_ptr(),
            *[ve.weight.data_ptr() for ve in m.value_embeds.values()])
        if where != getattr(self, "_captured_where", where):
            self.graph, self.warm = None, False
        self._captured_where = where

    # --------------------------------------------------------------------- step
    def _linear(self, x, w, out, aux=None, relu2=False, norm_input=False, next_w=None):
        """out = epi(norm?(x) @ w^T) (+ aux): GEMV for a few rows, tensor-core GEMM otherwise. `next_w`: the weight
        matrix the following kernel will stream; the GEMV's CTAs prefetch it into L2 (decode is latency-bound per
        kernel, so keeping HBM busy across kernel boundaries is what raises the weight-streaming rate)."""
        if self.use_gemv:
            self.C_.gemv_rows(x, w, out, aux, 1 if relu2 else 0, norm_input, next_w if PREFETCH_NEXT else None)
            return
        nat = self.nat
        if norm_input:
            self.C_.norm_fwd(x, self.xn2, None)
            x = self.xn2
        nat.gemm(x, w, out, aux=aux, beta=1.0 if aux is not None else 0.0,
                 epi=nat.EPI_RELU2 if relu2 else nat.EPI_LINEAR)

    def _forward(self):
        m, C_ = self.model, self.C_
        B, H, Hkv = self.B, self.H, self.Hkv
        nq = H * 128
        cache = self.cache
        idx = self.ids[:, 0]
        # embedding gather, norm, smear with the previous token's embedding and the update of that state: one kernel
        C_.decode_embed(self.ids, m.transformer.wte.weight, m.smear_gate.weight.detach().float().contiguous().view(-1),
                        m.smear_lambda.detach().float().view(1), self.prev, self.x_in)
        x0 = x = self.x_in
        backout_layer = m.config.n_layer // 2
        scale = 1.0 / (128 ** 0.5)
        for i, w in enumerate(self.w):
            # what the kernel after this layer's last GEMV streams: the next layer's QKV weights, or the head of lm_head
            after = self.w[i + 1]["qkv"] if i + 1 < len(self.w) else self.lm_head[:LM_HEAD_PREFETCH_ROWS]
            if self.use_gemv and B <= FOLD_MIX_ROWS:
                # mix + norm folded into the QKV GEMV; its first CTA writes xm and the gate's slice of xn
                C_.gemv_rows_mix(x, x0, m.resid_lambdas, m.x0_lambdas, i, w["qkv"], self.qkv, self.xm, self.xn,
                                 w["o"] if PREFETCH_NEXT else None)
            else:
                C_.mixnorm_fwd(x, x0, m.resid_lambdas, m.x0_lambdas, i, self.xm, self.xn, None)
                self._linear(self.xn, w["qkv"], self.qkv, next_w=w["o"])
            ve = m.value_embeds[str(i)].weight if str(i) in m.value_embeds else None
            kc, vc = cache.get_layer_cache(i)
            # a paged cache: one layer's page pools + the rows' page table; the row capacity bounds the append
            table = cache.table if self.paged else None
            t_max = cache.max_seq_len if self.paged else 0
            C_.decode_qkv_post(self.qkv, H, Hkv, self.cos, self.sin, cache.cache_seqlens,
                               self.xn if ve is not None else None, w["wg"] if ve is not None else None, ve,
                               idx if ve is not None else None, kc, vc, table, t_max)
            window = m.window_sizes[i][0]
            window = window if 0 <= window < cache.max_seq_len else -1
            C_.decode_attn(self.qkv[:, :nq], kc, vc, cache.cache_seqlens, H, Hkv, window, scale, self.scratch, self.y,
                           table)
            self._linear(self.y, w["o"], self.xa, aux=self.xm, next_w=w["fc"])
            self._linear(self.xa, w["fc"], self.h, relu2=True, norm_input=True, next_w=w["pr"])   # GEMV: norm(xa) folded in
            out = self.x_backout if i == backout_layer else self.xs[i & 1]
            self._linear(self.h, w["pr"], out, aux=self.xa, next_w=after)
            x = out
        C_.backout_norm_fwd(x, self.x_backout, m.backout_lambda.detach().float(), self.xn)
        self._linear(self.xn, self.lm_head, self.logits_bf16)
        C_.softcap_logits(self.logits_bf16, self.logits, m.config.vocab_size, ref_ops.SOFTCAP)
        cache.cache_seqlens.add_(1)

    def begin(self):
        """Start of a generation: take over the smear state the prefill left in the cache."""
        prev = self.cache.prev_embedding
        if prev is None:
            self.prev.zero_()
        else:
            self.prev.copy_(prev.reshape(self.B, self.C))
        self._refresh_weights()

    def _prepare(self):
        if self.weights_epoch != self.nat._weights_epoch or self.w is None:
            self._refresh_weights()


class LatentDecodeGraph(StepGraph):
    """Decode step of models over a paged latent store (`make_cache`).

    Up to GEMV_ROWS bf16 rows: a fixed set of serving kernels per layer. Both sublayers read the same normed rows, so after
    the product that reads them the feed-forward runs beside the attention on a second stream; kernels of one stream are
    launched so that each may start while the one before it ends:
        norm + everything that reads it (down-projections, gates, up-projection, router)
        main: query latent's norm + query projection, extra CTAs append to the store  ->  absorbed queries  ->  attention,
              split over keys  ->  splits merged + value projection
        side: activation  ->  down projection + gate;   or routing  ->  experts' gate and up  ->  experts' down + gate
        join: output projection + gated residual, the side's result added
    Otherwise (more rows, or float32): the model's forward over the rows, captured as it is."""

    def __init__(self, model, kv_cache):
        super().__init__(model, kv_cache)
        S = ops.serving_module()
        self.S = S
        cfg, B, dev = model.config, self.B, kv_cache.cache_seqlens.device
        self.logits = torch.empty(B, model.embed.shape[0], dtype=torch.float32, device=dev)[:, :cfg.vocab_size]
        self.fused = (B <= GEMV_ROWS and model.dtype == torch.bfloat16 and
                      all(S._S.expert_rows_supported(B, getattr(layer.mlp, "top", 1)) for layer in model.layers))
        if not self.fused:
            return
        f32 = lambda *shape: torch.empty(*shape, dtype=torch.float32, device=dev)
        b16 = lambda *shape: torch.empty(*shape, dtype=torch.bfloat16, device=dev)
        self.x, self.h = f32(B, model.width), b16(B, model.width)
        self.x0 = f32(B, model.width) if model.keep_x0 else None
        self.all_logits = f32(B, model.embed.shape[0])
        self.logits = self.all_logits[:, :cfg.vocab_size]
        layers = [layer for layer, _ in model.runs]
        most = lambda size: max((size(layer) for layer in layers), default=8)
        self.z = f32(B * most(lambda l: l.w_all.shape[0]))
        self.q = b16(B * most(lambda l: l.attn.w_q.shape[0]))
        self.qa = b16(B * most(lambda l: l.attn.heads * l.attn.kvp))
        self.y = b16(B * most(lambda l: l.attn.heads * l.attn.vp))
        self.act = b16(B * most(lambda l: 8 if l.mlp is None else l.mlp.fp * getattr(l.mlp, "top", 1)))
        self.ff = f32(B, model.width)                      # the feed-forward's gated contribution to the stream
        tops = [getattr(l.mlp, "top", 1) for l in layers] + [1]
        self.idx = torch.empty(B * max(tops), dtype=torch.int32, device=dev)
        self.wt = f32(B * max(tops))
        self.side = torch.cuda.Stream(device=dev)
        self.splits = [S.attention_splits(l.attn, B, min(kv_cache.max_seq_len, l.attn.window or kv_cache.max_seq_len), True)
                       for l in layers]
        self.ml = f32(max([B * l.attn.heads * s * 2 for l, s in zip(layers, self.splits)] + [2]))
        self.acc = f32(max([B * l.attn.heads * s * l.attn.kvp for l, s in zip(layers, self.splits)] + [8]))

    def _forward(self):
        if self.fused:
            self._fused_step()
            self.cache.cache_seqlens.add_(1)
        else:
            pos = self.cache._pos
            self.logits.copy_(self.model.forward(self.ids, kv_cache=self.cache)[:, 0])
            self.cache._pos = pos                # step() moves the host's mirror, replayed or not

    def _fused_step(self):
        m, K, B, cache, cfg = self.model, self.S._S, self.B, self.cache, self.model.config
        C, eps, mult = cfg.n_embd, cfg.eps, cfg.residual_mult
        table, lens, x = cache.table, cache.cache_seqlens, self.x
        ahead = lambda w: w if PREFETCH_NEXT else None
        view = lambda buf, n: buf[:B * n].view(B, n)
        K.embed_norm(self.ids, m.embed, cfg.vocab_size, m.final_norm, eps, C, x, self.x0, None)
        for run, (layer, _) in enumerate(m.runs):
            a, mlp = layer.attn, layer.mlp
            again = run + 1 < len(m.runs) and m.runs[run + 1][1]
            extra = self.x0 if again else None
            moe = hasattr(mlp, "top")
            z = view(self.z, layer.w_all.shape[0])
            q, qa, y = view(self.q, a.w_q.shape[0]), view(self.qa, a.heads * a.kvp), view(self.y, a.heads * a.vp)
            gate = lambda k: z[:, layer.gates[k]:layer.gates[k] + m.width]
            K.gemv_norm(x, layer.norm, eps, C, layer.w_all, z, self.h if moe else None, ahead(a.w_q))
            if mlp is not None:
                main = torch.cuda.current_stream()
                self.side.wait_stream(main)
                with torch.cuda.stream(self.side):
                    if moe:
                        idx, wt = (view(t, mlp.top) for t in (self.idx, self.wt))
                        K.route_topk(z[:, layer.n_in:], mlp.experts, idx, wt)
                        act = self.act[:B * mlp.top * mlp.fp].view(B * mlp.top, mlp.fp)
                        K.expert_rows(self.h, mlp.w_gate_up, mlp.w_down, idx, wt, act, self.ff, gate(1), layer.rg2_bias, mult, extra)
                    else:
                        act = view(self.act, mlp.fp)
                        K.poly_norm(z[:, layer.up_off:layer.n_in], mlp.act, eps, mlp.ff, act)
                        K.gemv_residual(act, mlp.w_down, self.ff, gate(1), layer.rg2_bias, mult, extra, accumulate=False)
            K.gemv_query_store(z, a.q_rank, a.q_norm, eps, a.w_q, q, a.c_off, a.kv_rank, a.kvp, a.kv_norm, a.rot_off,
                               a.rot_dim, a.freq, cache.pools[run], table, lens, ahead(a.w_kv))
            K.absorb_query(q, a.heads, a.w_uk, qa, True)
            splits = self.splits[run]
            K.latent_attention(qa, q, a.heads, a.dp, a.rot_dim, a.freq, a.kvp, cache.pools[run], table, lens, 1,
                               a.window or 0, a.scale, splits, self.ml, self.acc, True)
            K.latent_values(self.ml, self.acc, B, a.heads, splits, a.w_uv, y, True, ahead(a.w_o))
            if mlp is not None:
                main.wait_stream(self.side)
            after = m.runs[run + 1][0].w_all if run + 1 < len(m.runs) else m.embed[:LM_HEAD_PREFETCH_ROWS]
            K.gemv_residual(y, a.w_o, x, gate(0), layer.rg1_bias, mult, extra if mlp is None else self.ff, ahead(after),
                            pdl=mlp is None)
        K.gemv_norm(x, m.final_norm, eps, C, m.embed, self.all_logits)


class RecurrentDecodeGraph(StepGraph):
    """Decode step of models over a `RecurrentCache`.

    Up to GEMV_ROWS bf16 rows: one chain of kernels, each launched so that it may start while the one before it ends:
        input product  ->  mixer (delta rule; or window attention and fixed-decay heads side by side)  ->  output product
        ->  its norm, residual, next norm  ->  gate and up product with the activation  ->  down product  ->  norms
    Otherwise (more rows, float32, sizes a step kernel does not take): the model's forward over the rows, captured as it is."""

    def __init__(self, model, kv_cache):
        super().__init__(model, kv_cache)
        S = ops.serving_module()._S
        self.S = S
        cfg, B, dev = model.config, self.B, kv_cache.cache_seqlens.device
        self.all_logits = torch.empty(B, model.head.shape[0], dtype=torch.float32, device=dev)
        self.logits = self.all_logits[:, :cfg.vocab_size]

        def fits(mix):
            if hasattr(mix, "left"):
                return S.window_step_supported(False, mix.left.dp) and S.decay_step_supported(mix.right.dp, mix.right.vp)
            return S.delta_step_supported(mix.dp, mix.vp)

        self.fused = B <= GEMV_ROWS and model.dtype == torch.bfloat16 and all(fits(layer.mix) for layer in model.layers)
        if not self.fused:
            return
        f32 = lambda *shape: torch.empty(*shape, dtype=torch.float32, device=dev)
        b16 = lambda *shape: torch.empty(*shape, dtype=torch.bfloat16, device=dev)
        most = lambda size: max((size(layer) for layer in model.layers), default=8)
        self.x, self.h, self.out = f32(B, model.width), b16(B, model.width), f32(B, model.width)
        self.z = f32(B * most(lambda l: l.mix.w_all.shape[0]))
        self.y = b16(B * most(lambda l: l.mix.y_width))
        self.act = b16(B * most(lambda l: 8 if l.mlp is None else l.mlp.fp))
        self.o = f32(B * most(lambda l: l.mix.right.y_width if hasattr(l.mix, "right") else 8))

    def _forward(self):
        if self.fused:
            self._fused_step()
            self.cache.cache_seqlens.add_(1)
        else:
            pos = self.cache._pos
            self.logits.copy_(self.model.forward(self.ids, kv_cache=self.cache)[:, 0])
            self.cache._pos = pos                # step() moves the host's mirror, replayed or not

    def _fused_step(self):
        m, K, B, cache, cfg = self.model, self.S, self.B, self.cache, self.model.config
        C, eps, lens, table = cfg.n_embd, cfg.eps, cache.cache_seqlens, cache.table
        ahead = lambda w: w if PREFETCH_NEXT else None
        view = lambda buf, n: buf[:B * n].view(B, n)
        subs = m.sublayers()
        opening = lambda sub: sub.w_gate_up if hasattr(sub, "w_gate_up") else sub.w_all
        K.layer_norm_residual(self.ids, m.embed, cfg.vocab_size, m.embed_norm, self.x, m.first_norm, eps, C, self.h)
        for n, (sub, post, after, i) in enumerate(subs):
            following = opening(subs[n + 1][0]) if n + 1 < len(subs) else m.head[:LM_HEAD_PREFETCH_ROWS]
            if i is None:
                act = view(self.act, sub.fp)
                K.gemv_relu_glu(self.h, sub.w_gate_up, act, ahead(sub.w_down))
                K.gemv_plain(act, sub.w_down, self.out, ahead(following))
            else:
                z, y = view(self.z, sub.w_all.shape[0]), view(self.y, sub.y_width)
                K.gemv_plain(self.h, sub.w_all, z, ahead(sub.w_o))
                state = cache.states[i]
                if hasattr(sub, "left"):
                    a, b = sub.left, sub.right
                    K.parallel_step(z, a.sizes, a.reals, a.freq, cache.pools[i], table, lens, y[:, :a.y_width], b.sizes, b.reals, b.log_decay,
                                    state["S"], b.norm, view(self.o, b.y_width), cache.done, y[:, a.y_width:])
                else:
                    K.delta_step(z, sub.sizes, sub.conv, z[:, sub.channels + sub.y_width:], sub.neg_a, sub.dt_bias, state["ring"], state["S"],
                                 lens, sub.norm, sub.eps, sub.gate_off, y)
                K.gemv_plain(y, sub.w_o, self.out, ahead(following))
            K.layer_norm_residual(None, self.out, 0, post, self.x, after, eps, C, self.h)
        K.gemv_plain(self.h, m.head, self.all_logits)


def graph_path_applies(model, rows):
    """True when `rows` sample rows of this model decode through the captured-graph kernels."""
    if ops.get_kernel_mode() != "native":
        return False
    if hasattr(model, "make_cache"):
        return model.get_device().type == "cuda" and rows <= MAX_ROWS
    from nanochat_b200.models.gpt import GPT
    if not isinstance(model, GPT):
        return False
    cfg = model.config
    wte = model.transformer.wte.weight
    return (wte.is_cuda and cfg.n_embd // cfg.n_head == 128 and rows <= MAX_ROWS and cfg.n_embd % 8 == 0
            and common.COMPUTE_DTYPE == torch.bfloat16 and wte.dtype == torch.bfloat16)


def decode_graph_for(engine, kv_cache):
    """The DecodeGraph bound to `kv_cache` (created on first use), or None when the fast path does not apply."""
    model = engine.model
    if (not getattr(kv_cache, "pooled", False) or not kv_cache.cache_seqlens.is_cuda
            or not graph_path_applies(model, kv_cache.batch_size)):
        return None
    graphs = engine._decode_graphs
    g = graphs.get(id(kv_cache))
    if g is None or g.cache is not kv_cache or g.pool_version != getattr(kv_cache, "pool_version", 0):
        kind = globals()[getattr(model, "step_graph", "DecodeGraph")]
        g = kind(model, kv_cache)              # first use, or the page pool moved: capture on the new addresses
        graphs[id(kv_cache)] = g
    return g
