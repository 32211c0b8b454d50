"""Serving of the layered decoders (models/layered.py): scheduler, slots, pages, sampling and CUDA-graph decode are
:class:`~trl_b200.rollout.engine.RolloutEngine`'s; this module adds what a layer keeps between tokens and how it takes
one token further.

Every layer run has a cache of its own, also one that runs with another one's weights and every pass of a loop (a layer with ``kv_from``
reads that layer's instead):

    latent_attention   pages of latent rows ``[kv_rank | rotated key]`` behind the engine's block table (the window is a
                       mask: pages stay until the sequence ends)
    attention          pages of keys (normed, rotated) and pages of values (the projected keys where those serve as values);
                       a window is a mask here too.  With pooled blocks also, per slot, rows of the means of the complete ones
    mlstm              per slot an fp32 matrix state, its normaliser and running maximum
    rglru              per slot an fp32 state vector and the last inputs of the convolution
    hgrn2              per slot an fp32 matrix state
    parallel           what its two halves keep

An embedding of token pairs keeps the last token per slot.

A decode step is one graph: embed, then per layer norm (+ residual) -> input projection -> mixer -> output projection
-> norm (+ residual) -> up / activation -> down (mixer and feed-forward side by side: one norm kernel in front of both), or router -> choice -> gather -> experts -> sum (-> stream -> side gate -> side projection), then final norm, head and
sampler.  Norms on a sublayer's output ride on the norm kernel that follows.  With bf16 weights the projections are the
weight-streaming tcgen05 kernel; their fp32 sums are consumed and cleared by the next kernel.  fp32 models run the same
kernels' fp32 forms with library fp32 matrix products."""
from __future__ import annotations

import os

import torch

from ..models.decoder import SeqCtx
from ..models.layered import ExpertMlp
from ..ops import mixers as mx
from .engine import RolloutEngine


class _LatentSlots:
    """Decode side of one ``latent_attention`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li):
        from ..ops import cuda_mixers as K

        self.e, self.m = eng, m
        self.kr, self.width = K.latent_row(m.kv_rank, m.rot_dim)
        self.cache = torch.zeros(eng.num_blocks, eng.block_size, self.width, dtype=eng.dtype, device=eng.dev)
        self.table = m.rope.table(eng.max_len + 1, eng.dev) if m.rot_dim else None
        B = eng.max_seqs
        self.acc_in = eng.sums("in", m.w_in.shape[0])
        if m.q_rank:  # queries through a latent: prepared with the rest of the row
            self.acc_q, self.acc_prep = eng.sums("q", m.uq.shape[0]), self.acc_in
            self.cq = eng.scratch("cq", B, m.q_rank)
        else:
            self.acc_q, self.acc_prep, self.cq = self.acc_in[:, : m.q_rows], self.acc_in[:, m.q_rows:], None
        self.gate = eng.scratch("gate", B, m.heads, dtype=torch.float32) if m.gated else None
        self.q_lat = eng.scratch("q_lat", B, m.heads, self.width)
        self.o_lat = eng.scratch("o_lat", B, m.heads, m.kv_rank)
        self.o = eng.scratch("o", B, m.heads * m.vdim)
        # tensor-core decode; other sizes and fp32 run the CUDA-core kernels
        self.tc = eng.dtype == torch.bfloat16 and K.latent_decode_tc_ok(m, eng.block_size)
        if self.tc:
            tiles = -(-(m.window or eng.max_len) // 128) + 1
            ctas = B * -(-m.heads // 32)
            self.splits = max(1, min(8, tiles, 148 // ctas))
            self.q = eng.scratch("q", B, m.heads, m.dim + m.rot_dim)
            self.part_o = eng.scratch("part_o", B, m.heads * self.splits * m.kv_rank, dtype=torch.float32)
            self.part_ml = eng.scratch("part_ml", B, m.heads * self.splits * 2, dtype=torch.float32)

    def prompt_target(self, pages: "_Pages") -> dict:
        return dict(cache=self.cache, tok_slot=pages.tok_slot, block_table=self.e.block_table, block_size=self.e.block_size)

    def copy_pages(self, dst, src):
        self.cache.index_copy_(0, dst, self.cache.index_select(0, src))

    def copy_slots(self, dst, src):
        pass

    def attend(self):
        """Absorbed queries against the cached latent rows -> ``o_lat``."""
        from ..ops import cuda_mixers as K

        e = self.e
        if self.tc:
            K.latent_decode_tc(self.q_lat, self.cache, self.m, e.seq_lens, e.block_table, e.block_size, self.o_lat,
                               self.part_o, self.part_ml, self.splits)
        else:
            K.latent_decode(self.q_lat, self.cache, self.m, e.seq_lens, e.block_table, e.block_size, self.o_lat)

    def absorb(self):
        """``acc_q`` -> queries in the latent basis, ``q_lat``."""
        from ..ops import cuda_mixers as K

        e, m = self.e, self.m
        if self.tc:
            K.latent_query(self.acc_q, m, e.seq_lens, self.table, self.q, self.q_lat)
            K.head_gemm(self.q, m.uk.view(m.heads, m.dim, m.kv_rank), self.q_lat, w_mn=True)
        else:
            K.latent_absorb(self.acc_q, m, e.seq_lens, self.table, self.q_lat, True)

    def expand(self):
        """``o_lat`` -> gated head outputs, ``o``."""
        from ..ops import cuda_mixers as K

        m = self.m
        if self.tc:
            K.head_gemm(self.o_lat, m.uv.view(m.heads, m.vdim, m.kv_rank), self.o.view(-1, m.heads, m.vdim), scale=self.gate)
        else:
            K.latent_expand(self.o_lat, m, self.gate, self.e.seq_lens, self.o)

    def step(self, h, out):
        from ..ops import cuda_mixers as K

        e, m = self.e, self.m
        e.gemm(h, m.w_in, self.acc_in)
        K.latent_prep(self.acc_prep, m, e.seq_lens, self.table, clear=True, cq=self.cq, gate=self.gate, cache=self.cache,
                      block_table=e.block_table, block_size=e.block_size)
        if m.q_rank:
            e.gemm(self.cq, m.uq, self.acc_q)
        self.absorb()
        self.attend()
        self.expand()
        e.gemm(self.o, m.o, out)


class _MLstmSlots:
    """Decode side of one ``mlstm`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li):
        self.e, self.m = eng, m
        B, f32 = eng.max_seqs, dict(dtype=torch.float32, device=eng.dev)
        # the normaliser and the maximum are double-buffered by the parity of the token count (csrc/mixers.cu)
        self.state = (torch.zeros(B, m.heads, m.dim, m.vdim, **f32), torch.zeros(2, B, m.heads, m.dim, **f32),
                      torch.zeros(2, B, m.heads, **f32))
        self.acc_in = eng.sums("in", m.w_in.shape[0])
        self.o32 = eng.scratch("o32", B, m.heads, m.vdim, dtype=torch.float32)
        self.y = eng.scratch("o", B, m.heads * m.vdim)

    def prompt_target(self, pages: "_Pages") -> dict:
        return dict(seq_slot=pages.slots, state=self.state)

    def copy_pages(self, dst, src):
        pass

    def copy_slots(self, dst, src):
        S, n, m = self.state
        S.index_copy_(0, dst, S.index_select(0, src))
        n.index_copy_(1, dst, n.index_select(1, src))
        m.index_copy_(1, dst, m.index_select(1, src))

    def step(self, h, out):
        from ..ops import cuda_mixers as K

        e, m = self.e, self.m
        e.gemm(h, m.w_in, self.acc_in)
        K.mlstm_step(self.acc_in, m, e.seq_lens, self.state, self.o32)
        K.mlstm_out(self.o32, self.acc_in[:, m.heads * (2 * m.dim + m.vdim):], m, self.y, clear=self.acc_in)
        e.gemm(self.y, m.o, out)


class _AttentionSlots:
    """Decode side of one ``attention`` or ``attention_2`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li, acc=None, out=None, scale: float = 1.0):
        """A part of another mixer is given its columns ``acc`` of the input projection's sums, those of the output projection's
        operand (``out``) and the factor ``scale`` of its output."""
        from ..ops import cuda_mixers as K

        self.e, self.m = eng, m
        self.own = m.kv_from is None
        if self.own:
            shape = (eng.num_blocks, eng.block_size, m.kv_heads)
            self.k_cache = torch.zeros(*shape, m.dim, dtype=eng.dtype, device=eng.dev)
            self.v_cache = torch.zeros(*shape, m.vdim, dtype=eng.dtype, device=eng.dev)
        else:
            lender = eng.slots[m.kv_from]
            self.k_cache, self.v_cache = lender.k_cache, lender.v_cache
        self.temp = m.temperature.table(eng.max_len + 1, eng.dev) if m.temperature is not None else None
        B = eng.max_seqs
        self.w_in = m.w_in[: m.rows] if acc is None else None
        self.acc_in = eng.sums("in", m.rows) if acc is None else acc
        self.pools, self.scale = {}, scale
        if m.pool:
            shape = (B, eng.max_len // m.pool + 1, m.kv_heads)
            self.pools = dict(pool_k=torch.zeros(*shape, m.dim, dtype=eng.dtype, device=eng.dev),
                              pool_v=torch.zeros(*shape, m.vdim, dtype=eng.dtype, device=eng.dev))
        self.q = eng.scratch("q", B, m.heads, m.dim)
        self.table = m.rope.table(eng.max_len + 1, eng.dev) if m.rot else None
        self.g = eng.scratch("g", B, m.heads * m.vdim) if m.gate == "element" else None
        self.head_gate = eng.scratch("gate", B, m.heads, dtype=torch.float32) if m.gate == "head" else None
        self.o = eng.scratch("o", B, m.heads * m.vdim) if out is None else out
        # tensor-core decode; other sizes and fp32 run the CUDA-core kernel
        self.tc = eng.dtype == torch.bfloat16 and K.grouped_decode_tc_ok(m, eng.block_size)
        self.splits, self.part_o, self.part_ml = 1, None, None
        if self.tc:
            tiles = -(-eng.max_len // 128)
            if m.window:
                tiles = min(tiles, -(-m.window // 128) + 1 + -(-m.keep // 128))
                tiles += -(-max(0, eng.max_len - m.window) // (128 * m.pool)) if m.pool else 0
            self.splits = max(1, min(8, tiles, 148 // K.grouped_decode_tc_items(B, m)))
            if self.splits > 1:
                self.part_o = eng.scratch("part_o", B, m.heads * self.splits * m.vdim, dtype=torch.float32)
                self.part_ml = eng.scratch("part_ml", B, m.heads * self.splits * 2, dtype=torch.float32)

    def prompt_target(self, pages: "_Pages") -> dict:
        if not self.own:
            return {}
        pools = dict(pools=dict(seq_slot=pages.slots, **self.pools)) if self.pools else {}
        return dict(k_cache=self.k_cache, v_cache=self.v_cache, tok_slot=pages.tok_slot, block_table=self.e.block_table,
                    block_size=self.e.block_size, **pools)

    def copy_pages(self, dst, src):
        for c in (self.k_cache, self.v_cache) if self.own else ():
            c.index_copy_(0, dst, c.index_select(0, src))

    def copy_slots(self, dst, src):
        for c in self.pools.values():
            c.index_copy_(0, dst, c.index_select(0, src))

    def prepare(self):
        """``acc_in`` -> queries, gate logits, the new rows of the cache."""
        from ..ops import cuda_mixers as K

        e = self.e
        where = dict(k_cache=self.k_cache, v_cache=self.v_cache, block_table=e.block_table, block_size=e.block_size, pool=self.m.pool,
                     **self.pools) if self.own else {}
        K.attn_prep(self.acc_in, self.m, e.seq_lens, self.temp, table=self.table, q=self.q, g=self.g, head_gate=self.head_gate,
                    **self.m.prep, **where)

    def attend(self):
        from ..ops import cuda_mixers as K

        e = self.e
        args = (self.q, self.k_cache, self.v_cache, self.m, e.seq_lens, e.block_table, e.block_size, self.o, self.g)
        how = dict(head_gate=self.head_gate, pool=self.m.pool, out_scale=self.scale, **self.pools, **self.m.sight)
        if self.tc:
            K.grouped_decode_tc(*args, self.splits, self.part_o, self.part_ml, **how)
        else:
            K.grouped_decode(*args, **how)

    def mix(self):
        """Sums of the input projection -> operand of the output projection."""
        self.prepare()
        self.attend()

    def step(self, h, out):
        self.e.gemm(h, self.w_in, self.acc_in)
        self.mix()
        self.e.gemm(self.o, self.m.o, out)


class _RgLruSlots:
    """Decode side of one ``rglru`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li):
        from ..ops import cuda_mixers as K

        self.e, self.m = eng, m
        B, f32 = eng.max_seqs, dict(dtype=torch.float32, device=eng.dev)
        self.state = torch.zeros(B, m.width, **f32)
        self.conv_state = torch.zeros(B, m.taps - 1, m.width, **f32)
        self.acc_in = eng.sums("in", 2 * m.width)
        self.u = eng.scratch("u", B, m.width)
        self.y = eng.scratch("o", B, m.width)
        self.tc = eng.dtype == torch.bfloat16 and K.rglru_tc_ok(m)

    def prompt_target(self, pages: "_Pages") -> dict:
        return dict(seq_slot=pages.slots, state=self.state, conv_state=self.conv_state)

    def copy_pages(self, dst, src):
        pass

    def copy_slots(self, dst, src):
        for t in (self.state, self.conv_state):
            t.index_copy_(0, dst, t.index_select(0, src))

    def convolve(self):
        from ..ops import cuda_mixers as K

        K.conv_step(self.acc_in[:, self.m.width:], self.m, self.e.seq_lens, self.conv_state, self.u)

    def recur(self):
        from ..ops import cuda_mixers as K

        args = (self.u, self.acc_in[:, : self.m.width], self.m, self.e.seq_lens, self.state, self.y)
        if self.tc:
            K.rglru_step_tc(*args)
        else:
            K.rglru_step(mx.block_gates(self.u, self.m.gates), *args)

    def step(self, h, out):
        self.e.gemm(h, self.m.w_in, self.acc_in)
        self.convolve()
        self.recur()
        self.e.gemm(self.y, self.m.o, out)


class _HGrn2Slots:
    """Decode side of one ``hgrn2`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li, acc=None, out=None, scale: float = 1.0):
        """As :class:`_AttentionSlots`."""
        self.e, self.m, self.scale = eng, m, scale
        self.state = torch.zeros(eng.max_seqs, m.heads, m.dim, m.vdim, dtype=torch.float32, device=eng.dev)
        self.acc_in = eng.sums("in", sum(m.parts)) if acc is None else acc
        self.y = eng.scratch("o", eng.max_seqs, m.out_width) if out is None else out

    def prompt_target(self, pages: "_Pages") -> dict:
        return dict(seq_slot=pages.slots, state=self.state)

    def copy_pages(self, dst, src):
        pass

    def copy_slots(self, dst, src):
        self.state.index_copy_(0, dst, self.state.index_select(0, src))

    def mix(self):
        from ..ops import cuda_mixers as K

        K.hgrn2_step(self.acc_in, self.m, self.e.seq_lens, self.state, self.y, self.scale)

    def step(self, h, out):
        self.e.gemm(h, self.m.w_in, self.acc_in)
        self.mix()
        self.e.gemm(self.y, self.m.o, out)


class _ParallelSlots:
    """Decode side of one ``parallel`` layer: one product in front of both halves, one behind them."""

    def __init__(self, eng: "LayeredRolloutEngine", m, li):
        self.e, self.m = eng, m
        a, b = m.left.rows, m.left.out_width
        self.acc_in = eng.sums("in", m.w_in.shape[0])
        self.o = eng.scratch("o", eng.max_seqs, m.o.shape[1])
        self.left = SLOTS[m.left.kind](eng, m.left, li, self.acc_in[:, :a], self.o[:, :b], m.scales[0])
        self.right = SLOTS[m.right.kind](eng, m.right, li, self.acc_in[:, a:], self.o[:, b:], m.scales[1])

    def prompt_target(self, pages: "_Pages") -> dict:
        return dict(left=self.left.prompt_target(pages), right=self.right.prompt_target(pages))

    def copy_pages(self, dst, src):
        self.left.copy_pages(dst, src)
        self.right.copy_pages(dst, src)

    def copy_slots(self, dst, src):
        self.left.copy_slots(dst, src)
        self.right.copy_slots(dst, src)

    def step(self, h, out):
        self.e.gemm(h, self.m.w_in, self.acc_in)
        self.left.mix()
        self.right.mix()
        self.e.gemm(self.o, self.m.o, out)


SLOTS = {"latent_attention": _LatentSlots, "mlstm": _MLstmSlots, "attention": _AttentionSlots, "attention_2": _AttentionSlots,
         "rglru": _RgLruSlots, "hgrn2": _HGrn2Slots, "parallel": _ParallelSlots}


class _Pages:
    """``ctx.kv`` of a prompt forward: where layer ``li`` leaves its keys and values or its final state."""

    def __init__(self, eng, tok_slot, slots):
        self.e, self.tok_slot, self.slots = eng, tok_slot, slots

    def paged_cache(self, li):
        return self.e.slots[li].prompt_target(self)

    recurrent_state = paged_cache

    def last_tokens(self):
        return dict(tok_slot=self.tok_slot, prev=self.e.last_token)


class LayeredRolloutEngine(RolloutEngine):
    stateful = True

    def _check_model(self, max_model_len, block_size):
        if self.tp != 1:
            raise NotImplementedError("tensor-parallel decode of layered decoders")
        self.dtype = self.model.dtype
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise NotImplementedError(f"layered decoders are served in bfloat16 or float32, not {self.dtype}")
        return block_size or 64

    # ---- buffers: every layer of the list runs after the other, so they share activations -----------------
    def sums(self, name: str, n: int) -> torch.Tensor:
        """[max_seqs, n] fp32 accumulator, a view of the widest one asked for under ``name``; zero between steps."""
        return self._view(("sums", name), torch.float32, n)

    def scratch(self, name: str, *shape, dtype=None) -> torch.Tensor:
        n = 1
        for s in shape[1:]:
            n *= s
        return self._view((name,), dtype or self.dtype, n).view(shape)

    def _view(self, key, dtype, n):
        key = key + (dtype, n)
        if key not in self._buffers:
            self._buffers[key] = torch.zeros(self.max_seqs, n, dtype=dtype, device=self.dev)
        return self._buffers[key]

    def _alloc_layers(self, kv_splits):
        cfg, B, H = self.cfg, self.max_seqs, self.cfg.hidden_size
        self._buffers: dict = {}
        # weight-streaming GEMM: bf16, at most 128 rows, rows of 16 bytes; other shapes and fp32 use the library
        self._own_gemm = (os.environ.get("TRL_B200_DECODE_GEMM", "own") != "cublas" and self.dtype == torch.bfloat16
                          and B <= 128)
        self.last_token = torch.zeros(B, dtype=torch.int64, device=self.dev) if cfg.pairs else None
        self.slots: list = []  # a layer may look up an earlier one
        for li, (s, l) in enumerate(zip(cfg.layers, self.model.layers)):
            self.slots.append(SLOTS[s.kind](self, l.mixer, li))
        self._x = torch.zeros(B, H, dtype=torch.float32, device=self.dev)
        self._acc = self.sums("out", H)
        self._h = self.scratch("h", B, H)
        self._h2 = torch.zeros_like(self._h) if any(l.beside for l in self.model.layers) else None
        self._first = torch.zeros_like(self._x) if cfg.passes > 1 else None  # the embedding, which a loop adds again
        self._logits_buf = torch.zeros(B, cfg.vocab_size, dtype=self.dtype, device=self.dev)

    def _reset_sums(self):
        for key, t in self._buffers.items():
            if key[0] == "sums":
                t.zero_()

    def _copy_pages(self, dst, src):
        for s in self.slots:
            s.copy_pages(dst, src)

    def _copy_slots(self, dst, src):
        for s in self.slots:
            s.copy_slots(dst, src)
        if self.last_token is not None:
            self.last_token[dst] = self.last_token[src]

    def _head(self, hidden):
        return mx.linear(hidden, self.model.lm_head_weight)

    def _page_writer(self, tok_slot, ctx: SeqCtx, slots):
        return _Pages(self, tok_slot, slots)

    def _prefill_again(self, owners, pixels=None):
        # a recurrent state after the prompt exists nowhere any more: run the prompt into the new slot
        return self._prefill(owners, pixels)

    # ---- one decode step ------------------------------------------------------------------------------------
    def gemm(self, x, w, acc):
        """``acc`` (fp32, zeros) = ``x w^T``."""
        if self._own_gemm and x.shape[1] % 8 == 0:
            from ..ops import cuda as K

            K.decode_gemm(x, w, y32=acc)
        else:
            acc.copy_(mx.linear_f32(x, w))

    def _decode_logits(self):
        from ..ops import cuda as K

        was = K.set_pdl(self._pdl)
        try:
            return self._decode_layers()
        finally:
            K.set_pdl(was)

    def _decode_layers(self):
        from ..ops import cuda as K
        from ..ops import cuda_mixers as KM

        m, x, h, acc = self.model, self._x, self._h, self._acc
        if m.embed_norm is not None:
            n = m.embed_norm
            KM.embed_normed(self.next_input, m.embed_tokens, self.cfg.embed_scale, n.weight, n.eps, n.shift, out=x, copy=self._first)
        elif m.pair_embed is None:
            KM.embed_scaled(self.next_input, m.embed_tokens, self.cfg.embed_scale, out=x)
        else:
            p = self.cfg.pairs
            KM.embed_pairs(self.next_input, m.embed_tokens, self.cfg.embed_scale, m.pair_embed, p["mul_prev"], p["mul_cur"], self.seq_lens,
                           prev=self.last_token, decode=True, out=x)
        delta = post = None  # sums not yet added to the stream, and the norm they pass first
        now = dict(clear=True, out=h)
        for li, (layer, slots) in enumerate(zip(m.layers, self.slots)):
            if layer.beside:
                layer.read_both(x, delta, post, **now, out2=self._h2, **m.entrance(li, self._first))
                rows = None if layer.mlp is None else self.experts(self._h2, layer.mlp)
                slots.step(h, acc)
                delta, post = acc if rows is None else (acc, rows), None
                continue
            layer.read_mixer(x, delta, post, **now, **m.entrance(li, self._first))
            slots.step(h, acc)
            delta, post = acc, layer.norm1b
            if layer.mlp is not None:
                layer.read_mlp(x, delta, post, **now)
                if isinstance(layer.mlp, ExpertMlp):
                    self.experts(h, layer.mlp, acc)
                else:
                    self.gemm(self.mlp_act(h, layer.mlp), layer.mlp.down, acc)
                post = layer.norm2b
            if layer.side is not None:
                layer.read_side(x, delta, post, **now)
                self.gemm(self.side_act(h, layer.side, li), layer.side.proj, acc)
                post = layer.side.norm
        m.norm(x, self.dtype, delta, post, **now)
        if self._own_gemm and h.shape[1] % 8 == 0:
            return K.decode_gemm(h, m.lm_head_weight, out=self._logits_buf)
        return mx.linear(h, m.lm_head_weight)

    def mlp_act(self, h, mlp):
        """Activation of a feed-forward: fused into the product where the weight-streaming kernel runs."""
        from ..ops import cuda as K

        act = self.scratch("act", self.max_seqs, mlp.down.shape[1])
        if self._own_gemm and h.shape[1] % 8 == 0:
            return K.decode_gemm(h, mlp.w_in, out=act, **mlp.fused)
        return mlp.act(mx.linear(h, mlp.w_in), out=act)

    def experts(self, h, mlp, out=None):
        """Mixture of experts of the slots that are live; ``out`` (fp32) is stored to.  Without it the experts' rows are returned,
        not yet added up."""
        z = self.sums("router", mlp.n)
        self.gemm(h, mlp.router, z)
        return mx.experts(mlp, h, positions=self.seq_lens, logits=z, out=out, summed=out is not None)

    def side_act(self, h, side, li):
        from ..ops import cuda_mixers as KM

        z = self.sums("side", side.dim)
        self.gemm(h, side.gate, z)
        return KM.side_gate(z, self.next_input, self.model.side_embed, li * side.dim, clear=True,
                            out=self.scratch("side_act", self.max_seqs, side.dim))
