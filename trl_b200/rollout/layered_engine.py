"""Serving of the layered decoders (models/layered.py): scheduler, slots, pages, sampling and CUDA-graph decode are
:class:`~trl_b200.rollout.engine.RolloutEngine`'s; this module adds what a layer keeps between tokens and how it takes
one token further.

Every layer of the list has a cache of its own, also one that runs with another layer's weights:

    latent_attention   pages of latent rows ``[kv_rank | rotated key]`` behind the engine's block table (the window is a
                       mask: pages stay until the sequence ends)
    mlstm              per slot an fp32 matrix state, its normaliser and running maximum

A decode step is one graph: embed, then per layer norm (+ residual) -> input projection -> mixer -> output projection
-> norm (+ residual) -> up / GELU -> down, then final norm, head and sampler.  With bf16 weights the projections are
the weight-streaming tcgen05 kernel; their fp32 sums are consumed and cleared by the next kernel.  fp32 models run the
same kernels' fp32 forms with library fp32 matrix products."""
from __future__ import annotations

import os

import torch

from ..models.decoder import SeqCtx
from ..ops import mixers as mx
from .engine import RolloutEngine


class _LatentSlots:
    """Decode side of one ``latent_attention`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m):
        from ..ops import cuda_mixers as K

        self.e, self.m = eng, m
        self.kr, self.width = K.latent_row(m.kv_rank, m.rot_dim)
        self.cache = torch.zeros(eng.num_blocks, eng.block_size, self.width, dtype=eng.dtype, device=eng.dev)
        self.table = m.rope.table(eng.max_len + 1, eng.dev)
        B = eng.max_seqs
        self.acc_in = eng.sums("in", m.w_in.shape[0])
        self.acc_q = eng.sums("q", m.uq.shape[0])
        self.cq = eng.scratch("cq", B, m.q_rank)
        self.gate = eng.scratch("gate", B, m.heads, dtype=torch.float32)
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
        K.latent_prep(self.acc_in, m, e.seq_lens, self.table, clear=True, cq=self.cq, gate=self.gate, cache=self.cache,
                      block_table=e.block_table, block_size=e.block_size)
        e.gemm(self.cq, m.uq, self.acc_q)
        self.absorb()
        self.attend()
        self.expand()
        e.gemm(self.o, m.o, out)


class _MLstmSlots:
    """Decode side of one ``mlstm`` layer."""

    def __init__(self, eng: "LayeredRolloutEngine", m):
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


SLOTS = {"latent_attention": _LatentSlots, "mlstm": _MLstmSlots}


class _Pages:
    """``ctx.kv`` of a prompt forward: where layer ``li`` leaves its latents or its final state."""

    def __init__(self, eng, tok_slot, slots):
        self.e, self.tok_slot, self.slots = eng, tok_slot, slots

    def latent_cache(self, li):
        return self.e.slots[li].prompt_target(self)

    recurrent_state = latent_cache


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
        self.slots = [SLOTS[s.kind](self, l.mixer) for s, l in zip(cfg.layers, self.model.layers)]
        self._x = torch.zeros(B, H, dtype=torch.float32, device=self.dev)
        self._acc = self.sums("out", H)
        self._h = self.scratch("h", B, H)
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
        KM.embed_scaled(self.next_input, m.embed_tokens, self.cfg.embed_scale, out=x)

        def norm(n, delta):
            KM.dynamic_tanh(x, delta, n.alpha, n.weight, n.bias, self.dtype, clear=True, out=h)

        delta = None
        for layer, slots in zip(m.layers, self.slots):
            norm(layer.norm1, delta)
            slots.step(h, acc)
            delta = acc
            if layer.mlp is not None:
                norm(layer.norm2, delta)
                self.gemm(self._up_gelu(h, layer.mlp), layer.mlp.down, acc)
        norm(m.norm, delta)
        if self._own_gemm and h.shape[1] % 8 == 0:
            return K.decode_gemm(h, m.lm_head_weight, out=self._logits_buf)
        return mx.linear(h, m.lm_head_weight)

    def _up_gelu(self, h, mlp):
        from ..ops import cuda_mixers as KM

        act = self.scratch("act", self.max_seqs, mlp.up.shape[0])
        if self._own_gemm and h.shape[1] % 8 == 0:
            from ..ops import cuda as K

            return K.decode_gemm(h, mlp.up, out=act, gelu=True)
        return KM.gelu_erf(mx.linear(h, mlp.up), out=act)
