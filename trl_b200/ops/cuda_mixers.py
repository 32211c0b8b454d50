"""ctypes bindings of ``csrc/mixers.cu`` and of the tensor-core mixer kernels (inference only).

``model dtype`` below is bf16 or fp32; accumulators, gates, states and norms are fp32 in both."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong

import torch

from .cuda import _chk, _p, _s, lib, status_buffer


def _b(t) -> c_int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"layered decoders run in bfloat16 or float32, not {t.dtype}")
    return c_int(int(t.dtype == torch.bfloat16))


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


def latent_row(kv_rank: int, rot: int) -> tuple[int, int]:
    """(offset of the rotated part, width) of a latent row ``[kv_rank | pad | rot | pad]``: both parts start on 16 bytes."""
    return round8(kv_rank), round8(kv_rank) + round8(rot)


def embed_scaled(ids, emb, scale, out=None):
    T, (V, H) = ids.numel(), emb.shape
    out = torch.empty(T, H, dtype=torch.float32, device=emb.device) if out is None else out
    assert ids.dtype == torch.int64 and ids.is_contiguous() and emb.is_contiguous()
    _chk(lib().trlb_embed_scaled(_p(ids), _p(emb), _p(out), c_int(T), c_int(H), c_int(V), c_float(scale), _b(emb), _s()),
         "embed_scaled")
    return out


def dynamic_tanh(x, delta, alpha, w, b, dtype, clear=False, out=None):
    """``x += delta`` (in place; with ``clear`` delta is zeroed), returns ``tanh(alpha x) w + b`` in ``dtype``."""
    T, H = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and (delta is None or (delta.dtype == torch.float32
                                                                               and delta.is_contiguous()))
    out = torch.empty(T, H, dtype=dtype, device=x.device) if out is None else out
    _chk(lib().trlb_dynamic_tanh(_p(x), _p(delta), _p(alpha), _p(w), _p(b), _p(out), c_int(T), c_int(H), c_int(int(clear)),
                                 _b(out), _s()), "dynamic_tanh")
    return out


def gelu_erf(z, out=None):
    assert z.is_contiguous()
    out = torch.empty_like(z) if out is None else out
    _chk(lib().trlb_gelu_erf(_p(z), _p(out), c_longlong(z.numel()), _b(z), _s()), "gelu_erf")
    return out


def latent_prep(acc, m, positions, table, *, clear=False, tok_slot=None, cq=None, lat=None, gate=None, cache=None,
                block_table=None, block_size=0):
    """From the sums of a layer's input projection: normed query latent, latent row (dense and / or appended to the
    paged cache), sigmoid gates."""
    rows = acc.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    dt = m.o.dtype
    assert acc.dtype == torch.float32 and acc.stride(1) == 1 and positions.dtype == torch.int32
    cq = torch.empty(rows, m.q_rank, dtype=dt, device=acc.device) if cq is None else cq
    gate = torch.empty(rows, m.heads, dtype=torch.float32, device=acc.device) if gate is None else gate
    mb = 0 if block_table is None else block_table.shape[1]
    _chk(lib().trlb_latent_prep(_p(acc), c_longlong(acc.stride(0)), c_int(rows), c_int(m.q_rank), c_int(m.kv_rank),
                                c_int(m.rot_dim), c_int(m.heads), c_int(int(clear)), _p(m.q_norm), _p(m.kv_norm),
                                c_float(m.eps), _p(positions), _p(tok_slot), _p(table), c_int(table.shape[0]), _p(cq),
                                _p(lat), _p(gate), c_int(kr), c_int(w), _p(cache), _p(block_table), c_int(mb),
                                c_int(block_size), _b(cq), _s()), "latent_prep")
    return cq, gate


def rotate_q(q, m, positions, table):
    rows = q.shape[0]
    assert q.is_contiguous()
    _chk(lib().trlb_rotate_q(_p(q), c_int(rows), c_int(m.heads), c_int(m.dim), c_int(m.rot_dim), _p(positions), _p(table),
                             c_int(table.shape[0]), _b(q), _s()), "rotate_q")


def latent_prompt(q, kv, lat, m, positions, gate):
    """Windowed sink attention of packed prompts on the CUDA cores: any size, bf16 or fp32."""
    T = q.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    out = torch.empty(T, m.heads * m.vdim, dtype=q.dtype, device=q.device)
    assert q.is_contiguous() and kv.stride(1) == 1 and lat.is_contiguous()
    _chk(lib().trlb_latent_prompt(_p(q), _p(kv), c_longlong(kv.stride(0)), _p(lat), c_int(T), c_int(m.heads), c_int(m.dim),
                                  c_int(m.rot_dim), c_int(m.vdim), c_int(kr), c_int(w), c_int(m.window or 0),
                                  c_float(m.scale), _p(positions), _p(m.sink), _p(gate), _p(out), _b(q), _s()),
         "latent_prompt")
    return out


def latent_prompt_tc_ok(m) -> bool:
    return m.scale > 0 and bool(lib().trlb_latent_attn_tc_ok(c_int(m.heads), c_int(m.dim), c_int(m.rot_dim), c_int(m.vdim)))


def latent_prompt_tc(q, kv, lat, m, cu, gate):
    """:func:`latent_prompt` on the tensor cores (bf16; see ``latent_prompt_tc_ok``); ``cu`` int32 sequence starts."""
    T = q.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    out = torch.empty(T, m.heads * m.vdim, dtype=q.dtype, device=q.device)
    assert q.dtype == torch.bfloat16 and q.is_contiguous() and kv.stride(1) == 1 and lat.is_contiguous() and cu.dtype == torch.int32
    _chk(lib().trlb_latent_attn_tc(_p(q), _p(kv), c_longlong(kv.stride(0)), _p(lat[:, kr:]), c_longlong(w), _p(cu),
                                   c_int(cu.numel() - 1), c_int(T), c_int(m.heads), c_int(m.dim), c_int(m.rot_dim),
                                   c_int(m.vdim), c_int(m.window or 0), c_float(m.scale), _p(m.sink), _p(gate), _p(out),
                                   _p(status_buffer(q.device)), _s()), "latent_attn_tc")
    return out


def latent_absorb(qacc, m, positions, table, q_lat, clear):
    B = qacc.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    _chk(lib().trlb_latent_absorb(_p(qacc), c_longlong(qacc.stride(0)), _p(m.uk), _p(q_lat), c_int(B), c_int(m.heads),
                                  c_int(m.dim), c_int(m.rot_dim), c_int(m.kv_rank), c_int(kr), c_int(w), _p(positions),
                                  _p(table), c_int(table.shape[0]), c_int(int(clear)), _b(q_lat), _s()), "latent_absorb")


def latent_decode(q_lat, cache, m, seq_lens, block_table, block_size, o_lat):
    B = q_lat.shape[0]
    _, w = latent_row(m.kv_rank, m.rot_dim)
    _chk(lib().trlb_latent_decode(_p(q_lat), _p(cache), _p(o_lat), c_int(B), c_int(m.heads), c_int(m.kv_rank), c_int(w),
                                  c_int(m.window or 0), c_float(m.scale), _p(seq_lens), _p(block_table),
                                  c_int(block_table.shape[1]), c_int(block_size), _p(m.sink), _b(q_lat), _s()),
         "latent_decode")


def latent_expand(o_lat, m, gate, positions, out):
    B = o_lat.shape[0]
    _chk(lib().trlb_latent_expand(_p(o_lat), _p(m.uv), _p(gate), _p(out), c_int(B), c_int(m.heads), c_int(m.vdim),
                                  c_int(m.kv_rank), _p(positions), _b(out), _s()), "latent_expand")


def latent_decode_tc_ok(m, block_size: int) -> bool:
    """Whether :func:`latent_decode_tc` and :func:`head_gemm` serve a mixer's sizes (else the CUDA-core kernels do)."""
    _, w = latent_row(m.kv_rank, m.rot_dim)
    return m.scale > 0 and bool(lib().trlb_latent_decode_tc_ok(c_int(m.heads), c_int(m.dim), c_int(m.rot_dim), c_int(m.vdim),
                                                 c_int(m.kv_rank), c_int(w), c_int(block_size)))


def latent_decode_tc(q_lat, cache, m, seq_lens, block_table, block_size, o_lat, part_o, part_ml, splits):
    """:func:`latent_decode` on the tensor cores (bf16).  ``part_o`` [>= B heads splits kv_rank] and ``part_ml`` [>= 2 B heads
    splits] fp32 scratch."""
    B = q_lat.shape[0]
    _, w = latent_row(m.kv_rank, m.rot_dim)
    assert q_lat.dtype == torch.bfloat16 and cache.is_contiguous() and cache.shape[1] == block_size and cache.shape[2] == w
    assert part_o.numel() >= B * m.heads * splits * m.kv_rank and part_ml.numel() >= 2 * B * m.heads * splits
    _chk(lib().trlb_latent_decode_tc(_p(q_lat), _p(cache), c_int(cache.shape[0]), c_int(B), c_int(m.heads), c_int(m.kv_rank),
                                     c_int(w), c_int(m.window or 0), c_float(m.scale), _p(seq_lens),
                                     _p(block_table), c_int(block_table.shape[1]), c_int(block_size), _p(m.sink),
                                     c_int(splits), _p(part_o), _p(part_ml), _p(o_lat), _p(status_buffer(q_lat.device)), _s()),
         "latent_decode_tc")


def latent_query(qacc, m, positions, table, q, q_lat):
    """fp32 query sums (cleared) -> bf16 ``q`` and the rotated part of ``q_lat``."""
    B = qacc.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    _chk(lib().trlb_latent_query(_p(qacc), c_longlong(qacc.stride(0)), _p(q), _p(q_lat), c_int(B), c_int(m.heads), c_int(m.dim),
                                 c_int(m.rot_dim), c_int(kr), c_int(w), _p(positions), _p(table), c_int(table.shape[0]), _s()),
         "latent_query")


def head_gemm(x, w, y, *, w_mn: bool = False, scale=None):
    """``y[b, h] = scale[b, h] * x[b, h] w[h]^T`` per head: x [B, heads, >= K] (last dim dense), w [heads, M, K], or [heads, K,
    M] with ``w_mn`` (read MN-major, nothing is transposed in memory); y [B, heads, >= M] bf16."""
    (B, H), (_, a, b) = x.shape[:2], w.shape
    M, Kd = (b, a) if w_mn else (a, b)
    assert x.dtype == y.dtype == w.dtype == torch.bfloat16 and w.is_contiguous() and x.stride(2) == 1 and y.stride(2) == 1
    assert x.shape[2] >= Kd and y.shape[2] >= M and (scale is None or (scale.is_contiguous() and scale.shape == (B, H)))
    _chk(lib().trlb_head_gemm(_p(x), c_longlong(x.stride(0)), c_longlong(x.stride(1)), _p(w), c_int(int(w_mn)), _p(y),
                              c_longlong(y.stride(0)), c_longlong(y.stride(1)), _p(scale), c_int(B), c_int(H), c_int(M),
                              c_int(Kd), _p(status_buffer(x.device)), _s()), "head_gemm")
    return y


def mlstm_gates(z, bias, cap, heads):
    T = z.shape[0]
    assert z.is_contiguous()
    ig = torch.empty(T, heads, dtype=torch.float32, device=z.device)
    fg = torch.empty_like(ig)
    _chk(lib().trlb_mlstm_gates(_p(z), _p(bias), c_float(cap), c_int(T), c_int(heads), _p(ig), _p(fg), _s()), "mlstm_gates")
    return ig, fg


def mlstm_prompt(y, m, ig, fg, cu, seq_slot=None, state=None):
    """Token-by-token form for packed prompts; ``state`` (S, n, m) of ``seq_slot`` gets the final state."""
    T = y.shape[0]
    out = torch.empty(T, m.heads, m.vdim, dtype=torch.float32, device=y.device)
    S, n, mm = state if state is not None else (None, None, None)
    qd = m.heads * m.dim
    _chk(lib().trlb_mlstm_prompt(_p(y), c_longlong(y.stride(0)), c_int(qd), c_int(2 * qd), _p(ig), _p(fg), _p(cu),
                                 c_int(cu.numel() - 1), _p(seq_slot if state is not None else None), _p(S), _p(n), _p(mm),
                                 c_int(0 if S is None else S.shape[0]), c_int(m.heads), c_int(m.dim), c_int(m.vdim),
                                 c_float(m.dim ** -0.5), _p(out), _b(y), _s()), "mlstm_prompt")
    return out


def mlstm_chunk_ok(m) -> bool:
    return bool(lib().trlb_mlstm_chunk_ok(c_int(m.heads), c_int(m.dim), c_int(m.vdim)))


def mlstm_chunk(y, m, ig, fg, cu, seq_slot=None, state=None):
    """:func:`mlstm_prompt` in 128-token chunks on the tensor cores (bf16; see ``mlstm_chunk_ok``)."""
    T, H, n_seq = y.shape[0], m.heads, cu.numel() - 1
    assert y.dtype == torch.bfloat16 and y.stride(1) == 1 and cu.dtype == torch.int32
    chunks = int(lib().trlb_mlstm_chunks(c_int(T), c_int(n_seq)))
    f32 = dict(dtype=torch.float32, device=y.device)
    out = torch.empty(T, H, m.vdim, **f32)
    bgm, n_in = torch.empty(3, H, T, **f32), torch.empty(chunks, H, m.dim, **f32)
    parts = torch.empty(2, chunks, H, m.dim, m.vdim, dtype=torch.bfloat16, device=y.device)
    S, n, mm = state if state is not None else (None, None, None)
    qd = H * m.dim
    _chk(lib().trlb_mlstm_chunk(_p(y), c_longlong(y.stride(0)), c_int(qd), c_int(2 * qd), _p(ig), _p(fg), _p(cu), c_int(n_seq),
                                c_int(T), _p(seq_slot if state is not None else None), _p(S), _p(n), _p(mm),
                                c_int(0 if S is None else S.shape[0]), c_int(H), c_int(m.dim), c_int(m.vdim),
                                c_float(m.dim ** -0.5), _p(bgm[0]), _p(bgm[1]), _p(bgm[2]), _p(n_in), _p(parts[0]),
                                _p(parts[1]), _p(out), _p(status_buffer(y.device)), _s()), "mlstm_chunk")
    return out


def mlstm_step(acc, m, seq_lens, state, out):
    B = acc.shape[0]
    S, n, mm = state
    _chk(lib().trlb_mlstm_step(_p(acc), c_longlong(acc.stride(0)), _p(m.gate_bias), c_float(m.cap), _p(seq_lens), _p(S),
                               _p(n), _p(mm), c_int(S.shape[0]), c_int(B), c_int(m.heads), c_int(m.dim), c_int(m.vdim),
                               c_float(m.dim ** -0.5), _p(out), _s()), "mlstm_step")


def mlstm_out(o, g, m, out, clear=None):
    """``unit_rms(o) * norm * sigmoid(g)``; ``clear``: fp32 row sums (laid out like the input projection) to zero."""
    rows = o.shape[0]
    assert g.stride(1) == 1
    _chk(lib().trlb_mlstm_out(_p(o), _p(g), c_longlong(g.stride(0)), _b(g), _p(m.norm), c_float(m.eps), c_int(rows),
                              c_int(m.heads), c_int(m.vdim), _p(out), _b(out), _p(clear),
                              c_longlong(0 if clear is None else clear.stride(0)),
                              c_int(m.heads * (2 * m.dim + m.vdim)), _s()), "mlstm_out")
    return out
