"""ctypes bindings of ``csrc/mixers.cu``, ``csrc/grouped_attn.cu``, ``csrc/rglru.cu``, ``csrc/hgrn2.cu``, ``csrc/layered_moe.cu``
and of the tensor-core mixer kernels (inference only).

``model dtype`` below is bf16 or fp32; accumulators, gates, states and norms are fp32 in both."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong

import torch

from .cuda import _chk, _p, _s, lib, status_buffer


def _b(t) -> c_int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"layered decoders run in bfloat16 or float32, not {t.dtype}")
    return c_int(int(t.dtype == torch.bfloat16))


def _len(table) -> c_int:
    """Entries of a table by position (none: a mixer without one)."""
    return c_int(0 if table is None else table.shape[0])


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


def embed_normed(ids, emb, scale, w, eps, shift=0.0, out=None, copy=None):
    """fp32 ``emb[ids] * scale`` over its rms times ``shift + w``; ``copy`` gets it too."""
    T, (V, H) = ids.numel(), emb.shape
    out = torch.empty(T, H, dtype=torch.float32, device=emb.device) if out is None else out
    assert ids.dtype == torch.int64 and ids.is_contiguous() and emb.is_contiguous() and (copy is None or copy.shape == out.shape)
    _chk(lib().trlb_embed_normed(_p(ids), _p(emb), _p(w), _p(out), _p(copy), c_int(T), c_int(H), c_int(V), c_float(scale), c_float(eps),
                                 c_float(shift), _b(emb), _s()), "embed_normed")
    return out


def embed_pairs(ids, emb, scale, pairs, mul_prev, mul_cur, positions, tok_slot=None, prev=None, decode=False, out=None):
    """``emb[ids] * scale + pairs[row]`` with the row ``(previous * mul_prev + current * mul_cur) mod buckets`` of a table of
    ``buckets`` + 1 rows, the last one at position 0.  Prompts: ``prev`` (int64 by slot) gets every sequence's last token; decode:
    one row per slot, ``prev`` is the previous token and moves on where the position is not negative."""
    T, (V, H) = ids.numel(), emb.shape
    out = torch.empty(T, H, dtype=torch.float32, device=emb.device) if out is None else out
    assert ids.dtype == torch.int64 and ids.is_contiguous() and emb.is_contiguous() and pairs.is_contiguous()
    assert pairs.dtype == emb.dtype and pairs.shape[1] == H and positions.dtype == torch.int32 and positions.numel() >= T
    assert prev is None or prev.dtype == torch.int64
    _chk(lib().trlb_embed_pairs(_p(ids), _p(emb), _p(pairs), _p(out), c_int(T), c_int(H), c_int(V), c_float(scale), c_longlong(mul_prev),
                                c_longlong(mul_cur), c_longlong(pairs.shape[0] - 1), _p(positions), _p(tok_slot), _p(prev),
                                c_int(int(decode)), _b(emb), _s()), "embed_pairs")
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


def rms_residual(x, delta, post, w, eps, dtype, clear=False, out=None, shift=0.0, post_scale=None, gain=1.0, mult=1.0, anchor=None,
                 bump=None, w2=None, out2=None):
    """``x += mult * delta`` or, with ``post``, ``x += mult * delta / rms(delta) * (shift + post) * post_scale``, and ``x += anchor +
    bump`` (in place; with ``clear`` delta, of a pair the first one, is zeroed); returns ``x / rms(x) * (shift + w) * gain`` in
    ``dtype``, or ``x`` itself without ``w``, or with ``w2`` a pair.  ``delta``: a tensor, two, or a tensor and
    :class:`~trl_b200.ops.mixers.ExpertRows`."""
    T, H = x.shape

    def f32(t):
        return t is None or (t.dtype == torch.float32 and t.is_contiguous())

    more = y = row = weight = None
    if isinstance(delta, tuple):
        delta, more = delta
        if not isinstance(more, torch.Tensor):
            (y, row, weight), more = more, None
    assert x.dtype == torch.float32 and x.is_contiguous() and f32(delta) and f32(more) and f32(anchor) and f32(bump)
    assert y is None or (y.dtype == dtype and y.is_contiguous() and row.shape == weight.shape and row.shape[0] == T and y.shape[1] == H)
    out = torch.empty(T, H, dtype=dtype, device=x.device) if out is None else out
    if w2 is not None and out2 is None:
        out2 = torch.empty_like(out)
    _chk(lib().trlb_rms_residual(_p(x), _p(delta), _p(post), _p(post_scale), _p(w), _p(out), c_int(T), c_int(H), c_float(eps),
                                 c_float(shift), c_float(gain), c_float(mult), c_int(int(clear)), _p(more), _p(y), _p(row), _p(weight),
                                 c_int(0 if y is None else row.shape[1]), _p(anchor), _p(bump), _p(w2), _p(out2), _b(out), _s()), "rms_residual")
    return out if w2 is None else (out, out2)


def clamped_glu(z, limit, alpha, shift, out=None):
    """z [rows, 2n] = gate | up -> ``g sigmoid(alpha g) (u + shift)``, ``g = min(gate, limit)``, u = up within +- limit."""
    rows, n = z.shape[0], z.shape[1] // 2
    assert z.is_contiguous()
    out = torch.empty(rows, n, dtype=z.dtype, device=z.device) if out is None else out
    _chk(lib().trlb_clamped_glu(_p(z), _p(out), c_int(rows), c_int(n), c_float(limit), c_float(alpha), c_float(shift), _b(z), _s()),
         "clamped_glu")
    return out


def gelu_glu(z, out=None):
    """z [rows, 2n] = gate | up -> ``gelu_tanh(gate) * up``."""
    rows, n = z.shape[0], z.shape[1] // 2
    assert z.is_contiguous()
    out = torch.empty(rows, n, dtype=z.dtype, device=z.device) if out is None else out
    _chk(lib().trlb_gelu_glu(_p(z), _p(out), c_int(rows), c_int(n), _b(z), _s()), "gelu_glu")
    return out


def side_gate(z, ids, table, off, clear=False, out=None):
    """``gelu_tanh(z) * table[ids, off : off + n]`` in the dtype of the table; z [rows, n] fp32 or of that dtype."""
    rows, n = z.shape
    assert z.is_contiguous() and ids.dtype == torch.int64 and ids.is_contiguous() and table.is_contiguous() and off + n <= table.shape[1]
    assert z.dtype in (torch.float32, table.dtype)
    out = torch.empty(rows, n, dtype=table.dtype, device=z.device) if out is None else out
    _chk(lib().trlb_side_gate(_p(z), c_int(int(z.dtype == torch.float32)), _p(ids), _p(table), c_longlong(table.shape[1]), c_int(off),
                              c_int(rows), c_int(n), c_int(table.shape[0]), c_int(int(clear)), _p(out), _b(table), _s()), "side_gate")
    return out


def gelu_erf(z, out=None):
    assert z.is_contiguous()
    out = torch.empty_like(z) if out is None else out
    _chk(lib().trlb_gelu_erf(_p(z), _p(out), c_longlong(z.numel()), _b(z), _s()), "gelu_erf")
    return out


def latent_prep(acc, m, positions, table, *, clear=False, tok_slot=None, cq=None, lat=None, gate=None, cache=None,
                block_table=None, block_size=0):
    """From the sums of a layer's input projection (without the query rows of a mixer that has no query latent): normed query
    latent, latent row (dense and / or appended to the paged cache), sigmoid gates; the first and the last may be absent."""
    rows = acc.shape[0]
    gates = m.heads if m.gated else 0
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    dt = m.o.dtype
    assert acc.dtype == torch.float32 and acc.stride(1) == 1 and positions.dtype == torch.int32
    cq = torch.empty(rows, m.q_rank, dtype=dt, device=acc.device) if cq is None and m.q_rank else cq
    gate = torch.empty(rows, gates, dtype=torch.float32, device=acc.device) if gate is None and gates else gate
    mb = 0 if block_table is None else block_table.shape[1]
    _chk(lib().trlb_latent_prep(_p(acc), c_longlong(acc.stride(0)), c_int(rows), c_int(m.q_rank), c_int(m.kv_rank),
                                c_int(m.rot_dim), c_int(gates), c_int(int(clear)), _p(m.q_norm), _p(m.kv_norm),
                                c_float(m.eps), _p(positions), _p(tok_slot), _p(table), _len(table), _p(cq),
                                _p(lat), _p(gate), c_int(kr), c_int(w), _p(cache), _p(block_table), c_int(mb),
                                c_int(block_size), _b(m.o), _s()), "latent_prep")
    return cq, gate


def rotate_q(q, m, positions, table):
    rows = q.shape[0]
    assert q.is_contiguous()
    _chk(lib().trlb_rotate_q(_p(q), c_int(rows), c_int(m.heads), c_int(m.dim), c_int(m.rot_dim), _p(positions), _p(table),
                             c_int(table.shape[0]), _b(q), _s()), "rotate_q")


def mixer_attn_tc_ok(heads, kv_heads, dim, rot, vdim) -> bool:
    """Whether :func:`mixer_attn` runs bf16 prompts of these sizes on the tensor cores."""
    return bool(lib().trlb_mixer_attn_tc_ok(c_int(heads), c_int(kv_heads), c_int(dim), c_int(rot), c_int(vdim)))


def mixer_attn(q, k, v, *, heads, kv_heads, scale, ctx, rot=0, krot=None, window=None, keep=0, cap=None, sink=None,
               gate=None, gate_logits=None, pool=0, blocks=None, out=None, out_scale=1.0, tensor_cores=True):
    """Causal attention of packed prompts.  Rows of q: heads x (dim | rot), of k and v: kv_heads x dim / vdim, of krot: the rot
    elements that all heads' keys share (rows may be strided, their elements are dense) -> [T, heads vdim].  Keys at distance <
    ``window`` and the first ``keep`` of the sequence, or the means ``blocks`` of ``pool`` tokens before the window (see
    :func:`pool_blocks`); scores ``cap tanh(s / cap)``; ``exp(sink)`` in the denominator; ``gate`` (fp32 [T, heads]) or the sigmoid of
    ``gate_logits`` ([T, heads vdim] in the model dtype), and ``out_scale``, multiply the result (``out``: rows may be strided)."""
    T, dim, vdim = q.shape[0], k.shape[1] // kv_heads, v.shape[1] // kv_heads
    out = torch.empty(T, heads * vdim, dtype=q.dtype, device=q.device) if out is None else out
    assert out.shape == (T, heads * vdim) and out.stride(1) == 1 and out.dtype == q.dtype
    pk, pv = blocks if pool else (None, None)
    assert not pool or (pk.is_contiguous() and pv.is_contiguous() and pk.shape[0] == pv.shape[0] == T // pool + 1)
    assert q.shape[1] == heads * (dim + rot) and all(t.stride(1) == 1 for t in (q, k, v)) and (rot == 0 or krot.stride(1) == 1)
    mode = 1 if gate is not None else 2 if gate_logits is not None else 0
    assert mode != 1 or (gate.shape == (T, heads) and gate.dtype == torch.float32 and gate.is_contiguous())
    assert mode != 2 or (gate_logits.shape == out.shape and gate_logits.dtype == q.dtype and gate_logits.stride(1) == 1)
    gate = gate_logits if mode == 2 else gate
    rows = [c for t in (q, k, v, krot) for c in (_p(t), c_longlong(0 if t is None else t.stride(0)))]
    sizes = [c_int(x) for x in (T, heads, kv_heads, dim, rot, vdim, window or 0, keep)] + [c_float(scale), c_float(cap or 0.0)]
    tail = [_p(sink), c_int(mode), _p(gate), c_longlong(0 if gate is None else gate.stride(0)), c_int(pool), _p(pk), _p(pv), _p(out),
            c_longlong(out.stride(0)), c_float(out_scale)]
    aligned = all(t is None or (t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0) for t in (q, k, v, krot, out)) and (
        mode != 2 or (gate.data_ptr() % 16 == 0 and gate.stride(0) % 8 == 0))
    if q.dtype == torch.bfloat16 and tensor_cores and aligned and scale > 0 and mixer_attn_tc_ok(heads, kv_heads, dim, rot, vdim):
        cu = ctx.cu_seqlens
        assert cu.dtype == torch.int32
        _chk(lib().trlb_mixer_attn_tc(*rows, _p(cu), c_int(cu.numel() - 1), *sizes, *tail, _p(status_buffer(q.device)), _s()),
             "mixer_attn_tc")
    else:
        _chk(lib().trlb_mixer_attn(*rows, _p(ctx.positions.to(torch.int32)), *sizes, *tail, _b(q), _s()), "mixer_attn")
    return out


GATES = {None: 0, "head": 1, "element": 2}


def pool_blocks(k, v, cu, pool, seq_slot=None, pool_k=None, pool_v=None):
    """Means of blocks of ``pool`` rows of packed keys [T, kv_heads dim] and values: ([T // pool + 1, kv_heads dim], the same of the
    values); a sequence that starts at token a has its blocks from row ``a // pool`` on, rows of no block are zeros.  With
    ``seq_slot`` they also go to ``pool_k``, ``pool_v`` [slots, rows, kv_heads, dim / vdim]."""
    T = k.shape[0]
    assert k.stride(1) == 1 and v.stride(1) == 1 and k.dtype == v.dtype and cu.dtype == torch.int32
    pk, pv = (torch.empty(T // pool + 1, t.shape[1], dtype=t.dtype, device=t.device) for t in (k, v))
    slots, rows = (0, 0) if pool_k is None else pool_k.shape[:2]
    _chk(lib().trlb_pool_blocks(_p(k), c_longlong(k.stride(0)), c_int(k.shape[1]), _p(v), c_longlong(v.stride(0)), c_int(v.shape[1]), _p(cu),
                                c_int(cu.numel() - 1), c_int(T), c_int(pool), _p(pk), _p(pv), _p(seq_slot), c_int(slots), c_int(rows),
                                _p(pool_k), _p(pool_v), _b(k), _s()), "pool_blocks")
    return pk, pv


def _pools(pool, pool_k, pool_v):
    rows = 0 if pool_k is None else pool_k.shape[1]
    assert not pool or (pool_k.is_contiguous() and pool_v.is_contiguous() and pool_v.shape[:2] == pool_k.shape[:2])
    return [c_int(pool), c_int(rows)]


def attn_prep(y, m, positions, temp, *, q_norm=None, k_norm=None, unit=True, whole_norm=False, q_head=None, table=None, rot=0, halves=False, values=True,
              gates="element", tok_slot=None, q=None, k=None, g=None, head_gate=None, k_cache=None, v_cache=None, block_table=None,
              block_size=0, pool=0, pool_k=None, pool_v=None):
    """Rows ``y`` [q | k | v | g] of an attention mixer's input projection: normed queries (times ``temp`` by position) and keys,
    both rotated by ``table`` (their first ``rot`` elements, in pairs of neighbours or of ``halves``); keys and values to the paged
    cache; ``gates`` per head as fp32 sigmoids to ``head_gate``.  The norm is per head, with ``whole_norm`` over all heads, and times
    the weights ``q_norm`` / ``k_norm`` if there are any; without ``unit`` there is no norm.  ``q_head``: factors of the queries per
    head.  With ``pool`` the token that completes a block of that many leaves the block's means in its slot's rows of ``pool_k``,
    ``pool_v``.  Without ``values`` the keys as projected are the values.  Without
    ``q`` queries are replaced in place, keys too unless they go to ``k``; with ``q``
    (and ``g`` for gate logits per element) ``y`` is fp32 sums, and they are zeroed."""
    rows = y.shape[0]
    assert y.stride(1) == 1 and positions.dtype == torch.int32 and (q is None or y.dtype == torch.float32)
    assert (head_gate is None) == (gates != "head") and (k is None or (k.is_contiguous() and k.dtype == (getattr(m, "dtype", None) or m.o.dtype)))
    dt = getattr(m, "dtype", None) or m.o.dtype
    assert rot == 0 or (table.dtype == torch.float32 and table.shape[1] * 2 == rot)
    mb = 0 if block_table is None else block_table.shape[1]
    _chk(lib().trlb_attn_prep(_p(y), c_int(int(y.dtype == torch.float32)), c_longlong(y.stride(0)), c_int(rows), c_int(m.heads),
                              c_int(m.kv_heads), c_int(m.dim), c_int(m.vdim), c_int(int(m.kv_from is None)), c_int(int(values)),
                              c_int(GATES[gates]), c_float(m.eps), _p(positions), _p(tok_slot), _p(temp), _len(temp),
                              c_int(int(whole_norm)), _p(q_norm), _p(k_norm), c_int(rot), c_int(int(halves)),
                              _p(table), _len(table), _p(q), _p(k), _p(g), _p(head_gate), _p(k_cache), _p(v_cache),
                              _p(block_table), c_int(mb), c_int(block_size), c_int(int(unit)), _p(q_head), *_pools(pool, pool_k, pool_v),
                              _p(pool_k), _p(pool_v), c_int(int(dt == torch.bfloat16)), _s()), "attn_prep")


def grouped_decode(q, k_cache, v_cache, m, seq_lens, block_table, block_size, out, gate=None, *, head_gate=None, window=None, keep=0,
                   sink=None, pool=0, pool_k=None, pool_v=None, out_scale=1.0):
    """One token per slot on the CUDA cores: any size, bf16 or fp32.  q [B, heads, dim], gate logits [B, heads vdim], factors
    ``head_gate`` fp32 [B, heads]; ``window``, ``keep``, ``sink`` and ``out_scale`` as in :func:`mixer_attn`, ``pool`` and its rows as in :func:`attn_prep`; rows
    of ``out`` [B, heads vdim] may be strided."""
    B = q.shape[0]
    assert out.shape == (B, m.heads * m.vdim) and out.stride(1) == 1
    _chk(lib().trlb_grouped_decode(_p(q), _p(k_cache), _p(v_cache), _p(gate), _p(head_gate), _p(sink), _p(out), c_int(B), c_int(m.heads),
                                   c_int(m.kv_heads), c_int(m.dim), c_int(m.vdim), c_int(window or 0), c_int(keep), c_float(m.scale),
                                   c_float(m.cap or 0.0), _p(seq_lens), _p(block_table), c_int(block_table.shape[1]), c_int(block_size),
                                   *_pools(pool, pool_k, pool_v), _p(pool_k), _p(pool_v), c_longlong(out.stride(0)), c_float(out_scale),
                                   _b(q), _s()), "grouped_decode")


def grouped_decode_tc_ok(m, block_size: int) -> bool:
    return m.scale > 0 and bool(lib().trlb_grouped_decode_tc_ok(c_int(m.heads), c_int(m.kv_heads), c_int(m.dim), c_int(m.vdim),
                                                                c_int(block_size)))


def grouped_decode_tc_items(B: int, m) -> int:
    return int(lib().trlb_grouped_decode_tc_items(c_int(B), c_int(m.heads), c_int(m.kv_heads)))


def grouped_decode_tc(q, k_cache, v_cache, m, seq_lens, block_table, block_size, out, gate=None, splits=1, part_o=None, part_ml=None, *,
                      head_gate=None, window=None, keep=0, sink=None, pool=0, pool_k=None, pool_v=None, out_scale=1.0):
    """:func:`grouped_decode` on the tensor cores (bf16).  With ``splits`` > 1: ``part_o`` [>= B heads splits vdim] and
    ``part_ml`` [>= 2 B heads splits] fp32 scratch."""
    B = q.shape[0]
    assert q.dtype == torch.bfloat16 and q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.shape[1] == block_size and out.shape == (B, m.heads * m.vdim) and out.stride(1) == 1 and (gate is None or gate.is_contiguous())
    if splits > 1:
        assert part_o.numel() >= B * m.heads * splits * m.vdim and part_ml.numel() >= 2 * B * m.heads * splits
    _chk(lib().trlb_grouped_decode_tc(_p(q), _p(k_cache), _p(v_cache), _p(gate), _p(out), c_int(k_cache.shape[0]), c_int(B), c_int(m.heads),
                                      c_int(m.kv_heads), c_int(m.dim), c_int(m.vdim), c_int(window or 0), c_int(keep), c_float(m.scale),
                                      c_float(m.cap or 0.0), _p(sink), _p(head_gate), _p(seq_lens), _p(block_table),
                                      c_int(block_table.shape[1]), c_int(block_size), c_int(splits), _p(part_o), _p(part_ml),
                                      *_pools(pool, pool_k, pool_v), c_int(0 if pool_k is None else pool_k.shape[0]), _p(pool_k), _p(pool_v),
                                      c_longlong(out.stride(0)), c_float(out_scale), _p(status_buffer(q.device)), _s()), "grouped_decode_tc")


def moe_route(z, correction, top, *, positions=None, scores="sigmoid", renormalize=False, gain=1.0, clear=False):
    """fp32 logits z [T, E] (zeroed with ``clear``) -> (choice, rank, weight) [T, top] and counts [E]: the experts of the largest
    score (sigmoid or softmax) + correction, their place among the expert's tokens, their bare scores (over their sum with
    ``renormalize``) times ``gain``.  Rows of negative position choose nothing (-1)."""
    T, E = z.shape
    assert z.dtype == torch.float32 and z.is_contiguous() and (correction is None or correction.dtype == torch.float32)
    i32 = dict(dtype=torch.int32, device=z.device)
    choice, rank, weight = torch.empty(T, top, **i32), torch.empty(T, top, **i32), torch.empty(T, top, dtype=torch.float32, device=z.device)
    counts = torch.empty(E, **i32) if T <= 128 else torch.zeros(E, **i32)
    _chk(lib().trlb_moe_route(_p(z), _p(correction), _p(positions), c_int(T), c_int(E), c_int(top), c_int(int(renormalize)),
                              c_int({"sigmoid": 0, "softmax": 1}[scores]), c_float(gain), c_int(int(clear)), _p(choice), _p(rank), _p(weight), _p(counts), _s()), "moe_route")
    return choice, rank, weight, counts


def moe_gather(h, choice, rank, counts):
    """Rows of h [T, H] sorted by expert, one per choice -> (x [T top, H], row [T, top] where a choice stands (-1: none), offsets
    [E + 1]); rows past ``offsets[E]`` mean nothing."""
    (T, H), top, E = h.shape, choice.shape[1], counts.numel()
    assert h.is_contiguous()
    i32 = dict(dtype=torch.int32, device=h.device)
    x, row, offsets = torch.empty(T * top, H, dtype=h.dtype, device=h.device), torch.empty(T, top, **i32), torch.empty(E + 1, **i32)
    _chk(lib().trlb_moe_gather(_p(h), _p(choice), _p(rank), _p(counts), c_int(T), c_int(E), c_int(top), c_int(H), _p(x), _p(row),
                               _p(offsets), _b(h), _s()), "moe_gather")
    return x, row, offsets


def moe_sum(y, row, weight, out=None):
    """fp32 [T, H]: sum over the choices of ``weight * y[row]``."""
    (T, top), H = row.shape, y.shape[1]
    out = torch.empty(T, H, dtype=torch.float32, device=y.device) if out is None else out
    assert y.is_contiguous() and out.is_contiguous() and out.dtype == torch.float32
    _chk(lib().trlb_moe_sum(_p(y), _p(row), _p(weight), c_int(T), c_int(top), c_int(H), _p(out), _b(y), _s()), "moe_sum")
    return out


def moe_rows_gemm(a, w, offsets):
    """``a[r] w[e]^T`` for the rows r of expert e on the CUDA cores: any size, bf16 or fp32."""
    assert a.is_contiguous() and w.is_contiguous() and a.dtype == w.dtype and a.shape[1] == w.shape[2]
    out = torch.empty(a.shape[0], w.shape[1], dtype=a.dtype, device=a.device)
    _chk(lib().trlb_moe_rows_gemm(_p(a), _p(w), _p(offsets), _p(out), c_longlong(a.shape[0]), c_int(w.shape[0]), c_int(w.shape[1]),
                                  c_int(w.shape[2]), _b(a), _s()), "moe_rows_gemm")
    return out


def hgrn2_prompt(y, z, m, cu, seq_slot=None, state=None):
    """The recurrence over packed prompts, token by token: rows y [q | v] in the model dtype, z fp32 gate logits without bias ->
    fp32 [T, heads, vdim]; ``state`` [slots, heads, dim, vdim] of ``seq_slot`` gets the final one."""
    T, qd = y.shape[0], m.heads * m.dim
    assert y.stride(1) == 1 and z.stride(1) == 1 and z.dtype == torch.float32 and cu.dtype == torch.int32
    out = torch.empty(T, m.heads, m.vdim, dtype=torch.float32, device=y.device)
    _chk(lib().trlb_hgrn2_prompt(_p(y), c_longlong(y.stride(0)), c_int(qd), _p(z), c_longlong(z.stride(0)), _p(m.f_bias), _p(m.lower), _p(cu),
                                 c_int(cu.numel() - 1), _p(seq_slot if state is not None else None), _p(state),
                                 c_int(0 if state is None else state.shape[0]), c_int(m.heads), c_int(m.dim), c_int(m.vdim), _p(out), _b(y),
                                 _s()), "hgrn2_prompt")
    return out


def hgrn2_chunk_ok(m) -> bool:
    return bool(lib().trlb_hgrn2_chunk_ok(c_int(m.heads), c_int(m.dim), c_int(m.vdim)))


def hgrn2_chunk(y, z, m, cu, seq_slot=None, state=None, normed=None, scale=1.0):
    """:func:`hgrn2_prompt` in 128-token chunks on the tensor cores (bf16; see ``hgrn2_chunk_ok``).  With ``normed`` [T, heads vdim]
    (rows may be strided; vdim <= 128) that gets the outputs over their rms per head times the norm's weight and ``scale``, and is
    returned."""
    T, n_seq, qd = y.shape[0], cu.numel() - 1, m.heads * m.dim
    assert y.dtype == torch.bfloat16 and y.stride(1) == 1 and z.stride(1) == 1 and z.dtype == torch.float32 and cu.dtype == torch.int32
    assert normed is None or (normed.shape == (T, m.heads * m.vdim) and normed.stride(1) == 1 and normed.dtype == torch.bfloat16)
    out = torch.empty(T, m.heads, m.vdim, dtype=torch.float32, device=y.device) if normed is None else None
    parts = torch.empty(2, int(lib().trlb_hgrn2_chunks(c_int(T), c_int(n_seq))), m.heads, m.dim, m.vdim, dtype=torch.bfloat16, device=y.device)
    _chk(lib().trlb_hgrn2_chunk(_p(y), c_longlong(y.stride(0)), c_int(qd), _p(z), c_longlong(z.stride(0)), _p(m.f_bias), _p(m.lower), _p(cu),
                                c_int(n_seq), c_int(T), _p(seq_slot if state is not None else None), _p(state),
                                c_int(0 if state is None else state.shape[0]), c_int(m.heads), c_int(m.dim), c_int(m.vdim),
                                _p(m.norm if normed is not None else None), c_float(m.eps), c_float(scale), _p(normed),
                                c_longlong(0 if normed is None else normed.stride(0)), _p(out), _p(parts[0]), _p(parts[1]),
                                _p(status_buffer(y.device)), _s()), "hgrn2_chunk")
    return out if normed is None else normed


def head_norm(o, w, eps, dtype, out=None, scale=1.0):
    """o fp32 [T, heads, vdim] over its rms per head times ``w`` [vdim] and ``scale`` -> [T, heads vdim] (rows of ``out`` may be
    strided)."""
    T, H, E = o.shape
    out = torch.empty(T, H * E, dtype=dtype, device=o.device) if out is None else out
    assert o.is_contiguous() and o.dtype == torch.float32 and out.shape == (T, H * E) and out.stride(1) == 1 and out.dtype == dtype
    _chk(lib().trlb_head_norm(_p(o), _p(w), c_float(eps), c_int(T), c_int(H), c_int(E), c_float(scale), _p(out), c_longlong(out.stride(0)),
                              _b(out), _s()), "head_norm")
    return out


def hgrn2_step(sums, m, seq_lens, state, out, scale=1.0):
    """One token per slot: fp32 sums [B, q | v | z] (zeroed), state [slots, heads, dim, vdim] moves on; out [B, heads vdim] (rows
    may be strided) = outputs over their rms per head times the norm's weight and ``scale``."""
    B = sums.shape[0]
    assert sums.dtype == torch.float32 and sums.stride(1) == 1 and state.is_contiguous() and state.shape[0] >= B
    assert out.shape == (B, m.heads * m.vdim) and out.stride(1) == 1 and sums.shape[1] >= m.heads * (2 * m.dim + m.vdim)
    _chk(lib().trlb_hgrn2_step(_p(sums), c_longlong(sums.stride(0)), _p(m.f_bias), _p(m.lower), _p(m.norm), c_float(m.eps), c_float(scale),
                               _p(seq_lens), c_int(B), _p(state), c_int(m.heads), c_int(m.dim), c_int(m.vdim), _p(out),
                               c_longlong(out.stride(0)), _b(out), _s()), "hgrn2_step")


def conv_prompt(x, m, ctx, seq_slot=None, conv_state=None):
    """Causal per-channel convolution of packed prompts: x [T, width] (rows may be strided) -> [T, width]; ``conv_state`` [slots,
    taps - 1, width] of ``seq_slot`` gets the last inputs of every sequence."""
    T, C = x.shape
    assert x.stride(1) == 1
    u = torch.empty(T, C, dtype=x.dtype, device=x.device)
    cu = ctx.cu_seqlens
    _chk(lib().trlb_conv_prompt(_p(x), c_longlong(x.stride(0)), _p(m.x_bias), _p(m.conv), _p(m.conv_bias), _p(ctx.positions.to(torch.int32)),
                                c_int(T), c_int(C), c_int(m.taps), _p(cu), c_int(cu.numel() - 1), _p(seq_slot),
                                c_int(0 if conv_state is None else conv_state.shape[0]), _p(conv_state), _p(u), _b(x), _s()), "conv_prompt")
    return u


def conv_step(x, m, seq_lens, state, u):
    """One token per slot: x fp32 sums [B, width] (zeroed), state [B, taps - 1, width] moves on."""
    B, C = x.shape
    assert x.dtype == torch.float32 and x.stride(1) == 1
    _chk(lib().trlb_conv_step(_p(x), c_longlong(x.stride(0)), _p(m.x_bias), _p(m.conv), _p(m.conv_bias), _p(seq_lens), c_int(B), c_int(C),
                              c_int(m.taps), _p(state), _p(u), _b(u), _s()), "conv_step")


def rglru_tc_ok(m) -> bool:
    return bool(lib().trlb_rglru_tc_ok(c_int(m.width), c_int(m.blocks)))


def rglru_scan(z, u, y, m, ctx, seq_slot=None, state=None):
    """Recurrence of packed prompts on the CUDA cores.  z [T, 2, width] fp32 gate logits without their biases, u [T, width], y
    [T, width] GELU branch without its bias (rows may be strided); ``state`` [slots, width] of ``seq_slot`` gets the final one."""
    T, C = u.shape
    assert z.is_contiguous() and z.dtype == torch.float32 and u.is_contiguous() and y.stride(1) == 1
    out = torch.empty(T, C, dtype=u.dtype, device=u.device)
    cu = ctx.cu_seqlens
    _chk(lib().trlb_rglru_scan(_p(z), _p(u), _p(y), c_longlong(y.stride(0)), _p(m.lam), _p(m.gate_bias), _p(m.y_bias), _p(cu),
                               c_int(cu.numel() - 1), _p(seq_slot), c_int(0 if state is None else state.shape[0]), _p(state),
                               c_float(m.decay), c_int(C), _p(out), _b(u), _s()), "rglru_scan")
    return out


def rglru_prompt_tc(u, y, m, ctx, seq_slot=None, state=None):
    """Gate products and :func:`rglru_scan` in one tensor-core kernel (bf16; see ``rglru_tc_ok``)."""
    T, C = u.shape
    assert u.dtype == y.dtype == m.gates.dtype == torch.bfloat16 and u.is_contiguous() and m.gates.is_contiguous() and y.stride(1) == 1
    out = torch.empty(T, C, dtype=u.dtype, device=u.device)
    cu = ctx.cu_seqlens
    _chk(lib().trlb_rglru_prompt_tc(_p(u), _p(y), c_longlong(y.stride(0)), _p(m.gates), _p(m.lam), _p(m.gate_bias), _p(m.y_bias), _p(cu),
                                    c_int(cu.numel() - 1), c_int(T), _p(seq_slot), c_int(0 if state is None else state.shape[0]),
                                    _p(state), c_float(m.decay), c_int(C), c_int(m.blocks), _p(out), _p(status_buffer(u.device)), _s()),
         "rglru_prompt_tc")
    return out


def rglru_step(z, u, y, m, seq_lens, state, out):
    """One token per slot; y: fp32 sums of the GELU branch (zeroed)."""
    B, C = u.shape
    assert z.is_contiguous() and z.dtype == torch.float32 and u.is_contiguous() and y.stride(1) == 1
    _chk(lib().trlb_rglru_step(_p(z), _p(u), _p(y), c_longlong(y.stride(0)), _p(m.lam), _p(m.gate_bias), _p(m.y_bias), _p(seq_lens),
                               c_int(B), _p(state), c_float(m.decay), c_int(C), _p(out), _b(u), _s()), "rglru_step")


def rglru_step_tc(u, y, m, seq_lens, state, out):
    """Gate products and :func:`rglru_step` in one tensor-core kernel (bf16)."""
    B, C = u.shape
    assert u.dtype == torch.bfloat16 and u.is_contiguous() and m.gates.is_contiguous() and state.shape[0] >= B
    _chk(lib().trlb_rglru_step_tc(_p(u), _p(y), c_longlong(y.stride(0)), _p(m.gates), _p(m.lam), _p(m.gate_bias), _p(m.y_bias), _p(seq_lens),
                                  c_int(B), _p(state), c_float(m.decay), c_int(C), c_int(m.blocks), _p(out), _p(status_buffer(u.device)),
                                  _s()), "rglru_step_tc")


def latent_absorb(qacc, m, positions, table, q_lat, clear):
    B = qacc.shape[0]
    kr, w = latent_row(m.kv_rank, m.rot_dim)
    _chk(lib().trlb_latent_absorb(_p(qacc), c_longlong(qacc.stride(0)), _p(m.uk), _p(q_lat), c_int(B), c_int(m.heads),
                                  c_int(m.dim), c_int(m.rot_dim), c_int(m.kv_rank), c_int(kr), c_int(w), _p(positions),
                                  _p(table), _len(table), c_int(int(clear)), _b(q_lat), _s()), "latent_absorb")


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
                                 c_int(m.rot_dim), c_int(kr), c_int(w), _p(positions), _p(table), _len(table), _s()),
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
