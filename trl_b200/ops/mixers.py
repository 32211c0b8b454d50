"""Mechanisms of the layered decoders (models/layered.py) on packed prompts.

CUDA tensors run the kernels of ``csrc/mixers.cu``, ``csrc/grouped_attn.cu``, ``csrc/rglru.cu``, ``csrc/layered_moe.cu`` and the
tensor-core mixer kernels, in bf16 or fp32; CPU tensors run :mod:`trl_b200.oracle.mixers`.  On CUDA the kernels are inference only (prompts,
log-probs, generation).

A serving engine passes itself through ``ctx.kv``: ``paged_cache(li)`` and ``recurrent_state(li)`` say where layer ``li``
leaves what decoding continues from.  ``ctx.shared`` holds the keys and values that later layers of the same forward borrow."""
from __future__ import annotations

import contextlib
import math
from typing import NamedTuple

import torch
import torch.nn.functional as F

from ..oracle import mixers as _ref


def _k():
    from . import cuda_mixers

    return cuda_mixers


class RotarySpec:
    """Rotary positions with optional frequency scaling: YaRN's (``fast``, ``slow``) or Llama 3's (``low``, ``high``).
    ``table(n)``: fp32 [n, dims / 2, 2] (cos, sin), the magnitude of the scaling folded in; angles are evaluated in fp64 before
    they are rounded."""

    def __init__(self, dims: int, base: float, scaling: dict | None = None):
        self.dims, self.base, self.scaling = dims, base, dict(scaling) if scaling else None
        self._tables: dict = {}

    def frequencies(self) -> torch.Tensor:
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / self.dims)
        if self.scaling is None:
            return f
        s = self.scaling
        if "low" in s:
            turns = s["original"] * f / (2.0 * math.pi)  # of a pair in the original context
            keep = ((turns - s["low"]) / max(s["high"] - s["low"], 1e-9)).clamp(0.0, 1.0)
            keep = torch.where(turns < s["low"], 0.0, torch.where(turns > s["high"], 1.0, keep))
            return (1.0 - keep) * f / s["factor"] + keep * f

        def turns_to_dim(t):
            return self.dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(self.base))

        lo = max(math.floor(turns_to_dim(s["fast"])), 0)
        hi = min(math.ceil(turns_to_dim(s["slow"])), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / s["factor"] * ramp + f * (1.0 - ramp)

    @property
    def magnitude(self) -> float:
        return 1.0 if self.scaling is None or "low" in self.scaling else 0.1 * math.log(self.scaling["factor"]) + 1.0

    def table(self, n: int, device) -> torch.Tensor:
        key = str(device)
        t = self._tables.get(key)
        if t is None or t.shape[0] < n:
            size = max(256, 1 << (n - 1).bit_length())
            ang = torch.arange(size, dtype=torch.float64, device=device)[:, None] * self.frequencies().to(device)
            t = (torch.stack([ang.cos(), ang.sin()], -1) * self.magnitude).float().contiguous()
            self._tables[key] = t
        return t


class TemperatureSpec:
    """Factor of the query by position: ``1 + coef ln(floor((p + 1) / every) + 1)``, fp32 values of fp64 arithmetic."""

    def __init__(self, coef: float, every: float):
        self.coef, self.every = float(coef), every
        self._tables: dict = {}

    def table(self, n: int, device) -> torch.Tensor:
        key = str(device)
        t = self._tables.get(key)
        if t is None or t.shape[0] < n:
            size = max(256, 1 << (n - 1).bit_length())
            p = torch.arange(1, size + 1, dtype=torch.float64)
            t = (1.0 + self.coef * torch.log(torch.floor(p / self.every) + 1.0)).float().to(device)
            self._tables[key] = t
        return t


def check_can_run(w: torch.Tensor):
    if w.is_cuda and torch.is_grad_enabled() and w.requires_grad:
        raise NotImplementedError("the CUDA kernels of the layered decoders are inference only: run them under "
                                  "torch.no_grad(), or train on CPU tensors")


@contextlib.contextmanager
def _ieee_fp32():
    """fp32 matrix products in fp32 (no TF32), whatever the process default is."""
    was = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        yield
    finally:
        torch.backends.cuda.matmul.allow_tf32 = was


def linear(x, w):
    """``x W^T`` in the dtype of the inputs."""
    if x.is_cuda and x.dtype == torch.float32:
        with _ieee_fp32():
            return F.linear(x, w)
    return F.linear(x, w.to(x.dtype))


def linear_f32(x, w):
    """``x W^T`` with the fp32 accumulators as the result."""
    if x.is_cuda and x.dtype == torch.bfloat16:
        return torch.mm(x, w.t(), out_dtype=torch.float32)
    return linear(x, w)


def embed_scaled(ids, emb, scale):
    if emb.is_cuda:
        return _k().embed_scaled(ids, emb, scale)
    return F.embedding(ids, emb).float() * scale


def embed_pairs(ids, emb, scale, pairs, spec, positions, where):
    """Scaled embeddings plus the rows of a table of token pairs (flat packed ids); ``where``: a serving engine's last tokens."""
    if emb.is_cuda:
        return _k().embed_pairs(ids, emb, scale, pairs, spec["mul_prev"], spec["mul_cur"], positions.to(torch.int32), **where)
    rows = _ref.pair_rows(ids, positions, spec["mul_prev"], spec["mul_cur"], pairs.shape[0] - 1)
    return F.embedding(ids, emb).float() * scale + F.embedding(rows, pairs).float()


def embed_normed(ids, emb, scale, w, eps, shift=0.0):
    """fp32 embeddings times ``scale``, over their rms times ``shift + w``."""
    if emb.is_cuda:
        return _k().embed_normed(ids, emb, scale, w, eps, shift)
    return _ref.unit_rms(F.embedding(ids, emb).float() * scale, eps) * (shift + w)


def dynamic_tanh(x, delta, alpha, w, b, out_dtype, clear=False, out=None):
    """(norm of ``x + delta`` in ``out_dtype``, ``x + delta``); on CUDA the sum is formed in place."""
    if x.is_cuda:
        return _k().dynamic_tanh(x, delta, alpha, w, b, out_dtype, clear=clear, out=out), x
    x = x if delta is None else x + delta
    return _ref.dynamic_tanh(x, alpha, w, b).to(out_dtype), x


def rms_residual(x, delta, post, w, eps, out_dtype, clear=False, out=None, **kw):
    """(``s / rms(s) * w`` in ``out_dtype``, s) of ``s = x + delta``, where delta over its rms times ``post`` is added when
    ``post`` is given and s itself is the output when ``w`` is None; on CUDA the sum is formed in place.  ``shift`` is added to the
    weights, ``post_scale`` multiplies ``post``, ``gain`` the output.  ``mult`` multiplies delta, which may be a pair (of tensors, or a
    tensor and :class:`ExpertRows`) to be added up; ``anchor`` [T, H] and ``bump`` [H] are added as well; with a second weight
    ``w2`` (and ``out2``) the output is a pair."""
    if x.is_cuda:
        return _k().rms_residual(x, delta, post, w, eps, out_dtype, clear=clear, out=out, **kw), x
    kw.pop("out2", None)
    y, x = _ref.rms_residual(x, delta, post, w, eps, **kw)
    return (tuple(t.to(out_dtype) for t in y) if isinstance(y, tuple) else y.to(out_dtype)), x


class ExpertRows(NamedTuple):
    """What a mixture of experts gives before it is added up: token t's output is the sum over its choices c of
    ``weight[t, c] * y[row[t, c]]`` (a negative row: nothing)."""

    y: torch.Tensor
    row: torch.Tensor
    weight: torch.Tensor


def clamped_glu(z, limit, alpha, shift, out=None):
    return _k().clamped_glu(z, limit, alpha, shift, out=out) if z.is_cuda else _ref.clamped_glu(z, limit, alpha, shift)


def gelu_glu(z, out=None):
    return _k().gelu_glu(z, out=out) if z.is_cuda else _ref.gelu_glu(z)


def gelu_erf(z, out=None):
    return _k().gelu_erf(z, out=out) if z.is_cuda else F.gelu(z)


def experts(m, h, positions=None, logits=None, out=None, summed=True):
    """Mixture of experts: h [T, width] -> fp32 [T, width], or on CUDA without ``summed`` :class:`ExpertRows` for the kernel that
    adds them to the stream.  ``positions``: rows where they are negative choose nothing; ``logits``: fp32 sums of the router's
    product (zeroed), formed here when absent."""
    if not h.is_cuda:
        return _ref.experts(m, h.float())
    K = _k()
    z = linear_f32(h, m.router) if logits is None else logits
    choice, rank, weight, counts = K.moe_route(z, m.correction, m.top, positions=positions, clear=logits is not None,
                                               **m.routing)
    x, row, offsets = K.moe_gather(h, choice, rank, counts)
    if h.dtype == torch.bfloat16 and h.shape[1] % 8 == 0 and m.ff % 8 == 0:
        from . import cuda as KC

        act = KC.grouped_gemm(x, m.gate_up, offsets, m.ff, clamped_glu=m.glu)
        y = KC.grouped_gemm(act, m.down, offsets, h.shape[1])
    else:
        y = K.moe_rows_gemm(K.clamped_glu(K.moe_rows_gemm(x, m.gate_up, offsets), *m.glu), m.down, offsets)
    return K.moe_sum(y, row, weight, out=out) if summed else ExpertRows(y, row, weight)


def side_input(h, ids, table, off, gate, proj):
    """``proj (gelu_tanh(gate h) * table[ids, off : off + n])`` with fp32 sums."""
    z = linear(h, gate)
    if z.is_cuda:
        return linear_f32(_k().side_gate(z, ids, table, off), proj)
    return linear(F.gelu(z, approximate="tanh") * F.embedding(ids, table)[:, off:off + z.shape[1]].to(z.dtype), proj).float()


def latent_attention(m, h, ctx, li):
    if not h.is_cuda:
        return _ref.latent_attention(m, h.float(), ctx.positions, ctx.cu_seqlens)
    K = _k()
    pos = ctx.positions if ctx.positions.dtype == torch.int32 else ctx.positions.to(torch.int32)
    table = m.rope.table(ctx.max_seqlen, h.device) if m.rot_dim else None
    kr, width = K.latent_row(m.kv_rank, m.rot_dim)
    lat = torch.zeros(h.shape[0], width, dtype=h.dtype, device=h.device)
    cache = ctx.kv.paged_cache(li) if ctx.kv is not None else {}
    if m.q_rank:
        cq, gate = K.latent_prep(linear_f32(h, m.w_in), m, pos, table, lat=lat, **cache)
        q = linear(cq, m.uq)
    else:
        q = linear(h, m.w_in[: m.q_rows])
        _, gate = K.latent_prep(linear_f32(h, m.w_in[m.q_rows:]), m, pos, table, lat=lat, **cache)
    if m.rot_dim:
        K.rotate_q(q, m, pos, table)
    kv = linear(lat[:, : m.kv_rank], m.ukv)
    return linear_f32(latent_prompt_attention(q, kv, lat, m, ctx, gate), m.o)


def latent_prompt_attention(q, kv, lat, m, ctx, gate, tensor_cores=True):
    """Attention of packed prompts with latent keys and values, times the output gates (if any).  q [T, heads (dim | rot)]
    rotated, kv [T, heads dim | heads vdim], lat [T, latent row], gate [T, heads] -> [T, heads vdim]."""
    K = _k()
    kr, _ = K.latent_row(m.kv_rank, m.rot_dim)
    n = m.heads * m.dim
    return K.mixer_attn(q, kv[:, :n], kv[:, n:], heads=m.heads, kv_heads=m.heads, rot=m.rot_dim, krot=lat[:, kr:] if m.rot_dim else None,
                        scale=m.scale, window=m.window, sink=m.sink, gate=gate, ctx=ctx, tensor_cores=tensor_cores)


def attention(m, h, ctx, li):
    kept = ctx.shared[m.kv_from] if m.kv_from is not None else None
    if not h.is_cuda:
        out, kept = _ref.attention(m, h.float(), ctx.positions, ctx.cu_seqlens, kept)
    else:
        o, kept = attention_rows(m, linear(h, m.w_in), ctx, ctx.kv.paged_cache(li) if ctx.kv is not None else {}, kept)
        out = linear_f32(o, m.o)
    if li in ctx.shared:
        ctx.shared[li] = kept
    return out


def attention_rows(m, y, ctx, where, kept=None, out=None, scale=1.0):
    """From the rows ``y`` of the input projection (replaced in part) to what the output projection reads, times ``scale``, and the
    keys and values.  ``where`` (may be empty): the pages and slots that get them; ``kept``: those of the layer it borrows from."""
    K = _k()
    T, own, where = y.shape[0], kept is None, dict(where)
    pos = ctx.positions if ctx.positions.dtype == torch.int32 else ctx.positions.to(torch.int32)
    temp = m.temperature.table(ctx.max_seqlen, y.device) if m.temperature is not None else None
    table = m.rope.table(ctx.max_seqlen, y.device) if m.rot else None
    pools = where.pop("pools", {})
    q, k, v, g = y[:, : m.rows].split(m.parts, 1)
    # projected keys that are also the values stay as they are
    keys = torch.empty(T, m.kv_heads * m.dim, dtype=y.dtype, device=y.device) if own and not m.values else None
    gate = torch.empty(T, m.heads, dtype=torch.float32, device=y.device) if m.gate == "head" else None
    K.attn_prep(y, m, pos, temp, table=table, k=keys, head_gate=gate, **m.prep, **where)
    if own:
        kept = (k, v) if keys is None else (keys, k)
    blocks = K.pool_blocks(*kept, ctx.cu_seqlens, m.pool, **pools) if m.pool else None
    o = K.mixer_attn(q, *kept, heads=m.heads, kv_heads=m.kv_heads, scale=m.scale, cap=m.cap, **m.sight, gate=gate, pool=m.pool, blocks=blocks,
                     gate_logits=g if m.gate == "element" else None, ctx=ctx, out=out, out_scale=scale)
    return o, kept


def hgrn2(m, h, ctx, li):
    if not h.is_cuda:
        return _ref.hgrn2(m, h.float(), ctx.cu_seqlens)
    where = ctx.kv.recurrent_state(li) if ctx.kv is not None else {}
    return linear_f32(hgrn2_rows(m, linear(h, m.w_in[: m.rows]), linear_f32(h, m.w_in[m.rows:]), ctx, where), m.o)


def hgrn2_rows(m, y, z, ctx, where, out=None, scale=1.0):
    """From the rows ``y`` (query | value) and ``z`` (forget gate, fp32 sums) of the input projection to what the output projection
    reads, times ``scale``.  ``where`` (may be empty): the slots that get the final states."""
    K = _k()
    if m.vdim <= 128 and _hgrn2_tc(m, z, y, out):
        out = torch.empty(y.shape[0], m.out_width, dtype=y.dtype, device=y.device) if out is None else out
        return K.hgrn2_chunk(y, z, m, ctx.cu_seqlens, normed=out, scale=scale, **where)
    return K.head_norm(hgrn2_prompt_scan(m, y, z, ctx, where), m.norm, m.eps, y.dtype, out=out, scale=scale)


def _hgrn2_tc(m, z, *rows) -> bool:
    """Whether the tensor-core kernels take a mixer's sizes and these rows."""
    return (all(t is None or (t.dtype == torch.bfloat16 and t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0) for t in rows)
            and z.data_ptr() % 16 == 0 and z.stride(0) % 4 == 0 and _k().hgrn2_chunk_ok(m))


def hgrn2_prompt_scan(m, y, z, ctx, where, tensor_cores=True):
    """The recurrence over packed prompts -> fp32 [T, heads, vdim]."""
    K = _k()
    if tensor_cores and _hgrn2_tc(m, z, y):
        return K.hgrn2_chunk(y, z, m, ctx.cu_seqlens, **where)
    return K.hgrn2_prompt(y, z, m, ctx.cu_seqlens, **where)


def parallel(m, h, ctx, li):
    if not h.is_cuda:
        return _ref.parallel(m, h.float(), ctx.positions, ctx.cu_seqlens)
    a, b = m.left.rows, m.left.out_width
    where = ctx.kv.paged_cache(li) if ctx.kv is not None else dict(left={}, right={})
    y, z = linear(h, m.w_in[: m.rows]), linear_f32(h, m.w_in[m.rows:])
    o = torch.empty(h.shape[0], m.o.shape[1], dtype=h.dtype, device=h.device)
    attention_rows(m.left, y[:, :a], ctx, where["left"], out=o[:, :b], scale=m.scales[0])
    hgrn2_rows(m.right, y[:, a:], z, ctx, where["right"], out=o[:, b:], scale=m.scales[1])
    return linear_f32(o, m.o)


def block_gates(u, gates):
    """Block-diagonal products in fp32: u [T, C], gates [2, blocks, C / blocks (out), C / blocks (in)] -> [T, 2, C]."""
    T, C = u.shape
    n, blocks, w, _ = gates.shape
    with _ieee_fp32():
        z = torch.matmul(u.float().view(T, blocks, w).transpose(0, 1), gates.float().transpose(2, 3))  # [2, blocks, T, w]
    return z.permute(2, 0, 1, 3).reshape(T, n, C).contiguous()


def rglru(m, h, ctx, li):
    if not h.is_cuda:
        return _ref.rglru(m, h.float(), ctx.cu_seqlens)
    K = _k()
    y, x = linear(h, m.w_in).chunk(2, 1)
    where = ctx.kv.recurrent_state(li) if ctx.kv is not None else {}
    slot, state = where.get("seq_slot"), where.get("state")
    u = K.conv_prompt(x, m, ctx, slot, where.get("conv_state"))
    return linear_f32(rglru_prompt_scan(u, y, m, ctx, slot, state), m.o)


def rglru_prompt_scan(u, y, m, ctx, seq_slot=None, state=None, tensor_cores=True):
    """Gates, recurrence and multiplication by the GELU branch over packed prompts: u, y [T, width] -> [T, width]."""
    K = _k()
    if u.dtype == torch.bfloat16 and tensor_cores and K.rglru_tc_ok(m):
        return K.rglru_prompt_tc(u, y, m, ctx, seq_slot, state)
    return K.rglru_scan(block_gates(u, m.gates), u, y, m, ctx, seq_slot, state)


def mlstm_prompt_scan(y, m, ig, fg, ctx, where):
    """The recurrence over packed prompts.  y [T, q | k | v | ...] in the model dtype, log gates [T, heads] ->
    [T, heads, vdim] fp32; ``where`` (may be empty) says which slots get the final states."""
    K = _k()
    if y.dtype == torch.bfloat16 and K.mlstm_chunk_ok(m):
        return K.mlstm_chunk(y, m, ig, fg, ctx.cu_seqlens, **where)
    return K.mlstm_prompt(y, m, ig, fg, ctx.cu_seqlens, **where)


def mlstm(m, h, ctx, li):
    if not h.is_cuda:
        return _ref.mlstm(m, h.float(), ctx.cu_seqlens)
    K = _k()
    y = linear(h, m.w_in[: m.gate_row])
    ig, fg = K.mlstm_gates(linear_f32(h, m.w_in[m.gate_row:]), m.gate_bias, m.cap, m.heads)
    where = ctx.kv.recurrent_state(li) if ctx.kv is not None else {}
    o = mlstm_prompt_scan(y, m, ig, fg, ctx, where)
    out = torch.empty(h.shape[0], m.heads * m.vdim, dtype=h.dtype, device=h.device)
    K.mlstm_out(o, y[:, m.heads * (2 * m.dim + m.vdim):], m, out)
    return linear_f32(out, m.o)
