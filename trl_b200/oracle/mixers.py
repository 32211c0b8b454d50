"""PyTorch forms of the layered decoders' mechanisms: the execution path on CPU (differentiable, any float dtype) for
packed prompts.  Computations are vectorised over a sequence; nothing here keeps a cache."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def unit_rms(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rms_residual(x, delta, post, w, eps, shift=0.0, post_scale=None, gain=1.0, mult=1.0, anchor=None, bump=None, w2=None):
    """(``x + mult delta`` (delta over its rms times ``(shift + post) post_scale``, when given) ``+ anchor + bump`` (when given)) over
    its rms times ``(shift + w) gain`` (when given), with ``w2`` also times ``(shift + w2) gain``, and the sum.  A pair of deltas is
    their sum."""
    if delta is not None:
        if isinstance(delta, tuple):
            delta = delta[0] + delta[1]
        if post is not None:
            delta = unit_rms(delta, eps) * (shift + post)
            delta = delta if post_scale is None else delta * post_scale
        x = x + mult * delta
    for more in (anchor, bump):
        x = x if more is None else x + more
    y = x if w is None else unit_rms(x, eps)
    if w2 is not None:
        return (y * ((shift + w) * gain), y * ((shift + w2) * gain)), x
    return (y if w is None else y * ((shift + w) * gain)), x


def pair_rows(ids, positions, mul_prev, mul_cur, buckets):
    """Rows of the table of token pairs for packed sequences: the last one at position 0."""
    ids = ids.long()
    row = (ids.roll(1) * mul_prev + ids * mul_cur) % buckets
    return torch.where(positions > 0, row, torch.full_like(row, buckets))


def clamped_glu(z, limit, alpha, shift):
    g, u = z.chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + shift)


def gelu_glu(z):
    g, u = z.chunk(2, -1)
    return F.gelu(g, approximate="tanh") * u


def rotate_halves(x, cos, sin):
    """x [T, ..., n] with pairs (i, i + n / 2); cos / sin [T, n / 2]."""
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (x.shape[-1] // 2,)
    c, s = cos.view(shape), sin.view(shape)
    u, v = x.chunk(2, -1)
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def rotate_pairs(x, cos, sin):
    """x [T, ..., n] with pairs (2i, 2i + 1); cos / sin [T, n / 2]."""
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (x.shape[-1] // 2,)
    c, s = cos.view(shape), sin.view(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def sink_window_attention(q, k, v, scale, window, sink, cu, cap=None, keep=0, pool=0):
    """q [T, H, D], k [T, G, D], v [T, G, E] (H / G query heads read one key head), packed sequences by ``cu``; scores
    ``cap tanh(s / cap)``; softmax with ``exp(sink)`` added to the denominator (no such term without a sink); with a window the first
    ``keep`` keys of a sequence stay visible, or the means of the blocks of ``pool`` tokens that lie before it."""
    outs, per = [], q.shape[1] // k.shape[1]
    if per > 1:
        k, v = k.repeat_interleave(per, 1), v.repeat_interleave(per, 1)
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        n, blocks, ks, vs = b - a, 0, k[a:b], v[a:b]
        if pool and window is not None:
            blocks = n // pool
            ks, vs = (torch.cat([x, x[:blocks * pool].reshape(blocks, pool, *x.shape[1:]).mean(1)]) for x in (ks, vs))
        s = torch.einsum("qhd,khd->hqk", q[a:b], ks) * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        i = torch.arange(n, device=s.device)
        gap = i[:, None] - i[None, :]
        seen = (gap >= 0) if window is None else (gap >= 0) & ((gap < window) | (i < keep))
        if blocks:
            ends = torch.arange(blocks, device=s.device) * pool + pool - 1
            seen = torch.cat([seen, ends[None, :] <= i[:, None] - window], 1)
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.to(s.dtype)[:, None, None].expand(-1, n, 1)], -1)
        outs.append(torch.einsum("hqk,khe->qhe", torch.softmax(s, -1)[..., :n + blocks], vs))
    return torch.cat(outs)


def mlstm_parallel(q, k, v, ig, fg, cu):
    """Quadratic form of the recurrence: entry (t, j) weighs ``exp(F_t - F_j + i_j - m_t)`` with F the running sum of the
    log forget gates and ``m_t = max(F_t, max_j (F_t - F_j + i_j))`` (the running maximum starts at 0)."""
    outs = []
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        n = b - a
        c = fg[a:b].cumsum(0).T  # [H, n]
        d = c[:, :, None] - c[:, None, :] + ig[a:b].T[:, None, :]
        d = d.masked_fill(torch.ones(n, n, dtype=torch.bool).triu(1), float("-inf"))
        m = torch.maximum(d.amax(-1), c)  # [H, n]
        w = torch.exp(d - m[..., None]) * torch.einsum("qhd,khd->hqk", q[a:b], k[a:b])
        den = torch.maximum(w.sum(-1).abs(), torch.exp(-m)) + 1e-6
        outs.append((torch.einsum("hqk,khe->hqe", w, v[a:b]) / den[..., None]).transpose(0, 1))
    return torch.cat(outs)


def latent_attention(m, h, positions, cu):
    """``m``: a models.layered.LatentAttention; h [T, width] -> [T, width]."""
    T, H = h.shape[0], m.heads
    y = F.linear(h, m.w_in.to(h.dtype))
    q, kl, kr, g = y.split([m.q_rows, m.kv_rank, m.rot_dim, H if m.gated else 0], -1)
    if m.q_rank:
        q = F.linear(unit_rms(q, m.eps) * m.q_norm.to(h.dtype), m.uq.to(h.dtype))
    q = q.view(T, H, m.dim + m.rot_dim)
    lat = unit_rms(kl, m.eps) * m.kv_norm.to(h.dtype)
    k = F.linear(lat, m.uk.to(h.dtype)).view(T, H, m.dim)
    if m.rot_dim:
        table = m.rope.table(int(positions.max()) + 1 if T else 1, h.device).to(h.dtype)[positions.long()]
        cos, sin = table[..., 0], table[..., 1]
        q = torch.cat([q[..., : m.dim], rotate_pairs(q[..., m.dim:], cos, sin)], -1)
        k = torch.cat([k, rotate_pairs(kr, cos, sin)[:, None].expand(T, H, m.rot_dim)], -1)
    v = F.linear(lat, m.uv.to(h.dtype)).view(T, H, m.vdim)
    o = sink_window_attention(q, k, v, m.scale, m.window, m.sink, cu)
    if m.gated:
        o = o * torch.sigmoid(g)[..., None]
    return F.linear(o.reshape(T, H * m.vdim), m.o.to(h.dtype))


def attention(m, h, positions, cu, kept=None):
    """``m``: a models.layered.GroupedAttention; ``kept``: keys and values of the layer it borrows from.  Returns ([T, width],
    (keys, values))."""
    o, kept = attention_rows(m, F.linear(h, m.w_in.to(h.dtype))[:, : m.rows], positions, cu, kept)
    return F.linear(o, m.o.to(h.dtype)), kept


def attention_rows(m, h, positions, cu, kept=None):
    """Rows ``h`` of the input projection -> ([T, heads vdim], (keys, values))."""
    T, H, G = h.shape[0], m.heads, m.kv_heads
    q, k, v, g = h.split(m.parts, -1)

    def turned(x, n, w):
        """Norm (of all heads at once, or per head), weight, rotation."""
        if m.unit:
            x = unit_rms(x if m.whole_norm else x.reshape(T, n, m.dim), m.eps)
        x = (x if w is None else x * w.to(h.dtype)).reshape(T, n, m.dim)
        if not m.rot:
            return x
        table = m.rope.table(int(positions.max()) + 1 if T else 1, h.device).to(h.dtype)[positions.long()]
        turn = rotate_halves if m.halves else rotate_pairs
        return torch.cat([turn(x[..., : m.rot], table[..., 0], table[..., 1]), x[..., m.rot:]], -1)

    q = turned(q, H, m.q_norm)
    if m.temperature is not None:
        q = q * m.temperature.table(int(positions.max()) + 1 if T else 1, h.device).to(h.dtype)[positions.long()][:, None, None]
    if m.temp is not None:
        q = q * m.temp.to(h.dtype)[:, None]
    if kept is None:
        kept = turned(k, G, m.k_norm), (v if m.values else k).reshape(T, G, m.vdim)
    o = sink_window_attention(q, *kept, m.scale, m.window, m.sink, cu, m.cap, m.keep, m.pool)
    if m.gate == "head":
        o = o * torch.sigmoid(g)[..., None]
    o = o.reshape(T, H * m.vdim)
    return (o * torch.sigmoid(g) if m.gate == "element" else o), kept


def route(z, correction, top, renormalize=False, scores="sigmoid", gain=1.0):
    """Logits [T, E] -> (experts [T, top], weights [T, top])."""
    s = torch.softmax(z, -1) if scores == "softmax" else torch.sigmoid(z)
    idx = (s.detach() if correction is None else s.detach() + correction.to(z.dtype)).topk(top, -1).indices
    w = s.gather(1, idx)
    return idx, (w / (w.sum(-1, keepdim=True) + 1e-20) if renormalize else w) * gain


def experts(m, h):
    """``m``: a models.layered.ExpertMlp; h [T, width] -> [T, width]."""
    idx, w = route(F.linear(h, m.router.to(h.dtype)), m.correction, m.top, **m.routing)
    out = torch.zeros_like(h)
    for e in range(m.n):
        t, j = (idx == e).nonzero(as_tuple=True)
        y = F.linear(clamped_glu(F.linear(h[t], m.gate_up[e].to(h.dtype)), *m.glu), m.down[e].to(h.dtype))
        out = out.index_add(0, t, y * w[t, j][:, None])
    return out


def causal_conv(x, w, bias, cu):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start of every sequence."""
    taps = w.shape[1]
    outs = []
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        padded = F.pad(x[a:b].T[None], (taps - 1, 0))
        outs.append(F.conv1d(padded, w.to(x.dtype)[:, None], bias.to(x.dtype), groups=x.shape[1])[0].T)
    return torch.cat(outs)


def linear_recurrence(a, b, cu):
    """S_t = a_t S_(t-1) + b_t from S = 0, per channel.  Doubling: after step s an entry covers 2^s tokens."""
    outs = []
    for i, j in zip(cu[:-1].tolist(), cu[1:].tolist()):
        x, y, d = a[i:j], b[i:j], 1
        while d < j - i:
            y = torch.cat([y[:d], x[d:] * y[:-d] + y[d:]])
            x = torch.cat([x[:d], x[d:] * x[:-d]])
            d *= 2
        outs.append(y)
    return torch.cat(outs)


def rglru(m, h, cu):
    """``m``: a models.layered.RgLru."""
    T = h.shape[0]
    y, x = F.linear(h, m.w_in.to(h.dtype)).chunk(2, -1)
    y = F.gelu(y + m.y_bias.to(h.dtype), approximate="tanh")
    u = causal_conv(x + m.x_bias.to(h.dtype), m.conv, m.conv_bias, cu)
    z = torch.einsum("tbi,gboi->tgbo", u.view(T, m.blocks, -1), m.gates.to(h.dtype)).reshape(T, 2, -1)
    r, i = torch.sigmoid(z + m.gate_bias.to(h.dtype)).unbind(1)
    log_a = -m.decay * r * F.softplus(m.lam.to(h.dtype))
    b = torch.sqrt(-torch.expm1(2 * log_a)) * i * u
    return F.linear(linear_recurrence(torch.exp(log_a), b, cu) * y, m.o.to(h.dtype))


def mlstm(m, h, cu):
    """``m``: a models.layered.MLstm."""
    T, H = h.shape[0], m.heads
    y = F.linear(h, m.w_in.to(h.dtype))
    qd, vd = H * m.dim, H * m.vdim
    q, k, v, g, z = y.split([qd, qd, vd, vd, 2 * H], -1)
    z = m.cap * torch.tanh((z + m.gate_bias.to(h.dtype)) / m.cap)
    o = mlstm_parallel(q.view(T, H, m.dim) * m.dim ** -0.5, k.view(T, H, m.dim), v.view(T, H, m.vdim), z[:, :H],
                       F.logsigmoid(z[:, H:]), cu)
    o = unit_rms(o, m.eps).reshape(T, vd) * m.norm.to(h.dtype) * torch.sigmoid(g)
    return F.linear(o, m.o.to(h.dtype))


def hgrn2_scan(q, f, v, cu):
    """q, f [T, H, D], v [T, H, E] -> [T, H, E]: ``S = diag(f) S + (1 - f) v^T``, ``o = S^T q``."""
    outs = []
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=v.dtype, device=v.device)
        for t in range(a, b):
            S = f[t][..., None] * S + (1 - f[t])[..., None] * v[t][:, None]
            outs.append(torch.einsum("hd,hde->he", q[t], S))
    return torch.stack(outs)


def hgrn2_rows(m, h, cu):
    """``m``: a models.layered.HGrn2; rows ``h`` of its input projection -> [T, heads vdim]."""
    T, H = h.shape[0], m.heads
    q, v, z = h.split(m.parts, -1)
    low = m.lower.to(h.dtype)
    f = low + (1 - low) * torch.sigmoid(z + m.f_bias.to(h.dtype))
    o = hgrn2_scan(F.silu(q).reshape(T, H, m.dim), f.view(T, H, m.dim), v.reshape(T, H, m.vdim), cu)
    return (unit_rms(o, m.eps) * m.norm.to(h.dtype)).reshape(T, H * m.vdim)


def hgrn2(m, h, cu):
    return F.linear(hgrn2_rows(m, F.linear(h, m.w_in.to(h.dtype)), cu), m.o.to(h.dtype))


def parallel(m, h, positions, cu):
    """``m``: a models.layered.ParallelMixers."""
    y, a, outs = F.linear(h, m.w_in.to(h.dtype)), m.left.rows, []
    for side, rows, scale in ((m.left, y[:, :a], m.scales[0]), (m.right, y[:, a:], m.scales[1])):
        o = attention_rows(side, rows, positions, cu)[0] if side.kind.startswith("attention") else hgrn2_rows(side, rows, cu)
        outs.append(o * scale)
    return F.linear(torch.cat(outs, -1), m.o.to(h.dtype))
