"""PyTorch forms of the layered decoders' mechanisms: the execution path on CPU (differentiable, any float dtype) for
packed prompts.  Computations are vectorised over a sequence; nothing here keeps a cache."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def unit_rms(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rotate_pairs(x, cos, sin):
    """x [T, ..., n] with pairs (2i, 2i + 1); cos / sin [T, n / 2]."""
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (x.shape[-1] // 2,)
    c, s = cos.view(shape), sin.view(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def sink_window_attention(q, k, v, scale, window, sink, cu):
    """q, k [T, H, D], v [T, H, E], packed sequences by ``cu``; softmax with ``exp(sink)`` added to the denominator."""
    outs = []
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        n = b - a
        s = torch.einsum("qhd,khd->hqk", q[a:b], k[a:b]) * scale
        i = torch.arange(n)
        gap = i[:, None] - i[None, :]
        seen = (gap >= 0) if window is None else (gap >= 0) & (gap < window)
        s = s.masked_fill(~seen, float("-inf"))
        full = torch.cat([s, sink.to(s.dtype)[:, None, None].expand(-1, n, 1)], -1)
        outs.append(torch.einsum("hqk,khe->qhe", torch.softmax(full, -1)[..., :-1], v[a:b]))
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
    ql, kl, kr, g = y.split([m.q_rank, m.kv_rank, m.rot_dim, H], -1)
    table = m.rope.table(int(positions.max()) + 1 if T else 1, h.device).to(h.dtype)[positions.long()]
    cos, sin = table[..., 0], table[..., 1]
    q = F.linear(unit_rms(ql, m.eps) * m.q_norm.to(h.dtype), m.uq.to(h.dtype)).view(T, H, m.dim + m.rot_dim)
    q = torch.cat([q[..., : m.dim], rotate_pairs(q[..., m.dim:], cos, sin)], -1)
    lat = unit_rms(kl, m.eps) * m.kv_norm.to(h.dtype)
    kr = rotate_pairs(kr, cos, sin)
    k = F.linear(lat, m.uk.to(h.dtype)).view(T, H, m.dim)
    k = torch.cat([k, kr[:, None].expand(T, H, m.rot_dim)], -1)
    v = F.linear(lat, m.uv.to(h.dtype)).view(T, H, m.vdim)
    o = sink_window_attention(q, k, v, m.scale, m.window, m.sink, cu)
    o = o * torch.sigmoid(g)[..., None]
    return F.linear(o.reshape(T, H * m.vdim), m.o.to(h.dtype))


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
