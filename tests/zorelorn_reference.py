"""Plain, slow restatement of the Zorelorn decoder: one function per mechanism, one sequence at a time, every
recurrence run token by token.  The tests compare the framework's kernels, caches and engine with it; it shares no
code with them.  Everything is computed in the dtype of the weights it is given (float64 in most tests)."""
import math

import torch


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def unit_rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def yarn_frequencies(dims, base, scaling):
    """(frequencies [dims/2], magnitude of cos and sin) of a rotation over ``dims`` dimensions."""
    n = dims // 2
    f = [base ** (-2.0 * i / dims) for i in range(n)]
    if not scaling:
        return f, 1.0
    s, t0 = scaling["factor"], scaling["original"]

    def corr(turns):
        return dims * math.log(t0 / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(corr(scaling["fast"])), 0)
    hi = min(math.ceil(corr(scaling["slow"])), dims - 1)
    out = []
    for i in range(n):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / s * r + f[i] * (1 - r))
    return out, 0.1 * math.log(s) + 1.0


def rotate_interleaved(x, positions, freqs, mag):
    """x [T, ..., dims]: the pair (2i, 2i + 1) turned by position * freqs[i], lengths multiplied by mag."""
    y = x.clone()
    for t, p in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s = mag * math.cos(p * f), mag * math.sin(p * f)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * c - v * s
            y[t, ..., 2 * i + 1] = v * c + u * s
    return y


def sink_window_attention(q, k, v, scale, window, sink):
    """q, k [T, H, D], v [T, H, E]: causal attention over the last ``window`` positions (all when None); ``sink`` [H]
    adds exp(sink) to the denominator."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for t in range(T):
        a = 0 if window is None else max(0, t - window + 1)
        for h in range(H):
            s = (k[a:t + 1, h] @ q[t, h]) * scale
            m = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            out[t, h] = (e @ v[a:t + 1, h]) / (e.sum() + torch.exp(sink[h] - m))
    return out


def latent_attention(h, w, c, eps):
    """h [T, width] -> [T, width]; ``w``: the mixer's tensors by their leaf name, ``c``: its sizes."""
    T = h.shape[0]
    H, dn, dr, dv, r = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    q = unit_rms(h @ w["dq"].T, eps) * w["dq.norm"] @ w["uq"].T
    q = q.view(T, H, dn + dr)
    down = h @ w["dkv"].T
    lat = unit_rms(down[:, :r], eps) * w["dkv.norm"]
    freqs, mag = yarn_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
    pos = range(T)
    q_rot = rotate_interleaved(q[:, :, dn:], pos, freqs, mag)
    k_rot = rotate_interleaved(down[:, r:], pos, freqs, mag)
    k_up = (lat @ w["uk"].T).view(T, H, dn)
    v = (lat @ w["uv"].T).view(T, H, dv)
    qq = torch.cat([q[:, :, :dn], q_rot], -1)
    kk = torch.cat([k_up, k_rot[:, None].expand(T, H, dr)], -1)
    window = c["mask"]["size"] if c.get("mask") else None
    o = sink_window_attention(qq, kk, v, c["scale"], window, w["sink"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


def mlstm_recurrence(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, E], log gates i, f [T, H] -> [T, H, E]."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=v.dtype)
        n = torch.zeros(D, dtype=v.dtype)
        m = torch.zeros((), dtype=v.dtype)
        for t in range(T):
            m_new = torch.maximum(f[t, h] + m, i[t, h])
            keep, write = torch.exp(f[t, h] + m - m_new), torch.exp(i[t, h] - m_new)
            S = keep * S + write * torch.outer(k[t, h], v[t, h])
            n = keep * n + write * k[t, h]
            m = m_new
            out[t, h] = (S.T @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm_gates(h, w, cap):
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    z = cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-z))


def mlstm(h, w, c, eps):
    T = h.shape[0]
    H, d, e = c["heads"], c["dim"], c["vdim"]
    q = (h @ w["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].T).view(T, H, d)
    v = (h @ w["v"].T).view(T, H, e)
    i, f = mlstm_gates(h, w, c["gate_cap"])
    o = unit_rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * e)
    return (o * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def dense_gelu(h, up, down):
    z = h @ up.T
    return (0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))) @ down.T


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) gets the residual stream after every layer."""
    eps = cfg["norm"]["eps"]

    def norm(name, x):
        return dynamic_tanh(x, tensors[name + ".alpha"], tensors[name], tensors[name + ".b"])

    x = tensors["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for li, layer in enumerate(cfg["layers"]):
        owner = li
        while cfg["layers"][owner].get("weights_of") is not None:
            owner = cfg["layers"][owner]["weights_of"]
        p = f"l{owner}."
        w = {k[len(p) + 4:]: t for k, t in tensors.items() if k.startswith(p + "mix.")}
        x = x + MIXERS[layer["type"]](norm(p + "norm1", x), w, layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + dense_gelu(norm(p + "norm2", x), tensors[p + "mlp.up"], tensors[p + "mlp.down"])
        if layers_out is not None:
            layers_out.append(x)
    return norm("final.norm", x) @ tensors["head"].T
