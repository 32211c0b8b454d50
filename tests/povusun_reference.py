"""Plain, slow restatement of the Povusun decoder: one function per mechanism, one sequence at a time, every recurrence
run token by token.  The tests compare the framework's kernels, caches and engine with it; it shares no code with
them.  Everything is computed in the dtype of the weights it is given (float64 in most tests)."""
import math

import torch


def unit_rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def temperature(p, coef, every):
    """Factor of the query at position ``p``."""
    return 1 + coef * math.log(math.floor((p + 1) / every) + 1)


def cap_scores(s, cap):
    return s if cap is None else cap * torch.tanh(s / cap)


def grouped_attention(q, k, v, scale, cap):
    """q [T, H, D], k [T, G, D], v [T, G, E]; query head h reads key/value head h // (H / G); causal."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            s = cap_scores(k[:t + 1, h // per] @ q[t, h] * scale, cap)
            e = torch.exp(s - s.max())
            out[t, h] = (e @ v[:t + 1, h // per]) / e.sum()
    return out


def attention(h, w, c, eps, kept=None):
    """h [T, width] -> ([T, width], (keys, values)); ``kept``: the keys and values of the layer this one borrows from."""
    T = h.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = unit_rms((h @ w["q"].T).view(T, H, d), eps)
    if c.get("q_temp"):
        f = [temperature(p, c["q_temp"]["coef"], c["q_temp"]["every"]) for p in range(T)]
        q = q * torch.tensor(f, dtype=h.dtype)[:, None, None]
    if kept is None:
        kept = unit_rms((h @ w["k"].T).view(T, G, d), eps), (h @ w["v"].T).view(T, G, e)
    o = grouped_attention(q, *kept, c["scale"], c.get("softcap"))
    return (o.reshape(T, H * e) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, kept


def latent_attention(h, w, c, eps):
    T = h.shape[0]
    H, d, e = c["heads"], c["dim"], c["vdim"]
    q = (h @ w["q"].T).view(T, H, d)
    lat = rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps)
    k, v = (lat @ w["uk"].T).view(T, H, d), (lat @ w["uv"].T).view(T, H, e)
    return grouped_attention(q, k, v, c["scale"], None).reshape(T, H * e) @ w["o"].T


def causal_conv(x, taps, bias):
    """x [T, C]; taps [C, n], the last column weighs the current token."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            if t - j >= 0:
                y[t] += taps[:, n - 1 - j] * x[t - j]
    return y + bias


def block_gate(u, w, b):
    """sigmoid of a block-diagonal product: u [T, C], w [blocks, C / blocks (out), C / blocks (in)]."""
    n = w.shape[0]
    parts = u.view(u.shape[0], n, -1)
    return torch.stack([torch.sigmoid(parts[:, i] @ w[i].T + b[i]) for i in range(n)], 1).reshape(u.shape)


def rglru_recurrence(u, r, i, lam):
    S = torch.zeros_like(u[0])
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * torch.log1p(torch.exp(lam))
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru(h, w, c, eps):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    S = rglru_recurrence(u, block_gate(u, w["ra"], w["ra.b"]), block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return (S * y) @ w["o"].T


def clamped_glu(h, gate, up, down, limit):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def side_input(x, e, gate, proj, norm, eps):
    return rms_norm((gelu_tanh(x @ gate.T) * e) @ proj.T, norm, eps)


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) gets the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens)
    x = tensors["embed"][ids]
    kept = {}
    for li, layer in enumerate(cfg["layers"]):
        p = f"l{li}."
        w = {k[len(p) + 4:]: t for k, t in tensors.items() if k.startswith(p + "mix.")}
        h, c = rms_norm(x, tensors[p + "norm1"], eps), layer["mixer"]
        if layer["type"] == "attention":
            y, kept[li] = attention(h, w, c, eps, kept[c["kv_from"]] if c.get("kv_from") is not None else None)
        else:
            y = {"latent_attention": latent_attention, "rglru": rglru}[layer["type"]](h, w, c, eps)
        x = x + rms_norm(y, tensors[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            h = rms_norm(x, tensors[p + "norm2"], eps)
            y = clamped_glu(h, tensors[p + "mlp.gate"], tensors[p + "mlp.up"], tensors[p + "mlp.down"], layer["mlp"]["limit"])
            x = x + rms_norm(y, tensors[p + "norm2b"], eps)
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + side_input(x, tensors["side.embed"][ids, li * n:(li + 1) * n], tensors[p + "side.gate"],
                               tensors[p + "side.proj"], tensors[p + "side.norm"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, tensors["final.norm"], eps) @ tensors["embed"].T
