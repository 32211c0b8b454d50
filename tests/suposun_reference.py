"""Plain, slow restatement of the Suposun decoder: one function per mechanism, one sequence at a time, one query at a time.
The tests compare the framework's kernels, caches and engine with it; it shares no code with them.  Everything is computed in
the dtype of the weights it is given (float64 in most tests)."""
import math

import torch


def unit_rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_about_zero(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1 + w)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_row(prev, cur, mul_prev, mul_cur, buckets):
    """Row of the pair table; ``prev`` is None at a sequence's first token."""
    return buckets if prev is None else (prev * mul_prev + cur * mul_cur) % buckets


def embed(tokens, table, scale, pairs=None, spec=None):
    rows = []
    for t, tok in enumerate(tokens):
        x = table[tok] * scale
        if pairs is not None:
            x = x + pairs[bigram_row(tokens[t - 1] if t else None, tok, spec["mul_prev"], spec["mul_cur"], spec["buckets"])]
        rows.append(x)
    return torch.stack(rows)


def frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair, and the factor of cosine and sine."""
    f = [base ** (-2 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0

    def place(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / scaling["factor"] * ramp + f[i] * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, p, rot, halves):
    """x [..., dim] at position p: the first rot.dims elements as pairs (2i, 2i + 1), or (i, i + dims / 2) with ``halves``."""
    n = rot["dims"]
    freq, mag = frequencies(n, rot["base"], rot.get("scaling"))
    y = x.clone()
    for i, f in enumerate(freq):
        a, b = (i, i + n // 2) if halves else (2 * i, 2 * i + 1)
        c, s = math.cos(p * f) * mag, math.sin(p * f) * mag
        y[..., a], y[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
    return y


def visible(i, mask=None):
    """The positions that position i attends to."""
    mask = mask or {}
    size, keep = mask.get("size"), mask.get("keep_first", 0)
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep]


def attend(q, k, v, scale, cap=None, mask=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=v.dtype)
    for t in range(T):
        out[t] = attend_one(q[t], k[visible(t, mask)], v[visible(t, mask)], scale, cap, sink, per)
    return out


def attend_one(q, k, v, scale, cap, sink, per):
    """One query [H, D] over the keys it sees."""
    rows = []
    for h in range(q.shape[0]):
        s = k[:, h // per] @ q[h] * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
        e = torch.exp(s - top)
        total = e.sum() + (0 if sink is None else torch.exp(sink[h] - top))
        rows.append((e @ v[:, h // per]) / total)
    return torch.stack(rows)


def key_value_attention(h, w, c, eps):
    """Mixer 'attention': values are the projected keys, norms per head, adjacent pairs rotated, sink, gate per head."""
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    raw = (h @ w["k"].T).view(T, G, d)
    q = unit_rms((h @ w["q"].T).view(T, H, d), eps) * w["q.norm"]
    k = unit_rms(raw, eps) * w["k.norm"]
    if c.get("rot"):
        q = torch.stack([rotate(q[t], t, c["rot"], False) for t in range(T)])
        k = torch.stack([rotate(k[t], t, c["rot"], False) for t in range(T)])
    o = attend(q, k, raw, c["scale"], c.get("softcap"), c.get("mask"), w["sink"])
    o = o * torch.sigmoid(h @ w["g"].T)[..., None]
    return o.reshape(T, H * d) @ w["o"].T


def whole_norm_attention(h, w, c, eps, kept=None):
    """Mixer 'attention_2': norms over all heads at once, halves rotated.  Returns ([T, width], (keys, values)); ``kept``: those
    of the layer this one borrows from."""
    T, H, G, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def turned(x, n):
        x = x.view(T, n, d)
        return torch.stack([rotate(x[t], t, c["rot"], True) for t in range(T)]) if c.get("rot") else x

    q = turned(unit_rms(h @ w["q"].T, eps) * w["q.norm"], H)
    if kept is None:
        kept = turned(unit_rms(h @ w["k"].T, eps) * w["k.norm"], G), (h @ w["v"].T).view(T, G, e)
    o = attend(q, *kept, c["scale"], c.get("softcap"), c.get("mask"))
    return o.reshape(T, H * e) @ w["o"].T, kept


def dense_mlp(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def expert(h, gate, up, down, limit):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, router, correction, top):
    """One token: [(expert, weight)], chosen by the corrected scores and weighted by the bare ones."""
    s = torch.sigmoid(router @ h)
    order = sorted(range(len(s)), key=lambda e: -float(s[e] + correction[e]))
    return [(e, s[e]) for e in order[:top]]


def expert_mlp(h, w, c):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in route(h[t], w["router"], w["correction"], c["router"]["top"]):
            out[t] += s * expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], c["expert"]["limit"])
    return out


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) gets the residual stream after every layer."""
    eps, emb = cfg["norm"]["eps"], cfg.get("embedding") or {}
    x = embed(list(tokens), tensors["embed"], emb.get("scale", 1.0), tensors.get("bigram"), emb.get("bigram"))
    kept = {}
    for li, layer in enumerate(cfg["layers"]):
        p = f"l{li}."
        w = {k[len(p) + 4:]: t for k, t in tensors.items() if k.startswith(p + "mix.")}
        c = layer["mixer"]
        if layer["type"] == "attention":
            y = key_value_attention(x, w, c, eps)
        else:
            y, kept[li] = whole_norm_attention(x, w, c, eps, kept[c["kv_from"]] if c.get("kv_from") is not None else None)
        x = x + norm_about_zero(y, tensors[p + "norm1"], eps) * tensors[p + "ls1"]
        if layer["mlp"] is not None:
            w = {k[len(p) + 4:]: t for k, t in tensors.items() if k.startswith(p + "mlp.")}
            y = dense_mlp(x, w) if layer["mlp"]["kind"] == "dense" else expert_mlp(x, w, layer["mlp"])
            x = x + norm_about_zero(y, tensors[p + "norm2"], eps) * tensors[p + "ls2"]
        if layers_out is not None:
            layers_out.append(x)
    return norm_about_zero(x, tensors["final.norm"], eps) @ tensors["embed"].T * cfg.get("logit_scale", 1.0)
