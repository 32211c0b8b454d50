"""Plain, slow restatement of the Gerupel decoder: one function per mechanism, one sequence at a time, one query at a time.
The tests compare the framework's kernels, caches and engine with it; it shares no code with them.  Everything is computed in
the dtype of the weights it is given (float64 in most tests)."""
import math

import torch


def norm(x, w, eps):
    """x over its root mean square along the last dimension, times w."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def embed(tokens, table, w, eps):
    return norm(torch.stack([table[t] for t in tokens]), w, eps)


def frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair: long wavelengths are slowed down by ``factor``, short ones stay, those between
    are mixed."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2 * i / dims)
        if scaling is not None:
            turns = scaling["original"] * f / (2 * math.pi)  # in the original context
            low, high = scaling["low"], scaling["high"]
            if turns < low:
                f = f / scaling["factor"]
            elif turns <= high:
                s = (turns - low) / (high - low)
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, p, rot):
    """x [..., dim] at position p: the first rot.dims elements as pairs (i, i + dims / 2)."""
    n, y = rot["dims"], x.clone()
    for i, f in enumerate(frequencies(n, rot["base"], rot.get("scaling"))):
        c, s, j = math.cos(p * f), math.sin(p * f), i + n // 2
        y[..., i], y[..., j] = x[..., i] * c - x[..., j] * s, x[..., j] * c + x[..., i] * s
    return y


def sight(i, mask=None):
    """(tokens, blocks) that position i sees: a window, and the pooled blocks that ended before it."""
    if not mask or not mask.get("size"):
        return list(range(i + 1)), []
    size, P = mask["size"], mask.get("pool")
    tokens = [j for j in range(i + 1) if i - j < size]
    blocks = [b for b in range(i + 1) if b * P + P - 1 <= i - size] if P else []
    return tokens, blocks


def attend_one(q, k, v, scale, temp, mask, i):
    """The query [H, D] of position i over keys [T, G, D] and values [T, G, E], T > i -> [H, E].  Tokens and pooled blocks share a
    softmax with one more in its denominator."""
    tokens, blocks = sight(i, mask)
    P = (mask or {}).get("pool")
    keys = torch.cat([torch.stack([k[j] for j in tokens])] + [k[b * P:(b + 1) * P].mean(0)[None] for b in blocks])
    values = torch.cat([torch.stack([v[j] for j in tokens])] + [v[b * P:(b + 1) * P].mean(0)[None] for b in blocks])
    per, rows = q.shape[0] // k.shape[1], []
    for h in range(q.shape[0]):
        s = keys[:, h // per] @ q[h] * scale * temp[h]
        top = s.max().clamp(min=0)
        e = torch.exp(s - top)
        rows.append(e @ values[:, h // per] / (torch.exp(-top) + e.sum()))
    return torch.stack(rows)


def attention(h, w, c):
    """The windowed half: [T, width] -> [T, width]."""
    T, H, G, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, e)
    if c.get("rot"):
        q, k = (torch.stack([rotate(x[t], t, c["rot"]) for t in range(T)]) for x in (q, k))
    o = torch.stack([attend_one(q[t], k[:t + 1], v[:t + 1], c["scale"], w["temp"], c.get("mask"), t) for t in range(T)])
    return o.reshape(T, H * e) @ w["o"].T


def forget(z, lower):
    """Forget gates between ``lower`` and one."""
    return lower + (1 - lower) / (1 + torch.exp(-z))


def recurrence(q, f, v, S=None):
    """q, f [T, H, D], v [T, H, E] -> (o [T, H, E], state [H, D, E]); the gate that forgets also writes."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=v.dtype) if S is None else S
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def linear_attention(h, w, c, eps):
    """The recurrent half: [T, width] -> [T, width]."""
    T, H, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = silu(h @ w["q"].T).view(T, H, d)
    f = forget(h @ w["f"].T + w["f.b"], w["lower"]).view(T, H, d)
    o, _ = recurrence(q, f, (h @ w["v"].T).view(T, H, e))
    return norm(o, w["norm"], eps).reshape(T, H * e) @ w["o"].T


def parallel(h, w, c, eps):
    def side(name):
        return {k[len(name) + 1:]: t for k, t in w.items() if k.startswith(name + ".")}

    return c["left_scale"] * attention(h, side("left"), c["left"]) + c["right_scale"] * linear_attention(h, side("right"), c["right"], eps)


def route(z, top, scale):
    """Logits of one token -> [(expert, weight)]."""
    s = torch.softmax(z, 0)
    chosen = sorted(range(len(s)), key=lambda e: -float(s[e]))[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * scale) for e in chosen]


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def expert_mlp(h, w, c):
    out, r = torch.zeros_like(h), c["router"]
    for t in range(h.shape[0]):
        for e, s in route(w["router"] @ h[t], r["top"], r["scale"]):
            out[t] += s * expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def runs(cfg):
    """[(layer, pass that begins in front of it or None)] in the order of computation."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) gets the residual stream after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    first = x = embed(list(tokens), tensors["embed"], tensors["embed.norm"], eps)
    for li, t in runs(cfg):
        if t is not None:
            x = x + (first if t > 0 else 0) + tensors["loop.step"][t]
        p, layer = f"l{li}.", cfg["layers"][li]
        w = {k[len(p) + 4:]: v for k, v in tensors.items() if k.startswith(p + "mix.")}
        y = parallel(norm(x, tensors[p + "norm1"], eps), w, layer["mixer"], eps)
        if layer["mlp"] is not None:
            w = {k[len(p) + 4:]: v for k, v in tensors.items() if k.startswith(p + "mlp.")}
            y = y + expert_mlp(norm(x, tensors[p + "norm2"], eps), w, layer["mlp"])
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, tensors["final.norm"], eps) @ tensors["embed"].T
