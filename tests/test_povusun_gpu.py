"""Povusun on the GPU: every kernel of its mechanisms, the serving engine's caches and states, generation.

Models are compared with the plain restatement (povusun_reference.py) in float64; float32 models are held to rounding, bf16
models to bf16 rounding, and where that could hide a fault (a far key, a page border, a slow decay) the inputs are made so
that one score or one step stands out."""
import functools
import types

import pytest
import torch

import povusun_reference as ref
import povusun_util as U
from trl_b200.models import SeqCtx
from trl_b200.rollout.sampling import SamplingParams

pytestmark = pytest.mark.gpu

CFGS = {"odd": U.ODD, "tiles": U.TILES, "ones": U.ONES}
DTYPES = [torch.float32, torch.bfloat16]
f64 = torch.float64


def tol(name, dtype):
    # eight channels: a norm over eight values can blow up the rounding of a small one (typical rows are ten times better)
    return 2e-5 if dtype == torch.float32 else 0.2 if name == "ones" else 0.06


def dev(x, dtype=torch.float32):
    return x.to("cuda", dtype)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=f64)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


@functools.lru_cache(maxsize=None)
def model(name, dtype):
    return U.make(CFGS[name], dtype, "cuda")


@functools.lru_cache(maxsize=None)
def wanted(name, n, seed):
    toks = U.tokens(n, CFGS[name]["vocab"], seed)
    _, t = U.make(CFGS[name])
    return toks, U.logits(CFGS[name], t, toks)


def feed(name, dtype, slots=4, max_len=512, block=None, blocks=None):
    from trl_b200.rollout.engine import make_engine
    from trl_b200.rollout.feed import TokenFeed

    return TokenFeed(make_engine(model(name, dtype)[0], max_num_seqs=slots, max_model_len=max_len, block_size=block,
                                 num_blocks=blocks))


# ---- norms, feed-forward, side input ------------------------------------------------------------------------------
@pytest.mark.parametrize("H", [8, 33, 84, 1024, 1540, 4096, 8192, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_rms_residual(H, dtype):
    from trl_b200.ops import cuda_mixers as K

    r = gen(H)
    x, d, p, w = r(5, H) * 3, r(5, H) * 0.01, r(H), r(H)
    eps, t = 1e-4, (2e-6 if dtype == torch.float32 else 2e-2)
    for post, norm in ((p, w), (None, w), (p, None), (None, None)):
        for delta in (d, None):
            s = x if delta is None else x + (delta if post is None else ref.rms_norm(delta, post, eps))
            want = s if norm is None else ref.rms_norm(s, norm, eps)
            xg, dg = dev(x), None if delta is None else dev(delta)
            got = K.rms_residual(xg, dg, None if post is None else dev(post), None if norm is None else dev(norm), eps, dtype, clear=True)
            assert torch.allclose(got.double().cpu(), want, atol=t, rtol=t)
            assert torch.allclose(xg.double().cpu(), s, atol=1e-5, rtol=1e-6) and (dg is None or not dg.any())


@pytest.mark.parametrize("n", [1, 50, 136])
@pytest.mark.parametrize("limit", [0.6, 7.0])
@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_glu(n, limit, dtype):
    from trl_b200.ops import cuda_mixers as K

    z = (gen(n)(9, 2 * n) * 4).to(dtype).double()
    g, u = z[:, :n].clamp(max=limit), z[:, n:].clamp(-limit, limit)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    t = 2e-6 if dtype == torch.float32 else 1e-2
    assert torch.allclose(K.clamped_glu(dev(z, dtype), limit, 1.702, 1.0).double().cpu(), want, atol=t, rtol=t)


@pytest.mark.parametrize("B", [1, 20, 64, 100])
@pytest.mark.parametrize("n,k", [(24, 40), (128, 64), (200, 136), (1000, 72)])
def test_clamped_glu_in_the_decode_product(B, n, k):
    """Gate and up rows that do not start on a 128-row slab."""
    from trl_b200.ops import cuda as KC

    r = gen(B + n)
    x, w = r(B, k).bfloat16(), (r(2 * n, k) / k ** 0.5 * 2).bfloat16()
    z = x.double() @ w.double().T
    g, u = z[:, :n].clamp(max=1.1), z[:, n:].clamp(-1.1, 1.1)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    got = KC.decode_gemm(x.cuda(), w.cuda(), clamped_glu=(1.1, 1.702, 1.0))
    assert got.shape == (B, n) and torch.allclose(got.double().cpu(), want, atol=1e-2, rtol=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [5, 40, 260])
def test_side_gate(n, dtype):
    from trl_b200.ops import cuda_mixers as K

    r = gen(n)
    table, ids = r(11, 3 * n).to(dtype), torch.tensor([10, 0, 3, 3])
    for zt in {torch.float32, dtype}:
        z = (r(4, n) * 3).to(zt)
        zg = z.cuda()
        got = K.side_gate(zg, ids.cuda(), table.cuda(), 2 * n, clear=True)
        want = ref.gelu_tanh(z.double()) * table.double()[ids, 2 * n:]
        t = 2e-6 if dtype == torch.float32 else 1e-2
        assert torch.allclose(got.double().cpu(), want, atol=t, rtol=t) and not zg.any()


# ---- attention ----------------------------------------------------------------------------------------------------
def mixer(H, G, d, e, **kw):
    return types.SimpleNamespace(**{**dict(heads=H, kv_heads=G, dim=d, vdim=e, scale=0.3, cap=None, kv_from=None, eps=1e-5), **kw})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e", [(6, 3, 20, 28), (4, 1, 64, 128), (3, 3, 9, 5), (10, 2, 136, 8)])
@pytest.mark.parametrize("own", [True, False])
def test_attention_preparation(H, G, d, e, own, dtype):
    """Prompt rows (in place) and decode sums (cleared): unit-rms queries times the temperature, keys and values in the pages."""
    from trl_b200.ops import cuda_mixers as K

    r, rows, bs = gen(H + d), 5, 4
    m = mixer(H, G, d, e, kv_from=None if own else 0, o=torch.empty(0, dtype=dtype))
    kv = G if own else 0
    y = (r(rows, H * d + kv * (d + e) + H * e) * 2).to(dtype).double()
    pos, temp = [0, 3, 4, -1, 9], torch.linspace(1, 3, 12, dtype=f64)
    table = torch.tensor([[5, 1, 3], [2, 4, 6], [7, 8, 9], [10, 11, 12], [13, 14, 15]], dtype=torch.int32)
    q, k, v, g = y.split([H * d, kv * d, kv * e, H * e], 1)
    f = torch.tensor([temp[p] if p >= 0 else 1.0 for p in pos])[:, None, None]
    wq = ref.unit_rms(q.view(rows, H, d), 1e-5) * f
    wk = ref.unit_rms(k.view(rows, kv, d), 1e-5)
    t = 3e-6 if dtype == torch.float32 else 2e-2
    for sums in (False, True):
        kc, vc = torch.full((16, bs, G, d), 9.0, dtype=dtype, device="cuda"), torch.full((16, bs, G, e), 9.0, dtype=dtype, device="cuda")
        where = dict(k_cache=kc, v_cache=vc, block_table=table.cuda(), block_size=bs) if own else {}
        src = dev(y, torch.float32 if sums else dtype)
        buf = dict(q=torch.zeros(rows, H, d, dtype=dtype, device="cuda"), g=torch.zeros(rows, H * e, dtype=dtype, device="cuda")) if sums else {}
        K.attn_prep(src, m, i32(pos), dev(temp), **buf, **where)
        if sums:
            assert not src.any() and torch.allclose(buf["g"].double().cpu(), g, atol=t, rtol=t)
            got = buf["q"].double().cpu()
        else:
            got = src[:, :H * d].double().cpu().view(rows, H, d)
            assert torch.allclose(src[:, H * d:H * d + kv * d].double().cpu().view(rows, kv, d), wk, atol=t, rtol=t)
            assert torch.equal(src[:, H * d + kv * d:].double().cpu(), torch.cat([v, g], 1))
        assert torch.allclose(got, wq, atol=3 * t, rtol=t)
        written = 0
        for i, p in enumerate(pos):
            if p >= 0 and own:
                at = int(table[i, p // bs]), p % bs
                assert torch.allclose(kc[at].double().cpu(), wk[i], atol=t, rtol=t)
                assert torch.allclose(vc[at].double().cpu(), v[i].view(G, e), atol=t, rtol=t)
                written += 1
        assert int((kc != 9.0).flatten(2).any(2).sum()) == written


SHAPES = [(6, 3, 20, 28), (4, 4, 72, 48), (8, 1, 128, 128), (20, 2, 72, 136), (2, 1, 13, 9), (3, 1, 256, 256), (2, 2, 8, 8)]


def run_prompt(q, k, v, g, m, lens, dtype, tc=True):
    """Strided rows, as the projections leave them."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T = q.shape[0]
    y = dev(torch.cat([t.reshape(T, -1) for t in (q, k, v, g)], 1), dtype)
    qq, kk, vv, gg = y.split([q[0].numel(), k[0].numel(), v[0].numel(), g[0].numel()], 1)
    out = K.mixer_attn(qq, kk, vv, heads=m.heads, kv_heads=m.kv_heads, scale=m.scale, cap=m.cap, gate_logits=gg,
                       ctx=SeqCtx.from_lengths(lens, "cuda"), tensor_cores=tc)
    KC.check_status()
    return out.double().cpu().view(T, m.heads, m.vdim)


def want_prompt(q, k, v, g, m, lens):
    outs, a = [], 0
    for n in lens:
        outs.append(ref.grouped_attention(q[a:a + n], k[a:a + n], v[a:a + n], m.scale, m.cap))
        a += n
    return torch.cat(outs) * torch.sigmoid(g).view(-1, m.heads, m.vdim)


def attention_case(T, m, dtype, seed):
    r = gen(seed)
    return tuple(t.to(dtype).double() for t in (r(T, m.heads, m.dim), r(T, m.kv_heads, m.dim), r(T, m.kv_heads, m.vdim), r(T, m.heads * m.vdim)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("cap,scale", [(None, 0.1), (3.0, 0.1), (3.0, 0.7), (60.0, 0.02)])
def test_prompt_attention(shape, cap, scale, dtype):
    """Capped scores on all sides of where the polynomials for tanh end (small, middling and large scores)."""
    m, lens = mixer(*shape, cap=cap, scale=scale), [1, 150, 37, 2]
    case = attention_case(sum(lens), m, dtype, shape[2])
    want = want_prompt(*case, m, lens)
    for tc in (True, False):
        got = run_prompt(*case, m, lens, dtype, tc)
        t = 2e-5 if dtype == torch.float32 else 1e-2
        assert (got - want).abs().max() < t * want.abs().max()


@pytest.mark.parametrize("x", [0.01, 0.11, 0.13, 0.3, 0.36, 1.0, 5.0])
def test_capped_scores(x):
    """Two keys whose scores are +- cap x: the ratio of their weights gives the capped difference back."""
    cap = 8.0
    m = mixer(1, 1, 8, 8, scale=1.0, cap=cap)
    q, k, v, g = (torch.zeros(2, *s, dtype=f64) for s in ((1, 8), (1, 8), (1, 8), (8,)))
    q[1, 0, 0] = 1.0
    k[0, 0, 0], k[1, 0, 0] = cap * x, -cap * x
    k = k.bfloat16().double()
    v[0, 0, 0], v[1, 0, 1] = 1.0, 1.0
    w = torch.softmax(cap * torch.tanh(torch.stack([k[0, 0, 0], k[1, 0, 0]]) / cap), 0)
    for dtype in DTYPES:
        got = 2 * run_prompt(q, k, v, g, m, [2], dtype)[1, 0]  # gates of logit zero
        assert torch.allclose(got[:2], w, rtol=5e-3 if dtype == torch.bfloat16 else 1e-5, atol=1e-9)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap", [None, 30.0])
@pytest.mark.parametrize("distance", [0, 1, 127, 128, 129, 255, 256, 257])
def test_prompt_attention_far_key(distance, cap, dtype):
    """One key at a chosen distance outweighs all others: its value comes out alone, also across tile borders."""
    T, m = 258, mixer(4, 2, 64, 40, scale=1.0, cap=cap)
    q, k, v, g = attention_case(T, m, dtype, distance)
    q, k = q * 0.1, k * 0.1
    at = [t for t in (distance, 128, 200, 257) if t >= distance]
    for t in at:
        u = torch.nn.functional.normalize(gen(t)(64), dim=0) * 5
        q[t], k[t - distance] = u.to(dtype).double(), u.to(dtype).double()
    got = run_prompt(q, k, v, g, m, [T], dtype)
    for t in at:
        alone = v[t - distance].repeat_interleave(2, 0) * torch.sigmoid(g[t]).view(4, 40)
        assert (got[t] - alone).abs().max() < 0.03, (t, distance)


def test_many_prompt_tiles_finish():
    """Enough tiles that CTAs share SMs, prompts of several tiles: no wait runs out and runs repeat bit by bit."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T, H = 3072, 16
    r = torch.Generator(device="cuda").manual_seed(0)
    for d, e in ((128, 128), (64, 64), (192, 128), (72, 136)):
        q, k, v, g = (torch.randn(T, H * n, device="cuda", generator=r).bfloat16() for n in (d, d, e, e))
        ctx = SeqCtx.from_lengths([1024, 1, 1000, 1047], "cuda")
        for cap in (None, 20.0):
            outs = [K.mixer_attn(q, k, v, heads=H, kv_heads=H, scale=0.05, cap=cap, gate_logits=g, ctx=ctx) for _ in range(4)]
            KC.check_status()
            assert all(torch.equal(o, outs[0]) for o in outs) and torch.isfinite(outs[0]).all()


def paged(rows, bs, seed):
    """rows: per slot [n, ...] tensors -> (cache, table); pages in random order, unused rows hold a constant."""
    pages = [max(1, -(-len(r) // bs)) for r in rows]
    order = (torch.randperm(sum(pages), generator=torch.Generator().manual_seed(seed)) + 1).tolist()
    cache = torch.full((sum(pages) + 1, bs) + tuple(rows[0].shape[1:]), 3.0, dtype=f64)
    table = torch.zeros(len(rows), max(pages), dtype=torch.int32)
    for i, r in enumerate(rows):
        for p in range(pages[i]):
            table[i, p] = order.pop()
            part = r[p * bs:(p + 1) * bs]
            cache[table[i, p], :len(part)] = part
    return cache, table


def alone(q, k, v, m):
    """One query [heads, dim] over all keys: the last row of the restatement."""
    pad = torch.zeros(len(k) - 1, *q.shape, dtype=f64)
    per, rows = m.heads // m.kv_heads, []
    if len(k) < 130:
        return ref.grouped_attention(torch.cat([pad, q[None]]), k, v, m.scale, m.cap)[-1]
    for h in range(m.heads):
        s = ref.cap_scores(k[:, h // per] @ q[h] * m.scale, m.cap)
        e = torch.exp(s - s.max())
        rows.append(e @ v[:, h // per] / e.sum())
    return torch.stack(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape,bs,cap,scale", [((6, 3, 20, 28), 16, 4.0, 0.3), ((8, 2, 128, 128), 64, None, 0.09), ((20, 2, 72, 136), 32, 2.0, 0.5),
                                                ((4, 4, 64, 48), 128, 30.0, 0.05), ((9, 1, 8, 256), 8, 5.0, 0.4), ((2, 2, 256, 64), 64, None, 0.06),
                                                ((16, 1, 192, 40), 64, 50.0, 0.1), ((3, 1, 9, 5), 16, 1.0, 0.5)])
def test_decode_attention(shape, bs, cap, scale, dtype):
    """Ragged slots (idle ones included), several tiles and splits, groups above eight heads, both kernels."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    m, r = mixer(*shape, cap=cap, scale=scale), gen(sum(shape))
    lens = [0, 300, -1, 127, 128, 5, 255, 256]
    B = len(lens)
    ks = [(r(max(1, n + 1), m.kv_heads, m.dim) * 2).to(dtype).double() for n in lens]
    vs = [r(max(1, n + 1), m.kv_heads, m.vdim).to(dtype).double() for n in lens]
    kc, table = paged(ks, bs, 3)
    vc, _ = paged(vs, bs, 3)
    q, g = (r(B, m.heads, m.dim) * 2).to(dtype).double(), r(B, m.heads * m.vdim).to(dtype).double()
    args = (dev(q, dtype), dev(kc, dtype), dev(vc, dtype), m, i32(lens), table.cuda(), bs)
    outs = []
    for splits in ((0, 1, 3) if dtype == torch.bfloat16 and K.grouped_decode_tc_ok(m, bs) else (0,)):
        out = torch.full((B, m.heads * m.vdim), 7.0, dtype=dtype, device="cuda")
        if splits:
            part = torch.full((B, m.heads * splits * m.vdim), 5.0, device="cuda"), torch.full((B, m.heads * splits * 2), 5.0, device="cuda")
            K.grouped_decode_tc(*args, out, dev(g, dtype), splits, *part)
        else:
            K.grouped_decode(*args, out, dev(g, dtype))
        outs.append(out.double().cpu().view(B, m.heads, m.vdim))
    KC.check_status()
    assert len(outs) == 3 or dtype == torch.float32 or shape[2] % 8 or shape[3] % 8
    for b, n in enumerate(lens):
        if n < 0:
            continue
        want = alone(q[b], ks[b], vs[b], m) * torch.sigmoid(g[b]).view(m.heads, m.vdim)
        for got in outs:
            assert (got[b] - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pos,target", [(0, 0), (15, 0), (16, 0), (127, 127), (128, 0), (200, 0), (200, 127), (200, 128), (200, 200), (63, 47)])
def test_decode_attention_far_key(pos, target, dtype):
    from trl_b200.ops import cuda_mixers as K

    m, r, bs = mixer(4, 2, 64, 40, scale=1.0, cap=30.0), gen(pos + target), 16
    k, v, q = r(pos + 1, 2, 64) * 0.1, r(pos + 1, 2, 40), r(2, 4, 64) * 0.1
    u = torch.nn.functional.normalize(r(64), dim=0) * 5
    q[1], k[target] = u, u
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    (kc, table), (vc, _) = paged([k[:1], k], bs, pos), paged([v[:1], v], bs, pos)
    args = (dev(q, dtype), dev(kc, dtype), dev(vc, dtype), m, i32([-1, pos]), table.cuda(), bs)
    for tc in (False, True) if dtype == torch.bfloat16 else (False,):
        out = torch.full((2, 4 * 40), 7.0, dtype=dtype, device="cuda")
        (K.grouped_decode_tc if tc else K.grouped_decode)(*args, out)
        assert (out[1].double().cpu().view(4, 40) - v[target].repeat_interleave(2, 0)).abs().max() < 0.03


def test_many_idle_slots_in_decode():
    """More items than CTAs, most of them empty."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    m, r, B = mixer(8, 8, 64, 64, scale=0.1, cap=9.0), gen(1), 100
    lens = [-1] * B
    for b in (0, 1, 37, 62, 99):
        lens[b] = 3 * b + 2
    rows = [r(max(1, n + 1), 8, 64).bfloat16().double() for n in lens]
    cache, table = paged(rows, 64, 5)
    q = r(B, 8, 64).bfloat16().double()
    out = torch.full((B, 512), 7.0, dtype=torch.bfloat16, device="cuda")
    K.grouped_decode_tc(dev(q, torch.bfloat16), dev(cache, torch.bfloat16), dev(cache, torch.bfloat16), m, i32(lens), table.cuda(), 64, out)
    KC.check_status()
    for b, n in enumerate(lens):
        want = alone(q[b], rows[b], rows[b], m) if n >= 0 else torch.zeros(8, 64, dtype=f64)
        assert (out[b].double().cpu().view(8, 64) - want).abs().max() < 1e-2 * 4


def test_latent_attention_without_positions_gates_or_sink():
    """The latent mixer's decode kernels in the form that has only queries and latents."""
    from trl_b200.ops import cuda_mixers as K

    for H, rank, dtype in ((3, 40, torch.float32), (3, 40, torch.bfloat16), (40, 128, torch.bfloat16)):
        r, bs, lens = gen(H), 16, [70, -1, 0, 130]
        m = types.SimpleNamespace(heads=H, kv_rank=rank, rot_dim=0, dim=8, vdim=8, window=None, scale=0.2, sink=None)
        rows = [r(max(1, n + 1), rank).to(dtype).double() for n in lens]
        cache, table = paged(rows, bs, 1)
        q = r(4, H, rank).to(dtype).double()
        args = (dev(q, dtype), dev(cache, dtype), m, i32(lens), table.cuda(), bs)
        outs = [torch.zeros(4, H, rank, dtype=dtype, device="cuda") for _ in range(3)]
        K.latent_decode(*args, outs[0])
        if dtype == torch.bfloat16:
            for splits, out in ((1, outs[1]), (2, outs[2])):
                K.latent_decode_tc(*args, out, torch.full((4, H * splits * rank), 5.0, device="cuda"), torch.full((4, H * splits * 2), 5.0, device="cuda"), splits)
        for b, n in enumerate(lens):
            if n >= 0:
                w = torch.softmax(q[b] @ rows[b].T * 0.2, -1) @ rows[b]
                for out in outs[:3 if dtype == torch.bfloat16 else 1]:
                    assert (out[b].double().cpu() - w).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(w.abs().max()))


# ---- recurrence ---------------------------------------------------------------------------------------------------
def recurrent(C, blocks, taps, dtype, lam=None, seed=0):
    r = gen(seed + C)
    w = C // blocks
    p = dict(gates=(2 * r(2, blocks, w, w) / w ** 0.5).to(dtype).double(), gate_bias=r(2, C), y_bias=r(C), x_bias=r(C), conv=r(C, taps),
             conv_bias=r(C), lam=-4 + 3 * r(C) if lam is None else torch.full((C,), lam, dtype=f64))
    p = {k: v if k == "gates" else v.float().double() for k, v in p.items()}
    m = types.SimpleNamespace(width=C, blocks=blocks, taps=taps, decay=8.0, **{k: dev(v, dtype if k == "gates" else torch.float32) for k, v in p.items()})
    return m, types.SimpleNamespace(**p)


def want_recurrence(u, y, p, blocks):
    r = ref.block_gate(u, p.gates[0], p.gate_bias[0].view(blocks, -1))
    i = ref.block_gate(u, p.gates[1], p.gate_bias[1].view(blocks, -1))
    S = ref.rglru_recurrence(u, r, i, p.lam)
    return S, S * ref.gelu_tanh(y + p.y_bias)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(60, 3), (33, 1), (128, 4), (260, 6), (8, 2)])
def test_convolution(C, taps, dtype):
    """Prompts shorter and longer than the taps and than a thread's run of tokens; then one step from the kept inputs."""
    from trl_b200.ops import cuda_mixers as K

    m, p = recurrent(C, 1, taps, dtype)
    lens, slots = [1, 40, 2, 17, 5], [3, 0, 5, 1, 2]
    T, r = sum(lens), gen(taps)
    both = r(T, 2 * C).to(dtype).double()
    x = both[:, C:] + p.x_bias
    state = torch.full((6, taps - 1, C), 7.0, device="cuda")
    got = K.conv_prompt(dev(both, dtype)[:, C:], m, SeqCtx.from_lengths(lens, "cuda"), i32(slots), state).double().cpu()
    nxt = r(6, 2 * C)
    live = i32([7, 7, 7, 7, -1, 7])
    sums, u = dev(nxt), torch.full((6, C), 3.0, dtype=dtype, device="cuda")
    K.conv_step(sums[:, C:], m, live, state, u)
    assert not sums[:, C:].any() and sums[:, :C].all()
    kept, a, t = state.double().cpu(), 0, (1e-5 if dtype == torch.float32 else 2e-2)
    for n, s in zip(lens, slots):
        seq = torch.cat([x[a:a + n], nxt[s:s + 1, C:] + p.x_bias])
        want = ref.causal_conv(seq, p.conv, p.conv_bias)
        assert (got[a:a + n] - want[:n]).abs().max() < t * want.abs().max()
        assert (u[s].double().cpu() - want[n]).abs().max() < t * want.abs().max()
        if taps > 1:
            tail = torch.cat([torch.zeros(taps, C, dtype=f64), seq])[-(taps - 1):]
            assert torch.allclose(kept[s], tail, atol=1e-5)
        a += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,blocks,lam", [(60, 4, None), (33, 1, None), (272, 2, None), (96, 4, None), (128, 1, -14.0), (128, 1, 4.0), (256, 1, None), (320, 1, -9.0)])
def test_recurrence_prompt_and_step(C, blocks, lam, dtype):
    """Sequences that end at, before and after the borders of runs and tiles; decays from almost one to almost zero (the weight
    of the input is then far below, or at, one); the state is continued with a step."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K
    from trl_b200.ops import mixers as mx

    m, p = recurrent(C, blocks, 4, dtype, lam)
    lens, slots = [1, 16, 64, 65, 140, 15, 128], [3, 0, 5, 1, 7, 2, 4]
    T, r = sum(lens), gen(blocks)
    u, both = r(T, C).to(dtype).double(), r(T, 2 * C).to(dtype).double()
    ctx = SeqCtx.from_lengths(lens, "cuda")
    nu, ny = r(20, C).to(dtype).double(), r(20, C)
    live = torch.full((20,), -1)
    live[slots] = torch.tensor(lens)
    for tc in (False, True) if dtype == torch.bfloat16 and K.rglru_tc_ok(m) else (False,):
        state = torch.full((20, C), 7.0, device="cuda")
        got = mx.rglru_prompt_scan(dev(u, dtype), dev(both, dtype)[:, :C], m, ctx, i32(slots), state, tensor_cores=tc).double().cpu()
        after = state.double().cpu()
        sums, out = dev(torch.cat([ny, ny], 1)), torch.full((20, C), 3.0, dtype=dtype, device="cuda")
        if tc:
            K.rglru_step_tc(dev(nu, dtype), sums[:, :C], m, live.int().cuda(), state, out)
        else:
            K.rglru_step(mx.block_gates(dev(nu, dtype), m.gates), dev(nu, dtype), sums[:, :C], m, live.int().cuda(), state, out)
        KC.check_status()
        assert not sums[:, :C].any() and torch.equal(sums[:, C:].double().cpu(), ny.float().double())
        assert torch.equal(state[8:], torch.full((12, C), 7.0, device="cuda")) and not out[8:].any()
        a, t = 0, (1e-5 if dtype == torch.float32 else 1e-2)
        for n, s in zip(lens, slots):
            S, o = want_recurrence(torch.cat([u[a:a + n], nu[s:s + 1]]), torch.cat([both[a:a + n, :C], ny[s:s + 1]]), p, blocks)
            assert (got[a:a + n] - o[:n]).abs().max() < t * o.abs().max(), (tc, n)
            assert (out[s].double().cpu() - o[n]).abs().max() < t * o.abs().max()
            # the state stays fp32 in bf16 models too
            assert (after[s] - S[n - 1]).abs().max() < 2e-5 * S.abs().max()
            assert (state[s].double().cpu() - S[n]).abs().max() < 2e-5 * S.abs().max()
            a += n


@pytest.mark.parametrize("tc", [True, False])
def test_recurrence_remembers_the_first_token(tc):
    """One input at the start and none after it, with slow decay: what is left at the end is its share."""
    from trl_b200.ops import mixers as mx

    m, p = recurrent(64, 1, 4, torch.bfloat16, lam=-7.0)
    u = torch.zeros(300, 64, dtype=f64)
    u[0] = 4.0
    y = torch.full((300, 64), 2.0, dtype=f64)
    got = mx.rglru_prompt_scan(dev(u, torch.bfloat16), dev(y, torch.bfloat16), m, SeqCtx.from_lengths([300], "cuda"), tensor_cores=tc).double().cpu()
    _, want = want_recurrence(u, y, p, 1)
    assert want[-1].abs().max() > 0.02 and (got[-1] - want[-1]).abs().max() < 1e-2 * want[-1].abs().max()


# ---- whole model --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 70), ("tiles", 150), ("ones", 70), ("odd", 1), ("tiles", 2)])
def test_whole_prompt(name, n, dtype):
    toks, want = wanted(name, n, 1)
    m, _ = model(name, dtype)
    with torch.no_grad():
        got = m(torch.tensor([toks], device="cuda")).logits[0]
    assert U.rel(got, want) < tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles", "ones"])
@pytest.mark.parametrize("cut", [1, 2, 17, 63])
def test_prompt_then_tokens(name, cut, dtype):
    """A prompt of ``cut`` tokens, the rest one by one: first tokens, convolution tails, page borders (16-token pages)."""
    n = 70
    toks, want = wanted(name, n, 1)
    f = feed(name, dtype, block=16, max_len=96)
    got = [f.step([("a", toks[:cut], list(range(cut)))])[0]]
    for t in range(cut, n):
        got.append(f.step([("a", toks[t:t + 1], [0])])[0])
    assert U.rel(torch.cat(got), want) < tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(dtype):
    """Decoding over several tiles of the attention kernels and 64-token pages."""
    toks, want = wanted("tiles", 150, 1)
    f = feed("tiles", dtype, max_len=256)
    got = [f.step([("a", toks[:5], list(range(5)))])[0]]
    got += [f.step([("a", [t], [0])])[0] for t in toks[5:]]
    assert U.rel(torch.cat(got), want) < tol("tiles", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", [[2] * 10, [3, 2, 15], [10, 10]])
def test_portions(portions, dtype):
    toks, want = wanted("odd", 70, 1)
    f, at, got = feed("odd", dtype, block=16), 0, []
    for n in portions:
        got.append(f.step([("a", toks[at:at + n], list(range(n)))])[0])
        at += n
    assert U.rel(torch.cat(got), want[:at]) < tol("odd", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_unequal_batch_and_reused_slots(name, dtype):
    """Three unequal requests decode together, end at different times, and their slots and pages (the pool holds no more than
    they need) serve other requests afterwards."""
    lens = {"a": (70, 40), "b": (3, 1), "c": (33, 30)}
    f = feed(name, dtype, slots=3, block=16, max_len=80, blocks=11)
    for rnd in range(2):
        seqs = {k: wanted(name, n, 1 + rnd + i) for i, (k, (n, _)) in enumerate(lens.items())}
        got = {k: [] for k in lens}
        order = list(lens) if rnd == 0 else list(lens)[::-1]
        ents = [(f"{k}{rnd}", seqs[k][0][:lens[k][1]], list(range(lens[k][1]))) for k in order]
        for k, o in zip(order, f.step(ents)):
            got[k].append(o)
        for step in range(30):
            ents, end = [], []
            for k in order:
                t = lens[k][1] + step
                if t < lens[k][0]:
                    ents.append((f"{k}{rnd}", [seqs[k][0][t]], [0]))
                    if t == lens[k][0] - 1:
                        end.append(f"{k}{rnd}")
            for (r, _, _), o in zip(ents, f.step(ents, end)):
                got[r[0]].append(o)
        assert f.live == 0 and f.e.sched.num_free_blocks == 11
        for k in lens:
            assert U.rel(torch.cat(got[k]), seqs[k][1]) < tol(name, dtype), (rnd, k)


@functools.lru_cache(maxsize=None)
def greedy(prompt):
    _, t = U.make(U.ODD)
    seq = list(prompt)
    for _ in range(9):
        seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("n", [1, 3])
def test_greedy_generation_through_the_engine(n, graph):
    """More requests than slots: the scheduler admits, shares prompt pages and states, retires and admits again."""
    from trl_b200.rollout.engine import make_engine

    m, _ = model("odd", torch.float32)
    eng = make_engine(m, max_num_seqs=4, max_model_len=64, block_size=8, poll_every=3, use_cuda_graph=graph)
    prompts = [U.tokens(k, 197, 20 + k) for k in (5, 16, 1, 23)]
    for _ in range(2):
        outs = eng.generate(prompts, SamplingParams(n=n, max_tokens=9, greedy=True))
        for i, p in enumerate(prompts):
            for o in outs[i * n:(i + 1) * n]:
                assert o.token_ids == greedy(tuple(p)) and o.finish_reason == "length"


def test_bf16_generation_follows_the_fed_tokens():
    """Log-probs of a sampled bf16 run are those of the same tokens fed as one prompt."""
    from trl_b200.rollout.engine import make_engine

    m, _ = model("tiles", torch.bfloat16)
    eng = make_engine(m, max_num_seqs=3, max_model_len=128)
    prompts = [U.tokens(k, 197, k) for k in (30, 7, 64, 2)]
    outs = eng.generate(prompts, SamplingParams(n=2, max_tokens=20, temperature=1.0, seed=5))
    for o in outs:
        f = feed("tiles", torch.bfloat16, slots=2, max_len=128)
        toks = o.prompt_ids + o.token_ids
        lg = f.step([("x", toks[:-1], list(range(len(o.prompt_ids) - 1, len(toks) - 1)))])[0]
        lp = torch.log_softmax(lg, -1).cpu().gather(1, torch.tensor(o.token_ids)[:, None])[:, 0]
        assert (lp - torch.tensor(o.logprobs)).abs().max() < 0.06 * float(lg.std())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_command(tmp_path, dtype):
    """bin/trace_run in a process of its own: unequal requests, requests that end, logits in the order asked for."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    m, _ = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path / "m"))
    (tmp_path / "out").mkdir()
    (a, wa), (b, wb) = wanted("odd", 70, 1), wanted("odd", 70, 2)
    steps = [{"step": 0, "entries": [{"id": "b", "tokens": b[:5], "want": [4, 0]}, {"id": "a", "tokens": a[:60], "want": [59]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[60]], "want": []}, {"id": "b", "tokens": [b[5]], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[61]], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[:9], "want": [8]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype,
                        "--out", str(tmp_path / "out"), "--max-tokens", "80"], input="\n".join(map(json.dumps, steps)) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    want = {0: torch.stack([wb[4], wb[0], wa[59]]), 2: wa[61:62], 3: wb[8:9]}
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "2.f32", "3.f32"]
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4").copy()).view(-1, 197)
        assert U.rel(got, w) < tol("odd", getattr(torch, dtype))
