"""Suposun on the GPU: every kernel of its mechanisms, the serving engine's caches and states, generation.

Models are compared with the plain restatement (suposun_reference.py) in float64; float32 models are held to rounding, bf16
models to bf16 rounding, and where that could hide a fault (a key at an edge, a sink, a kept token) the inputs are made so that
one score stands out."""
import functools
import math
import types

import pytest
import torch

import suposun_reference as ref
import suposun_util as U
from trl_b200.models import SeqCtx
from trl_b200.rollout.sampling import SamplingParams

pytestmark = pytest.mark.gpu

CFGS = {"odd": U.ODD, "tiles": U.TILES, "ones": U.ONES, "plain": U.PLAIN}
DTYPES = [torch.float32, torch.bfloat16]
f64, bf16 = torch.float64, torch.bfloat16


def tol(name, dtype):
    # eight channels: a norm over eight values can blow up the rounding of a small one
    return 3e-5 if dtype == torch.float32 else 0.2 if name == "ones" else 0.06


def dev(x, dtype=torch.float32):
    return x.to("cuda", dtype)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=f64)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


@functools.lru_cache(maxsize=None)
def model(name, dtype):
    """bf16 models choose the same experts for every token: a choice that hangs on rounding says nothing about a kernel."""
    return U.make(CFGS[name], dtype, "cuda", clear=dtype == bf16)


@functools.lru_cache(maxsize=None)
def wanted(name, n, seed, dtype):
    toks = U.tokens(n, CFGS[name]["vocab"], seed)
    _, t = U.make(CFGS[name], clear=dtype == bf16)
    return toks, U.logits(CFGS[name], t, toks)


def feed(name, dtype, slots=4, max_len=512, block=None, blocks=None):
    from trl_b200.rollout.engine import make_engine
    from trl_b200.rollout.feed import TokenFeed

    return TokenFeed(make_engine(model(name, dtype)[0], max_num_seqs=slots, max_model_len=max_len, block_size=block,
                                 num_blocks=blocks))


# ---- embedding, norms, feed-forward ---------------------------------------------------------------------------------
@pytest.mark.parametrize("H", [8, 33, 1024])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("spec", [dict(mul_prev=29, mul_cur=11, buckets=23), dict(mul_prev=1, mul_cur=1, buckets=1)])
def test_pair_embedding(H, dtype, spec):
    """Prompts leave their last tokens in their slots; steps take them from there and move on, idle slots stay."""
    from trl_b200.ops import cuda_mixers as K

    r = gen(H)
    emb, pairs = r(19, H).to(dtype).double(), r(spec["buckets"] + 1, H).to(dtype).double()
    seqs, slots = [[3, 18, 0], [7], [5, 5, 5, 5, 1]], [4, 0, 2]
    flat = torch.tensor(sum(seqs, []), device="cuda")
    ctx = SeqCtx.from_lengths([3, 1, 5], "cuda")
    last = torch.full((6,), 11, dtype=torch.int64, device="cuda")
    got = K.embed_pairs(flat, dev(emb, dtype), 2.5, dev(pairs, dtype), spec["mul_prev"], spec["mul_cur"], ctx.positions,
                        tok_slot=i32([4] * 3 + [0] + [2] * 5), prev=last)
    want = torch.cat([ref.embed(s, emb, 2.5, pairs, spec) for s in seqs])
    assert torch.allclose(got.double().cpu(), want, atol=1e-5)
    assert last.tolist() == [7, 11, 1, 11, 0, 11]
    pos, nxt = i32([1, -1, 5, -1, 3, -1]), torch.tensor([2, 9, 12, 9, 18, 9], device="cuda")
    got = K.embed_pairs(nxt, dev(emb, dtype), 2.5, dev(pairs, dtype), spec["mul_prev"], spec["mul_cur"], pos, prev=last, decode=True)
    for s, slot in zip(seqs, slots):
        assert torch.allclose(got[slot].double().cpu(), ref.embed(s + [int(nxt[slot])], emb, 2.5, pairs, spec)[-1], atol=1e-5)
    assert last.tolist() == [2, 11, 12, 11, 18, 11]


@pytest.mark.parametrize("H", [8, 33, 1024, 1540, 4096, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_about_zero_with_layer_scale(H, dtype):
    from trl_b200.ops import cuda_mixers as K

    r = gen(H)
    x, d, p, s, w = r(5, H) * 3, r(5, H) * 0.01, r(H), r(H), r(H)
    eps, t = 1e-4, (3e-6 if dtype == torch.float32 else 2e-2)
    for scale in (s, None):
        for norm in (w, None):
            want_s = x + ref.norm_about_zero(d, p, eps) * (1 if scale is None else scale)
            want = want_s if norm is None else ref.norm_about_zero(want_s, norm, eps) * 0.4
            xg, dg = dev(x), dev(d)
            got = K.rms_residual(xg, dg, dev(p), None if norm is None else dev(norm), eps, dtype, clear=True, shift=1.0, gain=0.4,
                                 post_scale=None if scale is None else dev(scale))
            assert torch.allclose(got.double().cpu(), want, atol=t, rtol=t)
            assert torch.allclose(xg.double().cpu(), want_s, atol=1e-5, rtol=1e-6) and not dg.any()


@pytest.mark.parametrize("n", [1, 50, 136])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu_unit(n, dtype):
    from trl_b200.ops import cuda_mixers as K

    z = (gen(n)(9, 2 * n) * 4).to(dtype).double()
    t = 2e-6 if dtype == torch.float32 else 1e-2
    assert torch.allclose(K.gelu_glu(dev(z, dtype)).double().cpu(), ref.gelu_tanh(z[:, :n]) * z[:, n:], atol=t, rtol=t)


@pytest.mark.parametrize("B", [1, 20, 64, 100])
@pytest.mark.parametrize("n,k", [(24, 40), (128, 64), (200, 136)])
def test_gelu_unit_in_the_decode_product(B, n, k):
    from trl_b200.ops import cuda as KC

    r = gen(B + n)
    x, w = r(B, k).bfloat16(), (r(2 * n, k) / k ** 0.5 * 2).bfloat16()
    z = x.double() @ w.double().T
    got = KC.decode_gemm(x.cuda(), w.cuda(), gelu_glu=True)
    assert got.shape == (B, n) and torch.allclose(got.double().cpu(), ref.gelu_tanh(z[:, :n]) * z[:, n:], atol=1e-2, rtol=1e-2)


# ---- experts --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 7, 128, 129, 700])
@pytest.mark.parametrize("E,top", [(1, 1), (5, 5), (40, 3), (64, 8), (1000, 2)])
@pytest.mark.parametrize("renorm", [False, True])
def test_router(T, E, top, renorm):
    """Choices, weights, counts and places; idle rows choose nothing; one block and several."""
    from trl_b200.ops import cuda_mixers as K

    r = gen(T + E)
    z, c = r(T, E).float().double(), r(E).float().double()
    pos = torch.randint(0, 9, (T,), generator=torch.Generator().manual_seed(T)) - int(T > 3)
    zg = dev(z)
    choice, rank, weight, counts = K.moe_route(zg, dev(c), top, positions=i32(pos.tolist()), renormalize=renorm, clear=True)
    assert not zg.any()
    h = r(T, 12).float()
    x, row, offsets = K.moe_gather(h.cuda(), choice, rank, counts)
    choice, weight, counts, row, offsets, x = (t.cpu() for t in (choice, weight, counts, row, offsets, x))
    seen = torch.zeros(E, dtype=torch.int32)
    for t in range(T):
        if pos[t] < 0:
            assert (choice[t] == -1).all() and (row[t] == -1).all()
            continue
        want = ref.route(z[t], torch.eye(E, dtype=f64), c, top)
        total = sum(s for _, s in want) if renorm else 1.0
        assert choice[t].tolist() == [e for e, _ in want]
        assert torch.allclose(weight[t].double(), torch.stack([s / total for _, s in want]), atol=1e-6)
        for e, at in zip(choice[t].tolist(), row[t].tolist()):
            seen[e] += 1
            assert offsets[e] <= at < offsets[e + 1] and torch.equal(x[at], h[t].float())
    assert torch.equal(seen, counts) and torch.equal(offsets, torch.cat([torch.zeros(1), counts.cumsum(0)]).int())
    used = row[row >= 0]
    assert used.unique().numel() == used.numel() == int(offsets[-1])


def test_router_ties_and_garbage():
    """Equal scores go to the lower expert; logits that are not numbers still give experts that exist."""
    from trl_b200.ops import cuda_mixers as K

    z = torch.zeros(3, 70)
    z[1, 65] = z[1, 3] = 1.0
    z[2] = float("nan")
    choice, _, _, counts = K.moe_route(z.cuda(), None, 2)
    assert choice[0].tolist() == [0, 1] and choice[1].tolist() == [3, 65]
    assert ((choice >= 0) & (choice < 70)).all() and int(counts.sum()) == 6


def expert_case(H, n, E, top, dtype, seed=0, limit=0.8):
    r = gen(seed + H + E)
    t = {"router": 2 * r(E, H) / H ** 0.5, "correction": 0.5 * r(E), "gate_up": 2 * r(E, 2 * n, H) / H ** 0.5, "down": r(E, H, n) / n ** 0.5}
    t = {k: v.to(dtype if k != "correction" else torch.float32).double() for k, v in t.items()}
    m = types.SimpleNamespace(n=E, top=top, ff=n, glu=(limit, 1.702, 1.0), routing={},
                              **{k: dev(v, dtype if k != "correction" else torch.float32) for k, v in t.items()})
    w = dict(router=t["router"], correction=t["correction"])
    for e in range(E):
        w.update({f"e{e}.gate": t["gate_up"][e, :n], f"e{e}.up": t["gate_up"][e, n:], f"e{e}.down": t["down"][e]})
    return m, w, dict(router=dict(experts=E, top=top), expert=dict(ff=n, limit=limit))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,n,E,top", [(76, 17, 7, 3), (160, 136, 12, 4), (64, 8, 1, 1), (72, 200, 3, 3), (33, 5, 20, 1)])
@pytest.mark.parametrize("T", [1, 9, 150])
def test_experts(T, H, n, E, top, dtype):
    """Widths below, at and above the tiles of the grouped product, and those it does not take; the choices are made to be clear."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import mixers as mx

    m, w, c = expert_case(H, n, E, top, dtype)
    h = gen(T)(T, H).to(dtype).double()
    want = ref.expert_mlp(h, w, c)
    scores = torch.sigmoid(h @ w["router"].T) + w["correction"]
    order = scores.sort(-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == E else order[:, top - 1] - order[:, top] > 1e-4
    got = mx.experts(m, dev(h, dtype))
    assert got.dtype == torch.float32
    pos = torch.arange(T) % 5 - 1  # every fifth row idle
    z = mx.linear_f32(dev(h, dtype), m.router)
    out = torch.full((T, H), 7.0, device="cuda")
    mx.experts(m, dev(h, dtype), positions=i32(pos.tolist()), logits=z, out=out)
    KC.check_status()
    t = (1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())
    assert ((got.double().cpu() - want)[clear].abs() < t).all()
    live = pos >= 0
    assert ((out.double().cpu() - want)[clear & live].abs() < t).all() and not out[(~live).cuda()].any() and not z.any()


def test_expert_of_all_tokens_and_of_none():
    """Corrections that send every token to one expert of many: the others have no rows."""
    from trl_b200.ops import mixers as mx

    m, w, c = expert_case(64, 40, 30, 1, bf16)
    m.correction[17], w["correction"][17] = 9.0, 9.0
    h = gen(3)(300, 64).bfloat16().double()
    got = mx.experts(m, dev(h, bf16)).double().cpu()
    want = torch.sigmoid(h @ w["router"][17]) [:, None] * ref.expert(h, w["e17.gate"], w["e17.up"], w["e17.down"], 0.8)
    assert (got - want).abs().max() < 2e-2 * want.abs().max()


# ---- attention ------------------------------------------------------------------------------------------------------
def mixer(H, G, d, e, **kw):
    return types.SimpleNamespace(**{**dict(heads=H, kv_heads=G, dim=d, vdim=e, scale=0.3, cap=None, kv_from=None, eps=1e-4), **kw})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,rot,halves,scaling", [(6, 3, 20, 8, False, None), (4, 1, 128, 32, False, U.yarn()), (3, 3, 9, 4, True, None),
                                                      (5, 5, 48, 48, True, None), (20, 4, 64, 24, True, U.yarn()), (2, 1, 14, 14, False, None), (8, 2, 16, 0, False, None),
                                                      (32, 8, 128, 64, True, None), (72, 8, 128, 40, False, None)])
@pytest.mark.parametrize("whole", [False, True])
@pytest.mark.parametrize("kind", ["values", "keys", "borrowed"])
def test_attention_preparation(H, G, d, rot, halves, scaling, whole, kind, dtype):
    """Prompt rows (in place, or keys apart) and decode sums (cleared): norms per head or over all heads with weights, both
    rotations, keys as values, gates per head, rows of the pages."""
    from trl_b200.ops import cuda_mixers as K
    from trl_b200.ops.mixers import RotarySpec

    r, rows, bs, e = gen(H + d), 5, 4, d if kind == "keys" else 12
    own, values, gated = kind != "borrowed", kind == "values", kind == "keys"
    m = mixer(H, G, d, e, kv_from=None if own else 0, o=torch.empty(0, dtype=dtype))
    kv = G if own else 0
    parts = [H * d, kv * d, kv * e if values else 0, H if gated else 0]
    y = (r(rows, sum(parts)) * 2).to(dtype).double()
    qw, kw = 1 + 0.3 * r(H * d if whole else d), 1 + 0.3 * r(G * d if whole else d)
    pos = [0, 3, 4, -1, 9]
    block = torch.tensor([[5, 1, 3], [2, 4, 6], [7, 8, 9], [10, 11, 12], [13, 14, 15]], dtype=torch.int32)
    spec = dict(dims=rot, base=50.0, scaling=scaling)

    def prepared(x, n, w):
        x = (ref.unit_rms(x, 1e-4) * w).view(rows, n, d) if whole else ref.unit_rms(x.view(rows, n, d), 1e-4) * w
        return torch.stack([ref.rotate(x[i], p, spec, halves) if rot and p >= 0 else x[i] for i, p in enumerate(pos)])

    q, k, v, g = y.split(parts, 1)
    wq, t = prepared(q, H, qw), (5e-6 if dtype == torch.float32 else 2e-2)
    if own:
        wk, wv = prepared(k, G, kw), (v if values else k).reshape(rows, G, e)
    how = dict(q_norm=dev(qw), k_norm=dev(kw) if own else None, whole_norm=whole, rot=rot, halves=halves, values=values, gates="head" if gated else None,
               table=RotarySpec(rot, 50.0, scaling).table(12, "cuda") if rot else None)
    for sums in (False, True):
        kc, vc = torch.full((16, bs, G, d), 9.0, dtype=dtype, device="cuda"), torch.full((16, bs, G, e), 9.0, dtype=dtype, device="cuda")
        where = dict(k_cache=kc, v_cache=vc, block_table=block.cuda(), block_size=bs) if own else {}
        src = dev(y, torch.float32 if sums else dtype)
        gate = torch.full((rows, H), 7.0, device="cuda") if gated else None
        keys = torch.full((rows, kv * d), 7.0, dtype=dtype, device="cuda") if own and not values and not sums else None
        qb = torch.zeros(rows, H, d, dtype=dtype, device="cuda") if sums else None
        K.attn_prep(src, m, i32(pos), None, q=qb, k=keys, head_gate=gate, **how, **where)
        if gated:
            assert torch.allclose(gate.double().cpu(), torch.sigmoid(g), atol=1e-6)
        if sums:
            assert not src.any()
            got = qb.double().cpu()
        else:
            got = src[:, :H * d].double().cpu().view(rows, H, d)
            if own:
                gk = (src[:, H * d:H * d + kv * d] if values else keys).double().cpu().view(rows, kv, d)
                assert torch.allclose(gk, wk, atol=3 * t, rtol=t)
                assert torch.equal(src[:, H * d + (kv * d if values else 0):].double().cpu(), torch.cat([v, g] if values else [k, v, g], 1))
        assert torch.allclose(got, wq, atol=3 * t, rtol=t)
        written = 0
        for i, p in enumerate(pos):
            if p >= 0 and own:
                at = int(block[i, p // bs]), p % bs
                assert torch.allclose(kc[at].double().cpu(), wk[i], atol=3 * t, rtol=t)
                assert torch.allclose(vc[at].double().cpu(), wv[i], atol=t, rtol=t)
                written += 1
        assert int((kc != 9.0).flatten(2).any(2).sum()) == written == int((vc != 9.0).flatten(2).any(2).sum())


SHAPES = [(6, 3, 20, 28), (4, 4, 72, 48), (8, 1, 128, 128), (20, 2, 72, 136), (2, 1, 13, 9), (3, 1, 256, 256)]
MASKS = [dict(size=1), dict(size=30, keep_first=2), dict(size=130, keep_first=1), dict(size=60, keep_first=40), dict(size=20, keep_first=150), dict(size=200, keep_first=129),
         dict(size=1000, keep_first=5)]


def attention_case(T, m, dtype, seed):
    r = gen(seed)
    return (*(t.to(dtype).double() for t in (r(T, m.heads, m.dim), r(T, m.kv_heads, m.dim), r(T, m.kv_heads, m.vdim))), torch.sigmoid(r(T, m.heads)).float().double())


def want_rows(q, k, v, m, mask, sink, rows):
    """Rows of one sequence's attention, vectorised over keys only."""
    per = m.heads // m.kv_heads
    out = []
    for t in rows:
        vis = ref.visible(t, mask)
        out.append(ref.attend_one(q[t], k[vis], v[vis], m.scale, m.cap, sink, per))
    return torch.stack(out)


def run_prompt(q, k, v, g, m, mask, sink, lens, dtype, tc=True):
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T = q.shape[0]
    y = dev(torch.cat([t.reshape(T, -1) for t in (q, k, v)], 1), dtype)
    out = K.mixer_attn(*y.split([q[0].numel(), k[0].numel(), v[0].numel()], 1), heads=m.heads, kv_heads=m.kv_heads, scale=m.scale, cap=m.cap,
                       window=mask.get("size"), keep=mask.get("keep_first", 0), sink=None if sink is None else dev(sink),
                       gate=None if g is None else dev(g), ctx=SeqCtx.from_lengths(lens, "cuda"), tensor_cores=tc)
    KC.check_status()
    return out.double().cpu().view(T, m.heads, m.vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mask", range(len(MASKS)))
def test_prompt_attention(shape, mask, dtype):
    """Windows below, around and above a tile with kept tokens below, around and above one; sink, cap and gates."""
    mask = MASKS[mask]
    for cap, scale in ((3.0, 0.3), (None, 0.1)):
        m, lens = mixer(*shape, cap=cap, scale=scale), [1, 290, 37]
        q, k, v, g = attention_case(sum(lens), m, dtype, shape[2])
        sink = gen(1)(m.heads).float().double() + 1
        rows = [[0], [0, 1, 2, 29, 30, 31, 32, 59, 60, 61, 127, 128, 129, 150, 151, 160, 200, 230, 255, 256, 288, 289], [0, 1, 20, 36]]
        got = [run_prompt(q, k, v, g, m, mask, sink, lens, dtype, tc) for tc in (True, False)]
        a = 0
        for n, rs in zip(lens, rows):
            want = want_rows(q[a:a + n], k[a:a + n], v[a:a + n], m, mask, sink, rs) * g[a:a + n][rs][..., None]
            for o in got:
                assert (o[a:a + n][rs] - want).abs().max() < (2e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), (cap, n)
            a += n


def edge_places(size, keep, t):
    """Keys just inside and outside the window and the kept tokens of a query at t."""
    return [j for j in {0, keep - 1, keep, keep + 1, t - size - 1, t - size, t - size + 1, t - 1, t} if 0 <= j <= t]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,t", [(10, 3, 40), (10, 3, 12), (10, 3, 13), (128, 1, 140), (128, 4, 300), (127, 33, 300), (64, 128, 260), (129, 127, 384), (100, 0, 255), (1, 2, 256)])
def test_prompt_attention_at_the_edges(size, keep, t, dtype):
    """One key outweighs all others: its value comes out alone if it is visible, and nothing of it if it is not."""
    T, m, mask = t + 3, mixer(4, 2, 64, 40, scale=1.0, cap=40.0), dict(size=size, keep_first=keep)
    sink = torch.full((4,), -2.0, dtype=f64)
    for j in edge_places(size, keep, t):
        q, k, v, _ = attention_case(T, m, dtype, j)
        q, k = (q * 0.1).to(dtype).double(), (k * 0.1).to(dtype).double()
        u = torch.nn.functional.normalize(gen(t)(64), dim=0) * 5
        q[t], k[j] = u.to(dtype).double(), u.to(dtype).double()
        inside = t - j < size or j < keep
        want = want_rows(q, k, v, m, mask, sink, [t])[0]
        assert ((want - v[j].repeat_interleave(2, 0)).abs().max() < 0.01) == inside  # what the case is about
        for tc in (True, False):
            got = run_prompt(q, k, v, None, m, mask, sink, [T], dtype, tc)[t]
            assert (got - want).abs().max() < 0.03, (j, tc)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_attention_sinks(dtype):
    """Sinks far above, near and far below the scores; a cap must not touch them."""
    m, T = mixer(3, 1, 16, 16, scale=0.5, cap=2.0), 140
    q, k, v, _ = attention_case(T, m, dtype, 5)
    sink = torch.tensor([25.0, 1.0, -30.0], dtype=f64)
    for tc in (True, False):
        got = run_prompt(q, k, v, None, m, dict(size=50, keep_first=2), sink, [T], dtype, tc)
        want = want_rows(q, k, v, m, dict(size=50, keep_first=2), sink, [0, 30, 139])
        assert want[:, 0].abs().max() < 1e-7 and want[:, 2].abs().max() > 0.3
        assert (got[[0, 30, 139]] - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2)


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


def run_decode(q, ks, vs, lens, m, mask, sink, g, bs, dtype, seed=3):
    """Outputs of every kernel that takes the case: CUDA cores, tensor cores with one and several splits."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    B = len(lens)
    (kc, table), (vc, _) = paged(ks, bs, seed), paged(vs, bs, seed)
    args = (dev(q, dtype), dev(kc, dtype), dev(vc, dtype), m, i32(lens), table.cuda(), bs)
    kw = dict(window=mask.get("size"), keep=mask.get("keep_first", 0), sink=None if sink is None else dev(sink), head_gate=None if g is None else dev(g))
    outs = []
    for splits in ((0, 1, 3) if dtype == bf16 and K.grouped_decode_tc_ok(m, bs) else (0,)):
        out = torch.full((B, m.heads * m.vdim), 7.0, dtype=dtype, device="cuda")
        if splits:
            part = torch.full((B, m.heads * splits * m.vdim), 5.0, device="cuda"), torch.full((B, m.heads * splits * 2), 5.0, device="cuda")
            K.grouped_decode_tc(*args, out, None, splits, *part, **kw)
        else:
            K.grouped_decode(*args, out, **kw)
        outs.append(out.double().cpu().view(B, m.heads, m.vdim))
    KC.check_status()
    return outs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape,bs,cap,scale", [((6, 3, 20, 28), 16, 4.0, 0.3), ((8, 2, 128, 128), 64, None, 0.09), ((20, 2, 72, 136), 32, 2.0, 0.5),
                                                ((4, 4, 48, 48), 128, 30.0, 0.05), ((9, 1, 8, 256), 8, 5.0, 0.4), ((3, 1, 9, 5), 16, 1.0, 0.5)])
@pytest.mark.parametrize("mask", range(len(MASKS)))
def test_decode_attention(shape, bs, cap, scale, mask, dtype):
    """Ragged slots (idle ones included) whose windows start anywhere in a page and a tile; kept tokens; sinks and gates."""
    mask = MASKS[mask]
    m, r = mixer(*shape, cap=cap, scale=scale), gen(sum(shape))
    lens = [0, 300, -1, 127, 128, 29, 255, 189]
    ks = [(r(max(1, n + 1), m.kv_heads, m.dim) * 2).to(dtype).double() for n in lens]
    vs = [r(max(1, n + 1), m.kv_heads, m.vdim).to(dtype).double() for n in lens]
    q, g, sink = (r(len(lens), m.heads, m.dim) * 2).to(dtype).double(), torch.sigmoid(r(len(lens), m.heads)).float().double(), r(m.heads).float().double() + 1
    outs = run_decode(q, ks, vs, lens, m, mask, sink, g, bs, dtype)
    assert len(outs) == 3 or dtype == torch.float32 or shape[2] % 8 or shape[3] % 8
    for b, n in enumerate(lens):
        if n >= 0:
            vis = ref.visible(n, mask)
            want = ref.attend_one(q[b], ks[b][vis], vs[b][vis], m.scale, m.cap, sink, m.heads // m.kv_heads) * g[b][:, None]
            for got in outs:
                assert (got[b] - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,t", [(10, 3, 40), (10, 3, 12), (10, 3, 13), (16, 16, 47), (16, 16, 48), (128, 1, 140), (128, 4, 300), (127, 33, 300), (64, 128, 260),
                                         (129, 127, 384), (100, 0, 255), (1, 2, 256), (None, 0, 257)])
def test_decode_attention_at_the_edges(size, keep, t, dtype):
    m, mask = mixer(4, 2, 64, 40, scale=1.0, cap=40.0), dict(size=size, keep_first=keep)
    sink = torch.full((4,), -2.0, dtype=f64)
    for j in edge_places(size or 99, keep, t):
        r = gen(j)
        k, v, q = r(t + 1, 2, 64) * 0.1, r(t + 1, 2, 40), r(2, 4, 64) * 0.1
        u = torch.nn.functional.normalize(r(64), dim=0) * 5
        q[1], k[j] = u, u
        q, k, v = (x.to(dtype).double() for x in (q, k, v))
        vis = ref.visible(t, mask)
        want = ref.attend_one(q[1], k[vis], v[vis], 1.0, 40.0, sink, 2)
        assert ((want - v[j].repeat_interleave(2, 0)).abs().max() < 0.01) == (j in vis)
        for got in run_decode(q, [k[:1], k], [v[:1], v], [-1, t], m, mask, sink, None, 16, dtype, seed=j):
            assert (got[1] - want).abs().max() < 0.03, j


def test_windowed_decode_reads_no_page_outside_its_sight():
    """Pages that hold nothing visible are not read: what is in them does not matter, numbers or not."""
    from trl_b200.ops import cuda_mixers as K

    m, r, bs, n, mask = mixer(4, 2, 64, 64, scale=0.2), gen(0), 16, 400, dict(size=70, keep_first=18)
    k, v, q = (r(*s).bfloat16().double() for s in ((n + 1, 2, 64), (n + 1, 2, 64), (1, 4, 64)))
    vis = ref.visible(n, mask)
    pages = {j // bs for j in vis}
    hidden = [j for j in range(n + 1) if j // bs not in pages]
    assert len(hidden) > 200
    want = ref.attend_one(q[0], k[vis], v[vis], 0.2, None, None, 2)
    k[hidden], v[hidden] = float("nan"), float("nan")
    for got in run_decode(q, [k], [v], [n], m, mask, None, None, bs, bf16):
        assert (got[0] - want).abs().max() < 1e-2
    assert K.grouped_decode_tc_ok(m, bs)


def test_many_windowed_tiles_finish():
    """Enough tiles that CTAs share SMs: no wait runs out and runs repeat bit by bit."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T, H = 3072, 16
    r = torch.Generator(device="cuda").manual_seed(0)
    for d, e in ((128, 128), (48, 48), (192, 128), (72, 136)):
        q, k, v = (torch.randn(T, H * n, device="cuda", generator=r).bfloat16() for n in (d, d, e))
        ctx = SeqCtx.from_lengths([1024, 1, 1000, 1047], "cuda")
        for kw in (dict(window=300, keep=4), dict(window=90, keep=140, cap=20.0), dict(window=128, keep=128)):
            outs = [K.mixer_attn(q, k, v, heads=H, kv_heads=H, scale=0.05, ctx=ctx, **kw) for _ in range(4)]
            KC.check_status()
            assert all(torch.equal(o, outs[0]) for o in outs) and torch.isfinite(outs[0]).all()


# ---- whole model ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 70), ("tiles", 290), ("ones", 70), ("plain", 40), ("odd", 1), ("tiles", 2)])
def test_whole_prompt(name, n, dtype):
    toks, want = wanted(name, n, 1, dtype)
    m, _ = model(name, dtype)
    with torch.no_grad():
        got = m(torch.tensor([toks], device="cuda")).logits[0]
    assert U.rel(got, want) < tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles", "ones", "plain"])
@pytest.mark.parametrize("cut", [1, 2, 9, 17, 35])
def test_prompt_then_tokens(name, cut, dtype):
    """A prompt of ``cut`` tokens, the rest one by one: first tokens, window edges, page borders (16-token pages)."""
    n = 40
    toks, want = wanted(name, n, 1, dtype)
    f = feed(name, dtype, block=16, max_len=96)
    got = [f.step([("a", toks[:cut], list(range(cut)))])[0]]
    for t in range(cut, n):
        got.append(f.step([("a", toks[t:t + 1], [0])])[0])
    assert U.rel(torch.cat(got), want) < tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(dtype):
    """Decoding over several tiles of the attention kernels and 64-token pages, every window passing over decoded tokens."""
    toks, want = wanted("tiles", 290, 1, dtype)
    f = feed("tiles", dtype, max_len=320)
    got = [f.step([("a", toks[:5], list(range(5)))])[0]]
    got += [f.step([("a", [t], [0])])[0] for t in toks[5:]]
    assert U.rel(torch.cat(got), want) < tol("tiles", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", [[2] * 10, [3, 2, 15], [10, 10]])
def test_portions(portions, dtype):
    toks, want = wanted("odd", 40, 1, dtype)
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
    lens = {"a": (40, 20), "b": (3, 1), "c": (33, 30)}
    f = feed(name, dtype, slots=3, block=16, max_len=80, blocks=8)
    for rnd in range(2):
        seqs = {k: wanted(name, n, 1 + rnd + i, dtype) for i, (k, (n, _)) in enumerate(lens.items())}
        got = {k: [] for k in lens}
        order = list(lens) if rnd == 0 else list(lens)[::-1]
        ents = [(f"{k}{rnd}", seqs[k][0][:lens[k][1]], list(range(lens[k][1]))) for k in order]
        for k, o in zip(order, f.step(ents)):
            got[k].append(o)
        for step in range(20):
            ents, end = [], []
            for k in order:
                t = lens[k][1] + step
                if t < lens[k][0]:
                    ents.append((f"{k}{rnd}", [seqs[k][0][t]], [0]))
                    if t == lens[k][0] - 1:
                        end.append(f"{k}{rnd}")
            for (r, _, _), o in zip(ents, f.step(ents, end)):
                got[r[0]].append(o)
        assert f.live == 0 and f.e.sched.num_free_blocks == 8
        for k in lens:
            assert U.rel(torch.cat(got[k]), seqs[k][1]) < tol(name, dtype), (rnd, k)


@pytest.mark.parametrize("dtype", DTYPES)
def test_logits_do_not_depend_on_the_company(dtype):
    """The same request alone, in a batch, and in another slot: equal up to rounding."""
    a, b, c = (U.tokens(n, 193, n) for n in (30, 11, 23))
    want = None
    for others in ([], [b], [c, b]):
        f = feed("odd", dtype, block=16, max_len=64)
        ents = [(f"o{i}", o[:-6], []) for i, o in enumerate(others)] + [("a", a[:-6], list(range(24)))]
        got = [f.step(ents)[-1]]
        for s in range(6):
            got.append(f.step([(r, [(a if r == "a" else others[int(r[1])])[-6 + s]], [0]) for r, _, _ in ents])[-1])
        got = torch.cat(got)
        want = got.double().cpu() if want is None else want
        assert U.rel(got, want) < tol("odd", dtype)


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
    """More requests than slots: the scheduler admits, shares prompt pages and last tokens, retires and admits again."""
    from trl_b200.rollout.engine import make_engine

    m, _ = model("odd", torch.float32)
    eng = make_engine(m, max_num_seqs=4, max_model_len=64, block_size=8, poll_every=3, use_cuda_graph=graph)
    prompts = [U.tokens(k, 193, 20 + k) for k in (5, 16, 1, 23)]
    for _ in range(2):
        outs = eng.generate(prompts, SamplingParams(n=n, max_tokens=9, greedy=True))
        for i, p in enumerate(prompts):
            for o in outs[i * n:(i + 1) * n]:
                assert o.token_ids == greedy(tuple(p)) and o.finish_reason == "length"


def test_bf16_generation_follows_the_fed_tokens():
    """Log-probs of a sampled bf16 run are those of the same tokens fed as one prompt."""
    from trl_b200.rollout.engine import make_engine

    m, _ = model("tiles", bf16)
    eng = make_engine(m, max_num_seqs=3, max_model_len=128)
    prompts = [U.tokens(k, 200, k) for k in (30, 7, 64, 2)]
    outs, off = eng.generate(prompts, SamplingParams(n=2, max_tokens=20, temperature=1.0, seed=5)), []
    for o in outs:
        f = feed("tiles", bf16, slots=2, max_len=128)
        toks = o.prompt_ids + o.token_ids
        lg = f.step([("x", toks[:-1], list(range(len(o.prompt_ids) - 1, len(toks) - 1)))])[0]
        lp = torch.log_softmax(lg, -1).cpu().gather(1, torch.tensor(o.token_ids)[:, None])[:, 0]
        off.append((lp - torch.tensor(o.logprobs)).abs() / float(lg.std()))
    assert float(torch.cat(off).max()) < 0.06


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_command(tmp_path, dtype):
    """bin/trace_run in a process of its own: unequal requests, requests that end, logits in the order asked for."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    m, _ = U.make(U.ODD, bf16, clear=True)  # the checkpoint is bf16 in both runs
    m.save_pretrained(str(tmp_path / "m"))
    (tmp_path / "out").mkdir()
    (a, wa), (b, wb) = wanted("odd", 70, 1, bf16), wanted("odd", 40, 2, bf16)
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
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4").copy()).view(-1, 193)
        assert U.rel(got, w) < tol("odd", getattr(torch, dtype))
