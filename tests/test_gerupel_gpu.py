"""Gerupel on the GPU: every kernel of its mechanisms, the serving engine's caches and states, generation.

Models are compared with the plain restatement (gerupel_reference.py) in float64; float32 models are held to rounding, bf16
models to bf16 rounding, and where that could hide a fault (a key or a block at an edge, the one in the denominator) the inputs are
made so that one score stands out."""
import functools
import types

import pytest
import torch

import gerupel_reference as ref
import gerupel_util as U
from trl_b200.models import SeqCtx
from trl_b200.rollout.sampling import SamplingParams

pytestmark = pytest.mark.gpu

CFGS = {"odd": U.ODD, "tiles": U.TILES, "ones": U.ONES, "plain": U.PLAIN}
DTYPES = [torch.float32, torch.bfloat16]
f64, bf16 = torch.float64, torch.bfloat16


def cfg_of(name, dtype):
    return U.every_expert(CFGS[name]) if dtype == bf16 else CFGS[name]


def tol(name, dtype):
    # eight channels: a norm over eight values can blow up the rounding of a small one
    return 5e-5 if dtype == torch.float32 else 0.2 if name == "ones" else 0.06


def dev(x, dtype=torch.float32):
    return x.to("cuda", dtype)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=f64)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


@functools.lru_cache(maxsize=None)
def model(name, dtype):
    return U.make(cfg_of(name, dtype), dtype, "cuda")


@functools.lru_cache(maxsize=None)
def wanted(name, n, seed, dtype):
    toks = U.tokens(n, CFGS[name]["vocab"], seed)
    c = cfg_of(name, dtype)
    return toks, U.logits(c, U.make(c)[1], toks)


def feed(name, dtype, slots=4, max_len=512, block=None, blocks=None):
    from trl_b200.rollout.engine import make_engine
    from trl_b200.rollout.feed import TokenFeed

    return TokenFeed(make_engine(model(name, dtype)[0], max_num_seqs=slots, max_model_len=max_len, block_size=block, num_blocks=blocks))


# ---- embedding, norms -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H", [8, 33, 1024, 5000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_norm(H, dtype):
    from trl_b200.ops import cuda_mixers as K

    emb, w = gen(H)(19, H).to(dtype).double(), gen(1)(H)
    ids, copy = [3, 0, 18, 3], torch.zeros(4, H, device="cuda")
    got = K.embed_normed(torch.tensor(ids, device="cuda"), dev(emb, dtype), 2.5, dev(w), 1e-2, copy=copy)
    want = ref.norm(emb[ids] * 2.5, w, 1e-2)
    assert torch.allclose(got.double().cpu(), want, atol=1e-5) and torch.equal(got, copy)
    got = K.embed_normed(torch.tensor(ids, device="cuda"), dev(emb, dtype), 1.0, dev(w), 1e-4, shift=1.0)
    assert torch.allclose(got.double().cpu(), ref.norm(emb[ids], 1 + w, 1e-4), atol=1e-5)


@pytest.mark.parametrize("H", [8, 33, 1024, 1540, 4096, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norms_around_the_stream(H, dtype):
    """Sums of two outputs, or of one and of experts' rows, times a constant; what a loop adds; one and two norms."""
    from trl_b200.ops import cuda_mixers as K
    from trl_b200.ops.mixers import ExpertRows

    r, T = gen(H), 5
    x, a, b, first, step, w, w2 = r(T, H) * 3, r(T, H), r(T, H), r(T, H), r(H), r(H), r(H)
    y, wt = r(9, H).to(dtype).double(), r(T, 2).float().double()
    row = torch.tensor([[8, 0], [-1, 3], [2, 2], [-1, -1], [5, 7]])
    rows = torch.stack([sum((wt[t, c] * y[row[t, c]] for c in range(2) if row[t, c] >= 0), torch.zeros(H, dtype=f64)) for t in range(T)])
    t = 3e-6 if dtype == torch.float32 else 2e-2
    deltas = [(None, 0), (a, a), ((a, b), a + b), ((a, ExpertRows(dev(y, dtype), i32(row.tolist()), dev(wt))), a + rows)]
    for delta, added in deltas:
        for loop in (False, True):
            xg, d1 = dev(x), dev(a)
            d = None if delta is None else d1 if delta is a else (d1, dev(b) if delta[1] is b else delta[1])
            want_s = x + 0.3 * added + (first + step if loop else 0)
            kw = dict(anchor=dev(first), bump=dev(step)) if loop else {}
            got = K.rms_residual(xg, d, None, dev(w), 1e-4, dtype, clear=True, mult=0.3, w2=dev(w2) if loop else None, **kw)
            for o, n in zip(got if loop else (got,), (w, w2)):
                assert torch.allclose(o.double().cpu(), ref.norm(want_s, n, 1e-4), atol=t, rtol=t)
            assert torch.allclose(xg.double().cpu(), want_s, atol=1e-5, rtol=1e-6) and (delta is None or not d1.any())


# ---- experts --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 7, 128, 129, 700])
@pytest.mark.parametrize("E,top", [(1, 1), (5, 5), (40, 3), (64, 8), (1000, 2)])
def test_router(T, E, top):
    """Choices, weights, counts and places; idle rows choose nothing; one block and several; scores far apart."""
    from trl_b200.ops import cuda_mixers as K

    z = (gen(T + E)(T, E) * 3).float().double()
    z[0, 0] = 300.0  # all other scores vanish
    pos = torch.randint(0, 9, (T,), generator=torch.Generator().manual_seed(T)) - int(T > 3)
    zg = dev(z)
    choice, rank, weight, counts = K.moe_route(zg, None, top, positions=i32(pos.tolist()), scores="softmax", renormalize=True, gain=1.7, clear=True)
    assert not zg.any()
    h = gen(1)(T, 12).float()
    x, row, offsets = K.moe_gather(h.cuda(), choice, rank, counts)
    choice, weight, counts, row, offsets, x = (t.cpu() for t in (choice, weight, counts, row, offsets, x))
    seen = torch.zeros(E, dtype=torch.int32)
    for t in range(T):
        if pos[t] < 0:
            assert (choice[t] == -1).all() and (row[t] == -1).all()
            continue
        want = ref.route(z[t], top, 1.7)
        assert t == 0 or choice[t].tolist() == [e for e, _ in want]
        assert choice[t, 0] == want[0][0] and torch.allclose(weight[t].double(), torch.stack([s for _, s in want]), atol=1e-6)
        for e, at in zip(choice[t].tolist(), row[t].tolist()):
            seen[e] += 1
            assert offsets[e] <= at < offsets[e + 1] and torch.equal(x[at], h[t].float())
    assert torch.equal(seen, counts) and torch.equal(offsets, torch.cat([torch.zeros(1), counts.cumsum(0)]).int())
    used = row[row >= 0]
    assert used.unique().numel() == used.numel() == int(offsets[-1])


def test_router_ties_and_garbage():
    """Equal scores go to the lower expert; logits that are not numbers still give experts that exist."""
    from trl_b200.ops import cuda_mixers as K

    z = torch.zeros(4, 70)
    z[1, 65] = z[1, 3] = 1.0
    z[2] = float("nan")
    z[3, 7] = float("nan")
    choice, _, weight, counts = K.moe_route(z.cuda(), None, 2, scores="softmax", renormalize=True)
    assert choice[0].tolist() == [0, 1] and choice[1].tolist() == [3, 65] and torch.allclose(weight[:2].cpu(), torch.full((2, 2), 0.5))
    assert ((choice >= 0) & (choice < 70)).all() and int(counts.sum()) == 8


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,n,E,top", [(76, 17, 7, 3), (160, 136, 12, 4), (64, 8, 1, 1), (72, 200, 3, 3), (33, 5, 20, 1)])
@pytest.mark.parametrize("T", [1, 9, 150])
def test_experts(T, H, n, E, top, dtype):
    """Widths below, at and above the tiles of the grouped product, and those it does not take; the choices are made to be clear."""
    from trl_b200.models.layered import SoftmaxExpertMlp
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import mixers as mx

    r = gen(H + E)
    spec = U.moe(n, E, top, 1.3)
    m = SoftmaxExpertMlp(types.SimpleNamespace(hidden_size=H), spec, dtype, "cuda").requires_grad_(False)
    w = {}
    for name, t in m.tensors("").items():
        w[name] = (2 * r(*t.shape) / t.shape[1] ** 0.5).to(dtype).double()
        t.copy_(w[name])
    h = gen(T)(T, H).to(dtype).double()
    want = ref.expert_mlp(h, w, spec)
    order = (h @ w["router"].T).sort(-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == E else order[:, top - 1] - order[:, top] > 1e-3
    got = m(dev(h, dtype))
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
    # not added up: the kernel that adds them to the stream does it
    rows = m(dev(h, dtype), summed=False)
    x = torch.zeros(T, H, device="cuda")
    mx.rms_residual(x, (torch.zeros(T, H, device="cuda"), rows), None, torch.ones(H, device="cuda"), 1e-4, dtype)
    assert torch.allclose(x, got, atol=t)


# ---- windowed attention over pooled blocks --------------------------------------------------------------------------
def mixer(H, G, d, e, **kw):
    return types.SimpleNamespace(**{**dict(heads=H, kv_heads=G, dim=d, vdim=e, scale=0.3, cap=None, kv_from=None, eps=1e-4), **kw})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,rot,scaling", [(6, 3, 20, 28, 8, None), (4, 1, 128, 72, 32, U.llama3()), (3, 3, 9, 5, 4, None), (5, 5, 48, 48, 48, U.llama3()),
                                                 (20, 4, 64, 8, 16, None), (8, 2, 16, 16, 0, None), (32, 8, 128, 128, 128, None), (2, 1, 40, 256, 24, None)])
def test_attention_preparation(H, G, d, e, rot, scaling, dtype):
    """Prompt rows in place and decode sums (cleared): no norms, a factor per query head, rotated halves, rows of the pages, and in
    decode the means of the blocks that a token completes."""
    from trl_b200.ops import cuda_mixers as K
    from trl_b200.ops.mixers import RotarySpec

    r, rows, bs, P = gen(H + d), 5, 4, 3
    m = mixer(H, G, d, e, o=torch.empty(0, dtype=dtype))
    parts = [H * d, G * d, G * e]
    y, temp = (r(rows, sum(parts)) * 2).to(dtype).double(), r(H)
    pos = [0, 2, 5, -1, 9]  # the second and the third complete a block
    block = torch.tensor([[5, 1, 3], [2, 4, 6], [7, 8, 9], [10, 11, 12], [13, 14, 15]], dtype=torch.int32)
    spec, t = dict(dims=rot, base=50.0, scaling=scaling), (5e-6 if dtype == torch.float32 else 2e-2)

    def turned(x):
        return torch.stack([ref.rotate(x[i], p, spec) if rot and p >= 0 else x[i] for i, p in enumerate(pos)])

    q, k, v = y.split(parts, 1)
    wq, wk, wv = turned(q.view(rows, H, d)) * temp[:, None], turned(k.view(rows, G, d)), v.view(rows, G, e)
    how = dict(unit=False, q_head=dev(temp), rot=rot, halves=True, gates=None, table=RotarySpec(rot, 50.0, scaling).table(12, "cuda") if rot else None)
    for sums in (False, True):
        kc, vc = ((r(16, bs, G, n)).to(dtype).double() for n in (d, e))
        kg, vg = dev(kc, dtype), dev(vc, dtype)
        pools = dict(pool=P, pool_k=torch.full((rows, 4, G, d), 9.0, dtype=dtype, device="cuda"), pool_v=torch.full((rows, 4, G, e), 9.0, dtype=dtype, device="cuda"))
        src = dev(y, torch.float32 if sums else dtype)
        qb = torch.zeros(rows, H, d, dtype=dtype, device="cuda") if sums else None
        K.attn_prep(src, m, i32(pos), None, q=qb, **how, k_cache=kg, v_cache=vg, block_table=block.cuda(), block_size=bs, **(pools if sums else {}))
        if sums:
            assert not src.any()
            got = qb.double().cpu()
        else:
            got = src[:, :H * d].double().cpu().view(rows, H, d)
            assert torch.allclose(src[:, H * d:H * d + G * d].double().cpu().view(rows, G, d), wk, atol=3 * t, rtol=t)
            assert torch.equal(src[:, H * d + G * d:].double().cpu(), v)
        assert torch.allclose(got, wq, atol=3 * t, rtol=t)
        for i, p in enumerate(pos):
            if p >= 0:
                at = int(block[i, p // bs]), p % bs
                assert torch.allclose(kg[at].double().cpu(), wk[i], atol=3 * t, rtol=t) and torch.allclose(vg[at].double().cpu(), wv[i], atol=t, rtol=t)
        if not sums:
            continue
        for i, b in ((1, 0), (2, 1)):
            for cache, mean in ((kg, pools["pool_k"]), (vg, pools["pool_v"])):
                want = torch.stack([cache[int(block[i, p // bs]), p % bs].double().cpu() for p in range(b * P, b * P + P)]).mean(0)
                assert torch.allclose(mean[i, b].double().cpu(), want, atol=t, rtol=t)
        for mean in (pools["pool_k"], pools["pool_v"]):
            assert int((mean != 9.0).flatten(2).any(2).sum()) == 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kn,vn", [(12, 20), (5, 9), (1024, 512)])
@pytest.mark.parametrize("P", [1, 3, 16])
def test_means_of_blocks(P, kn, vn, dtype):
    """Sequences shorter than a block, of whole blocks and with a rest; strided rows; the slots' rows; rows of no block are zeros."""
    from trl_b200.ops import cuda_mixers as K

    lens, slots = [7, 2, 48, 1, 35], [3, 0, 4, 1, 5]
    T, ctx = sum(lens), SeqCtx.from_lengths(lens, "cuda")
    y = gen(P)(T, kn + vn + 3).to(dtype).double()
    yg = dev(y, dtype)
    G = 1
    pool_k, pool_v = (torch.full((6, 40, G, n), 9.0, dtype=dtype, device="cuda") for n in (kn, vn))
    pk, pv = K.pool_blocks(yg[:, :kn], yg[:, kn:kn + vn], ctx.cu_seqlens, P, seq_slot=i32(slots), pool_k=pool_k, pool_v=pool_v)
    assert pk.shape == (T // P + 1, kn) and pv.shape == (T // P + 1, vn)
    used, a, t = torch.zeros(T // P + 1, dtype=torch.bool), 0, (1e-6 if dtype == torch.float32 else 1e-2)
    for n, slot in zip(lens, slots):
        for b in range(n // P):
            want = y[a + b * P:a + b * P + P].mean(0)
            assert not used[a // P + b]
            used[a // P + b] = True
            assert torch.allclose(pk[a // P + b].double().cpu(), want[:kn], atol=t, rtol=t) and torch.allclose(pv[a // P + b].double().cpu(), want[kn:kn + vn], atol=t, rtol=t)
            if b < 40:
                assert torch.equal(pool_k[slot, b, 0], pk[a // P + b]) and torch.equal(pool_v[slot, b, 0], pv[a // P + b])
        assert (pool_k[slot, n // P:] == 9.0).all()
        a += n
    assert not pk[(~used).cuda()].any() and not pv[(~used).cuda()].any() and (pool_k[2] == 9.0).all()


SHAPES = [(6, 3, 20, 28), (4, 4, 72, 48), (8, 1, 128, 128), (20, 2, 72, 136), (2, 1, 13, 9), (3, 1, 256, 256)]
MASKS = [dict(size=1, pool=1), dict(size=30, pool=2), dict(size=130, pool=7), dict(size=60, pool=60), dict(size=20, pool=100), dict(size=1000, pool=5), dict(size=33, pool=1)]


def attention_case(T, m, dtype, seed):
    r = gen(seed)
    return tuple(t.to(dtype).double() for t in (r(T, m.heads, m.dim), r(T, m.kv_heads, m.dim), r(T, m.kv_heads, m.vdim)))


def run_prompt(q, k, v, m, mask, lens, dtype, tc=True, scale=1.0):
    """Output rows stand between others that must stay as they are."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T, n = q.shape[0], m.heads * m.vdim
    y = dev(torch.cat([t.reshape(T, -1) for t in (q, k, v)], 1), dtype)
    qg, kg, vg = y.split([q[0].numel(), k[0].numel(), v[0].numel()], 1)
    ctx = SeqCtx.from_lengths(lens, "cuda")
    out = torch.full((T, n + 24), 7.0, dtype=dtype, device="cuda")
    K.mixer_attn(qg, kg, vg, heads=m.heads, kv_heads=m.kv_heads, scale=m.scale, window=mask["size"], sink=torch.zeros(m.heads, device="cuda"), ctx=ctx, tensor_cores=tc,
                 pool=mask["pool"], blocks=K.pool_blocks(kg, vg, ctx.cu_seqlens, mask["pool"]), out=out[:, 8:8 + n], out_scale=scale)
    KC.check_status()
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + n:] == 7.0).all()
    return out[:, 8:8 + n].double().cpu().view(T, m.heads, m.vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mask", range(len(MASKS)))
def test_prompt_attention(shape, mask, dtype):
    """Windows below, around and above a tile, blocks of one and of many tokens, more blocks than a tile holds."""
    mask = MASKS[mask]
    m, lens = mixer(*shape, scale=0.1), [1, 290, 37]
    q, k, v = attention_case(sum(lens), m, dtype, shape[2])
    rows = [[0], [0, 1, 2, 29, 30, 31, 32, 59, 60, 61, 119, 120, 121, 127, 128, 129, 150, 160, 162, 163, 164, 200, 255, 256, 288, 289], [0, 1, 20, 36]]
    got = [run_prompt(q, k, v, m, mask, lens, dtype, tc, -0.7) for tc in (True, False)]
    a, one = 0, torch.ones(m.heads, dtype=f64)
    for n, rs in zip(lens, rows):
        for t in rs:
            want = -0.7 * ref.attend_one(q[a + t], k[a:a + n], v[a:a + n], m.scale, one, mask, t)
            for o in got:
                assert (o[a + t] - want).abs().max() < (2e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), (n, t)
        a += n


EDGES = [(10, 3, 40), (10, 3, 12), (10, 3, 13), (128, 1, 140), (128, 4, 300), (127, 33, 300), (64, 128, 260), (129, 127, 384), (100, 5, 255), (1, 2, 256), (16, 16, 47),
         (16, 16, 48), (20, 1, 290)]


def edge_places(size, P, t):
    """Keys just inside and outside the window of a query at t, in the last block it sees, in the next one, and far away."""
    last = max(0, t - size + 1) // P  # blocks seen
    return [j for j in {0, last * P - P, last * P - 1, last * P, last * P + P - 1, t - size - 1, t - size, t - size + 1, t - 1, t} if 0 <= j <= t]


def edge_case(size, P, t, j, dtype):
    """All keys of token j's block (or, inside the window, its own) outweigh the others."""
    m, mask = mixer(4, 2, 64, 40, scale=1.0), dict(size=size, pool=P)
    q, k, v = attention_case(t + 3, m, dtype, j)
    q, k = (q * 0.1).to(dtype).double(), (k * 0.1).to(dtype).double()
    u = (torch.nn.functional.normalize(gen(t)(64), dim=0) * 5).to(dtype).double()
    q[t] = u
    inside = t - j < size
    span = [j] if inside else [i for i in range(j // P * P, j // P * P + P) if i <= t - size]
    k[span] = u
    want = ref.attend_one(q[t], k[:t + 1], v[:t + 1], 1.0, torch.ones(4, dtype=f64), mask, t)
    alone = v[span].mean(0).repeat_interleave(2, 0)
    assert ((want - alone).abs().max() < 0.01) == (inside or j // P in ref.sight(t, mask)[1])  # what the case is about
    return m, mask, q, k, v, want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,P,t", EDGES)
def test_prompt_attention_at_the_edges(size, P, t, dtype):
    """One key, or one block, outweighs all others: its value comes out alone if it is visible, and nothing of it if it is not."""
    for j in edge_places(size, P, t):
        m, mask, q, k, v, want = edge_case(size, P, t, j, dtype)
        for tc in (True, False):
            got = run_prompt(q, k, v, m, mask, [t + 3], dtype, tc)[t]
            assert (got - want).abs().max() < 0.03, (j, tc)


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


def run_decode(q, ks, vs, lens, m, mask, bs, dtype, seed=3, scale=1.0):
    """Outputs of every kernel that takes the case: CUDA cores, tensor cores with one and several splits.  Rows of means that no
    complete block has filled hold a constant."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    B, P, n = len(lens), mask["pool"], m.heads * m.vdim
    (kc, table), (vc, _) = paged(ks, bs, seed), paged(vs, bs, seed)
    rows = max(lens) // P + 2
    pools = {}
    for name, xs in (("pool_k", ks), ("pool_v", vs)):
        pool = torch.full((B, rows) + tuple(xs[0].shape[1:]), 3.0, dtype=f64)
        for i, x in enumerate(xs):
            for b in range((lens[i] + 1) // P):
                pool[i, b] = x[b * P:b * P + P].mean(0)
        pools[name] = dev(pool, dtype)
    args = (dev(q, dtype), dev(kc, dtype), dev(vc, dtype), m, i32(lens), table.cuda(), bs)
    kw = dict(window=mask["size"], sink=torch.zeros(m.heads, device="cuda"), pool=P, out_scale=scale, **pools)
    outs = []
    for splits in ((0, 1, 3) if dtype == bf16 and K.grouped_decode_tc_ok(m, bs) else (0,)):
        out = torch.full((B, n + 24), 7.0, dtype=dtype, device="cuda")
        if splits:
            part = torch.full((B, n * splits), 5.0, device="cuda"), torch.full((B, m.heads * splits * 2), 5.0, device="cuda")
            K.grouped_decode_tc(*args, out[:, 8:8 + n], None, splits, *part, **kw)
        else:
            K.grouped_decode(*args, out[:, 8:8 + n], **kw)
        assert (out[:, :8] == 7.0).all() and (out[:, 8 + n:] == 7.0).all()
        outs.append(out[:, 8:8 + n].double().cpu().view(B, m.heads, m.vdim))
    KC.check_status()
    return outs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape,bs", [((6, 3, 20, 28), 16), ((8, 2, 128, 128), 64), ((20, 2, 72, 136), 32), ((4, 4, 48, 48), 128), ((9, 1, 8, 256), 8), ((3, 1, 9, 5), 16)])
@pytest.mark.parametrize("mask", range(len(MASKS)))
def test_decode_attention(shape, bs, mask, dtype):
    """Ragged slots (idle ones included) whose windows start anywhere in a page, a tile and a block."""
    mask = MASKS[mask]
    m, r = mixer(*shape, scale=0.1), gen(sum(shape))
    lens = [0, 300, -1, 127, 128, 29, 255, 189, 60]
    ks = [(r(max(1, n + 1), m.kv_heads, m.dim) * 2).to(dtype).double() for n in lens]
    vs = [r(max(1, n + 1), m.kv_heads, m.vdim).to(dtype).double() for n in lens]
    q = (r(len(lens), m.heads, m.dim) * 2).to(dtype).double()
    outs = run_decode(q, ks, vs, lens, m, mask, bs, dtype, scale=-0.7)
    assert len(outs) == 3 or dtype == torch.float32 or shape[2] % 8 or shape[3] % 8
    for b, n in enumerate(lens):
        if n >= 0:
            want = -0.7 * ref.attend_one(q[b], ks[b], vs[b], m.scale, torch.ones(m.heads, dtype=f64), mask, n)
            for got in outs:
                assert (got[b] - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,P,t", EDGES)
def test_decode_attention_at_the_edges(size, P, t, dtype):
    for j in edge_places(size, P, t):
        m, mask, q, k, v, want = edge_case(size, P, t, j, dtype)
        k, v = k[:t + 1], v[:t + 1]
        for got in run_decode(torch.stack([q[0], q[t]]), [k[:1], k], [v[:1], v], [-1, t], m, mask, 16, dtype, seed=j):
            assert (got[1] - want).abs().max() < 0.03, j


def test_one_in_the_denominator():
    """Scores far above, at and far below zero."""
    m, mask = mixer(3, 1, 16, 16, scale=1.0), dict(size=50, pool=4)
    q, k, v = attention_case(140, m, bf16, 5)
    k[:] = 0.25  # score of head h: 4 q[h]
    q[:, 0], q[:, 1], q[:, 2] = 8.0, 0.0, -8.0
    want = torch.stack([ref.attend_one(q[t], k, v, 1.0, torch.ones(3, dtype=f64), mask, t) for t in (0, 30, 139)])
    assert want[:, 2].abs().max() < 1e-9 and (want[0, 1] - v[0, 0] / 2).abs().max() < 1e-12
    for tc in (True, False):
        assert (run_prompt(q, k, v, m, mask, [140], bf16, tc)[[0, 30, 139]] - want).abs().max() < 1e-2
    for t, w in ((0, want[0]), (30, want[1]), (139, want[2])):
        for got in run_decode(q[t:t + 1], [k[:t + 1]], [v[:t + 1]], [t], m, mask, 16, bf16):
            assert (got[0] - w).abs().max() < 1e-2


def test_many_tiles_finish():
    """Enough tiles that CTAs share SMs: no wait runs out and runs repeat bit by bit."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import cuda_mixers as K

    T, H = 3072, 16
    r = torch.Generator(device="cuda").manual_seed(0)
    ctx = SeqCtx.from_lengths([1024, 1, 1000, 1047], "cuda")
    for d, e in ((128, 128), (48, 48), (192, 128), (72, 136)):
        q, k, v = (torch.randn(T, H * n, device="cuda", generator=r).bfloat16() for n in (d, d, e))
        for window, P in ((300, 4), (90, 1), (128, 128)):
            blocks = K.pool_blocks(k, v, ctx.cu_seqlens, P)
            outs = [K.mixer_attn(q, k, v, heads=H, kv_heads=H, scale=0.05, ctx=ctx, window=window, pool=P, blocks=blocks) for _ in range(4)]
            KC.check_status()
            assert all(torch.equal(o, outs[0]) for o in outs) and torch.isfinite(outs[0]).all()


# ---- linear attention with forget gates -----------------------------------------------------------------------------
def recurrent_case(T, H, d, e, dtype, seed, kind="mixed"):
    """(mixer, rows [q | v], gate logits, what the recurrence reads).  Gates from never to always forgetting, or all of one kind."""
    r = gen(seed + d + e)
    y = r(T, H * (d + e)).to(dtype).double()
    z, b = (3 * r(T, H * d)).float().double(), (3 * r(H * d)).float().double()
    low = (torch.sigmoid(2 * r(H * d)) * (r(H * d) > 0)).float().double()
    if kind == "slow":
        z, b, low = z * 0.1 + 9, b * 0, low * 0
    elif kind == "fast":  # nothing survives a token
        z, b, low = z - 30, b * 0, low * 0
    elif kind == "bounds":  # gates at their bounds in turn: everything is replaced, or nothing changes
        z, b, low = torch.where(r(T, H * d) > 0, 200.0, -200.0).double(), b * 0, low * 0
    m = types.SimpleNamespace(heads=H, dim=d, vdim=e, out_width=H * e, f_bias=dev(b), lower=dev(low), norm=dev(1 + 0.3 * r(e)), eps=1e-4)
    q, v = y.split([H * d, H * e], 1)
    return m, y, z, (ref.silu(q).view(T, H, d), ref.forget(z + b, low).view(T, H, d), v.view(T, H, e))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,e", [(1, 1, 1), (3, 18, 10), (2, 40, 72), (4, 64, 128), (2, 128, 128), (1, 128, 136), (2, 8, 24), (1, 200, 40), (1, 300, 16)])
@pytest.mark.parametrize("kind", ["mixed", "slow", "fast", "bounds"])
def test_prompt_recurrence(H, d, e, kind, dtype):
    """Sequences below, at and above a chunk; final states in their slots; on the tensor cores and token by token."""
    from trl_b200.ops import cuda as KC
    from trl_b200.ops import mixers as mx

    lens, slots = [1, 128, 290, 7, 129, 33], [2, 5, 0, 4, 1, 6]
    T, ctx = sum(lens), SeqCtx.from_lengths(lens, "cuda")
    m, y, z, (q, f, v) = recurrent_case(T, H, d, e, dtype, 1, kind)
    for tc in (True, False):
        state = torch.full((8, H, d, e), 7.0, device="cuda")
        # rows behind other columns, as a half of a larger projection
        yg, zg = torch.cat([torch.ones(T, 8), y], 1).to("cuda", dtype)[:, 8:], torch.cat([torch.ones(T, 4), z], 1).float().cuda()[:, 4:]
        got = mx.hgrn2_prompt_scan(m, yg, zg, ctx, dict(seq_slot=i32(slots), state=state), tensor_cores=tc)
        KC.check_status()
        a = 0
        for n, slot in zip(lens, slots):
            o, S = ref.recurrence(q[a:a + n], f[a:a + n], v[a:a + n])
            t = 3e-5
            assert (got[a:a + n].double().cpu() - o).abs().max() < t * max(1.0, float(o.abs().max())), (tc, n)
            assert (state[slot].double().cpu() - S).abs().max() < t * max(1.0, float(S.abs().max())), (tc, n)
            a += n
        assert (state[[3, 7]] == 7.0).all()
    # with the norm behind it, into rows between others
    out, a = torch.full((T, H * e + 24), 7.0, dtype=dtype, device="cuda"), 0
    mx.hgrn2_rows(m, yg, zg, ctx, {}, out=out[:, 8:8 + H * e], scale=-0.3)
    KC.check_status()
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + H * e:] == 7.0).all()
    for n in lens:
        o, _ = ref.recurrence(q[a:a + n], f[a:a + n], v[a:a + n])
        want = -0.3 * ref.norm(o, m.norm.double().cpu(), 1e-4).reshape(n, -1)
        off = (out[a:a + n, 8:8 + H * e].double().cpu() - want).abs()
        assert (off < (2e-4 if dtype == torch.float32 else 1e-2) * (1 + want.abs())).all()
        a += n


def test_recurrence_remembers_one_token():
    """A token that writes much into channels which forget nothing is read back hundreds of tokens later."""
    from trl_b200.ops import mixers as mx

    T, H, d, e = 700, 2, 64, 64
    m, y, z, _ = recurrent_case(T, H, d, e, bf16, 3, "slow")
    z[:], y[:, :H * d] = 40.0, 0.01  # f is one in fp32: nothing is forgotten, nothing written
    z[37, 5] = -40.0
    y[699, 5] = 6.0
    y = y.bfloat16().double()
    ctx = SeqCtx.from_lengths([T], "cuda")
    for tc in (True, False):
        got = mx.hgrn2_prompt_scan(m, dev(y, bf16), dev(z), ctx, {}, tensor_cores=tc).double().cpu()
        want = ref.silu(y[699, 5]) * y[37, H * d:H * d + e]
        assert (got[699, 0] - want).abs().max() < 1e-4 and got[:37].abs().max() < 1e-6 and got[:, 1].abs().max() < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,e", [(1, 1, 1), (3, 18, 10), (2, 40, 72), (4, 64, 128), (2, 128, 128), (1, 5, 300)])
def test_recurrent_step(H, d, e, dtype):
    """Steps from random states against the restatement; idle slots keep theirs; sums are cleared; rows between others."""
    from trl_b200.ops import cuda_mixers as K

    B, steps = 5, 4
    m, y, z, (q, f, v) = recurrent_case(B * steps, H, d, e, torch.float32, 2)
    S = gen(4)(B, H, d, e)
    state = dev(S)
    live = [0, 1, 3, 4]
    for s in range(steps):
        at = slice(s * B, s * B + B)
        sums = torch.full((B, 4 + H * (2 * d + e)), 5.0, device="cuda")
        sums[:, 4:] = dev(torch.cat([y[at], z[at]], 1))
        out = torch.full((B, H * e + 24), 7.0, dtype=dtype, device="cuda")
        K.hgrn2_step(sums[:, 4:], m, i32([s, 9, -1, 0, 3]), state, out[:, 8:8 + H * e], scale=0.6)
        assert not sums[:, 4:].any() and (sums[:, :4] == 5.0).all() and (out[:, :8] == 7.0).all() and (out[:, 8 + H * e:] == 7.0).all()
        for b in live:
            o, S[b] = ref.recurrence(q[at][b:b + 1], f[at][b:b + 1], v[at][b:b + 1], S[b])
            want = (0.6 * ref.norm(o[0], m.norm.double().cpu(), 1e-4)).reshape(-1)
            t = 2e-5 if dtype == torch.float32 else 2e-2
            assert torch.allclose(out[b, 8:8 + H * e].double().cpu(), want, atol=t, rtol=t)
            assert torch.allclose(state[b].double().cpu(), S[b], atol=1e-5, rtol=1e-5)
        assert torch.equal(state[2].cpu(), S[2].float())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,e", [(1, 1), (3, 10), (4, 128), (2, 136)])
def test_norm_per_head(H, e, dtype):
    from trl_b200.ops import cuda_mixers as K

    o, w = gen(e)(77, H, e), gen(1)(e)
    out = torch.full((77, H * e + 8), 7.0, dtype=dtype, device="cuda")
    K.head_norm(dev(o), dev(w), 1e-2, dtype, out=out[:, 4:4 + H * e], scale=-0.4)
    t = 3e-6 if dtype == torch.float32 else 1e-2
    assert torch.allclose(out[:, 4:4 + H * e].double().cpu(), -0.4 * ref.norm(o, w, 1e-2).reshape(77, -1), atol=t, rtol=t)
    assert (out[:, :4] == 7.0).all() and (out[:, 4 + H * e:] == 7.0).all()


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
    """A prompt of ``cut`` tokens, the rest one by one: first tokens, window and block edges, page borders (16-token pages)."""
    n = 40
    toks, want = wanted(name, n, 1, dtype)
    f = feed(name, dtype, block=16, max_len=96)
    got = [f.step([("a", toks[:cut], list(range(cut)))])[0]]
    for t in range(cut, n):
        got.append(f.step([("a", toks[t:t + 1], [0])])[0])
    assert U.rel(torch.cat(got), want) < tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(dtype):
    """Decoding over several tiles of the attention kernels and 64-token pages, every window passing over decoded tokens, more blocks
    than a tile."""
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
    """More requests than slots: the scheduler admits, shares prompt pages, copies means and states, retires and admits again."""
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

    m, _ = U.make(U.every_expert(U.ODD), bf16)  # the checkpoint is bf16 in both runs
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
