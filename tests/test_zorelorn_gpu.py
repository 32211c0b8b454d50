"""Zorelorn on the GPU: every kernel of its mechanisms, the serving engine's caches and states, generation.

The models are compared with the plain restatement (zorelorn_reference.py) in float64; float32 models are held to
rounding, bf16 models to bf16 rounding, and where that could hide a fault (a key at a window's edge, a sink, a far
key) the inputs are made so that one score stands out."""
import functools
import types

import pytest
import torch

import zorelorn_reference as ref
import zorelorn_util as U
from trl_b200.models import SeqCtx
from trl_b200.rollout.sampling import SamplingParams

pytestmark = pytest.mark.gpu

CFGS = {"odd": U.ODD, "tiles": U.TILES, "ones": U.ONES}
TOL = {torch.float32: 3e-5, torch.bfloat16: 0.12}
DTYPES = [torch.float32, torch.bfloat16]


def dev(x, dtype=torch.float32):
    return x.to("cuda", dtype)


@functools.lru_cache(maxsize=None)
def model(name, dtype):
    m, t = U.make(CFGS[name], dtype, "cuda")
    return m, t


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


# ---- mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H", [88, 33])
@pytest.mark.parametrize("dtype", DTYPES)
def test_dynamic_tanh(H, dtype):
    from trl_b200.ops import cuda_mixers as K

    x, d = torch.randn(7, H, dtype=torch.float64) * 3, torch.randn(7, H, dtype=torch.float64)
    w, b, a = torch.randn(H, dtype=torch.float64), torch.randn(H, dtype=torch.float64), torch.tensor(0.8, dtype=torch.float64)
    xg, dg = dev(x), dev(d)
    got = K.dynamic_tanh(xg, dg, dev(a), dev(w), dev(b), dtype, clear=True)
    want = ref.dynamic_tanh(x + d, a, w, b)
    tol = 1e-6 if dtype == torch.float32 else 2e-2
    assert torch.allclose(got.double().cpu(), want, atol=tol, rtol=tol)
    assert torch.allclose(xg.double().cpu(), x + d, atol=1e-6) and not dg.any()


@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu(dtype):
    from trl_b200.ops import cuda_mixers as K

    z = torch.linspace(-9, 9, 1001, dtype=torch.float64).to(dtype)
    want = 0.5 * z.double() * (1 + torch.erf(z.double() / 2 ** 0.5))
    tol = 1e-6 if dtype == torch.float32 else 1e-2
    assert torch.allclose(K.gelu_erf(z.cuda()).double().cpu(), want, atol=tol, rtol=tol)


def attention_case(T, m, dtype, seed=0):
    """Random q (head by head, rotated part last), keys / values and latent rows in the product's layouts."""
    from trl_b200.ops import cuda_mixers as K

    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64).to(dtype).double()
    q = rnd(T, m.heads, m.dim + m.rot_dim)
    kn, v, kr = rnd(T, m.heads, m.dim), rnd(T, m.heads, m.vdim), rnd(T, m.rot_dim)
    gate = torch.rand(T, m.heads, generator=g, dtype=torch.float64)
    off, w = K.latent_row(m.kv_rank, m.rot_dim)
    lat = torch.zeros(T, w, dtype=torch.float64)
    lat[:, off:off + m.rot_dim] = kr
    return q, kn, v, kr, gate, lat


def run_attention(m, q, kn, v, gate, lat, lens, dtype):
    from trl_b200.ops import mixers as mx

    T = q.shape[0]
    ctx = SeqCtx.from_lengths(lens, "cuda")
    kv = torch.cat([kn.reshape(T, -1), v.reshape(T, -1)], 1)
    out = mx.latent_prompt_attention(dev(q.reshape(T, -1), dtype), dev(kv, dtype), dev(lat, dtype), m, ctx, dev(gate))
    return out.double().cpu().view(T, m.heads, m.vdim)


def want_attention(m, q, kn, v, kr, gate, lens):
    k = torch.cat([kn, kr[:, None].expand(-1, m.heads, -1)], -1)
    outs, a = [], 0
    for n in lens:
        s = slice(a, a + n)
        outs.append(ref.sink_window_attention(q[s], k[s], v[s], m.scale, m.window, m.sink.double()))
        a += n
    return torch.cat(outs) * gate[..., None]


def spec(heads, dim, rot, vdim, window, scale=0.2, kv_rank=40):
    s = torch.linspace(-2, 3, heads)
    return types.SimpleNamespace(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, window=window, scale=scale, kv_rank=kv_rank,
                                 sink=s, eps=1e-5)


SHAPES = [(2, 64, 64, 64), (3, 24, 8, 40), (1, 128, 64, 128), (2, 72, 16, 136), (2, 13, 6, 9), (2, 16, 48, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [1, 5, 128, 131, None])
def test_prompt_attention(shape, window, dtype):
    lens = [1, 200, 37, 2]
    m = spec(*shape, window)
    q, kn, v, kr, gate, lat = attention_case(sum(lens), m, dtype)
    mg = types.SimpleNamespace(**{**m.__dict__, "sink": m.sink.cuda()})
    got = run_attention(mg, q, kn, v, gate, lat, lens, dtype)
    want = want_attention(m, q, kn, v, kr, gate, lens)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    assert (got - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 64, 127, 128, 129, 190])
def test_prompt_attention_window_edge(window, dtype):
    """The key at distance window - 1 dominates when visible; the one at distance window, as strong, must not be seen."""
    T = 200
    m = spec(2, 64, 32, 64, window, scale=1.0)
    m.sink = torch.full((2,), -5.0)
    mg = types.SimpleNamespace(**{**m.__dict__, "sink": m.sink.cuda()})
    for target in (window - 1, window):
        q, kn, v, kr, gate, lat = attention_case(T, m, dtype, seed=window)
        q, kn, kr, lat = q * 0.1, kn * 0.1, kr * 0.0, lat * 0.0
        at = [t for t in (window, 191, 199) if 0 <= t - target]
        for t in at:
            u = torch.nn.functional.normalize(torch.randn(64, dtype=torch.float64), dim=0)
            q[t, :, :64] = (u * 6).to(dtype).double()
            kn[t - target] = (u * 6).to(dtype).double()
        got = run_attention(mg, q, kn, v, gate, lat, [T], dtype)
        for t in at:
            seen = target == window - 1
            share = ((got[t] - v[t - target] * gate[t][:, None]).abs().max() < 0.05)
            assert bool(share) == seen, (t, target)
        want = want_attention(m, q, kn, v, kr, gate, [T])
        assert (got - want).abs().max() < (2e-5 if dtype == torch.float32 else 1.5e-2) * want.abs().max()


def test_prompt_attention_sink_weight():
    """One key with score 0 against a sink s: the value comes out times 1 / (1 + exp(s)), once per head."""
    m = spec(3, 64, 64, 64, 4)
    m.sink = torch.tensor([0.0, 2.0, -30.0])
    mg = types.SimpleNamespace(**{**m.__dict__, "sink": m.sink.cuda()})
    for dtype in DTYPES:
        q, kn, v, kr, gate, lat = attention_case(1, m, dtype)
        got = run_attention(mg, q * 0, kn, v, torch.ones_like(gate), lat, [1], dtype)
        want = v[0] / (1 + m.sink.double().exp())[:, None]
        assert torch.allclose(got[0], want, rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,E", [(2, 40, 64), (3, 20, 28), (1, 64, 128), (1, 128, 256), (2, 256, 72), (1, 1, 1)])
@pytest.mark.parametrize("forget", [0.0, 4.0])
def test_mlstm_prompt(H, D, E, forget, dtype):
    """Several sequences, chunk borders inside them, gates from nearly closed to dominating; then the state is right
    too: it is continued with a step kernel call."""
    from trl_b200.ops import cuda_mixers as K
    from trl_b200.ops import mixers as mx

    lens = [1, 130, 64, 65, 200]
    T = sum(lens)
    g = torch.Generator().manual_seed(H * D + E)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    qd, vd = H * D, H * E
    y = rnd(T, 2 * qd + 2 * vd).to(dtype).double()
    ig = (4 * rnd(T, H)).clamp(-9, 9)
    fg = torch.nn.functional.logsigmoid(forget + 3 * rnd(T, H))
    ig[150] = 9.0  # one token that outweighs the rest of its sequence
    m = types.SimpleNamespace(heads=H, dim=D, vdim=E, eps=1e-5, cap=9.0, gate_bias=torch.zeros(2 * H, device="cuda"))
    slots = torch.tensor([4, 0, 2, 5, 1], dtype=torch.int32, device="cuda")
    f32 = dict(dtype=torch.float32, device="cuda")
    state = (torch.full((6, H, D, E), 7.0, **f32), torch.full((2, 6, H, D), 7.0, **f32), torch.full((2, 6, H), 7.0, **f32))
    ctx = SeqCtx.from_lengths(lens, "cuda")
    got = mx.mlstm_prompt_scan(dev(y, dtype), m, dev(ig), dev(fg), ctx, dict(seq_slot=slots, state=state)).double().cpu()
    q = y[:, :qd].view(T, H, D) * D ** -0.5
    k, v = y[:, qd:2 * qd].view(T, H, D), y[:, 2 * qd:2 * qd + vd].view(T, H, E)
    # the step after each prompt: gates through the kernel's own cap and sigmoid
    nxt = rnd(6, 2 * qd + 2 * vd + 2 * H)
    lens_t = torch.full((6,), -1, dtype=torch.int32, device="cuda")
    lens_t[slots.long()] = torch.tensor(lens, dtype=torch.int32, device="cuda")
    out = torch.zeros(6, H, E, **f32)
    K.mlstm_step(dev(nxt), m, lens_t, state, out)
    w = {"i": torch.zeros(H, H, dtype=torch.float64), "f": torch.zeros(H, H, dtype=torch.float64)}
    a, tol = 0, (2e-4 if dtype == torch.float32 else 1e-2)
    for s, n in enumerate(lens):
        sl, r = slice(a, a + n), int(slots[s])
        w["i.b"], w["f.b"] = nxt[r, -2 * H:-H], nxt[r, -H:]
        i1, f1 = ref.mlstm_gates(torch.zeros(1, H, dtype=torch.float64), w, m.cap)
        want = ref.mlstm_recurrence(torch.cat([q[sl], nxt[r, :qd].view(1, H, D) * D ** -0.5]),
                                    torch.cat([k[sl], nxt[r, qd:2 * qd].view(1, H, D)]),
                                    torch.cat([v[sl], nxt[r, 2 * qd:2 * qd + vd].view(1, H, E)]),
                                    torch.cat([ig[sl], i1]), torch.cat([fg[sl], f1]))
        have = torch.cat([got[sl], out[r:r + 1].double().cpu()])
        # a position's error against what its neighbours weigh: the normaliser can be close to zero
        err = (have - want).abs().amax(-1) / (want.abs().amax(-1) + want.abs().mean())
        assert err.max() < tol, (s, float(err.max()))
        a += n


# ---- whole model --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 70), ("tiles", 200), ("ones", 20), ("odd", 1), ("tiles", 2)])
def test_whole_prompt(name, n, dtype):
    toks, want = wanted(name, n, 1)
    m, _ = model(name, dtype)
    with torch.no_grad():
        got = m(torch.tensor([toks], device="cuda")).logits[0]
    assert U.rel(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles", "ones"])
@pytest.mark.parametrize("cut", [1, 2, 17, 64, 65])
def test_prompt_then_tokens(name, cut, dtype):
    """A prompt of ``cut`` tokens, the rest one by one: window edges, page borders (16-token pages), first tokens."""
    n = 70
    toks, want = wanted(name, n, 1)
    f = feed(name, dtype, block=16, max_len=96)
    got = [f.step([("a", toks[:cut], list(range(cut)))])[0]]
    for t in range(cut, n):
        got.append(f.step([("a", toks[t:t + 1], [0])])[0])
    assert U.rel(torch.cat(got), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_decode_over_a_wide_window(dtype):
    """Decoding past the edge of a window of 150 and over several 64-token pages."""
    toks, want = wanted("tiles", 200, 1)
    f = feed("tiles", dtype, max_len=256)
    got = [f.step([("a", toks[:140], list(range(140)))])[0]]
    got += [f.step([("a", [t], [0])])[0] for t in toks[140:]]
    assert U.rel(torch.cat(got), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", [[2] * 10, [3, 2, 15], [10, 10]])
def test_portions(portions, dtype):
    toks, want = wanted("odd", 70, 1)
    f, at, got = feed("odd", dtype, block=16), 0, []
    for n in portions:
        got.append(f.step([("a", toks[at:at + n], list(range(n)))])[0])
        at += n
    assert U.rel(torch.cat(got), want[:at]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_unequal_batch_and_reused_slots(name, dtype):
    """Three unequal requests decode together, end at different times, and their slots and pages (the pool holds no
    more than they need) serve other requests afterwards."""
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
            assert U.rel(torch.cat(got[k]), seqs[k][1]) < TOL[dtype], (rnd, k)


def test_far_key_and_window_edge_in_decode():
    """Absorbed decode attention against the expanded form: one cached key stands out, just inside or outside."""
    from trl_b200.ops import cuda_mixers as K

    H, r, dr, bs, window = 3, 40, 16, 16, 50
    off, w = K.latent_row(r, dr)
    for dtype in DTYPES:
        for heads, pos, target in [(H, 120, window - 1), (H, 120, window), (H, 120, 0), (H, 31, 31), (H, 49, 49), (H, 50, 50),
                                   (20, 120, window - 1), (20, 120, window)]:
            m = types.SimpleNamespace(heads=heads, kv_rank=r, rot_dim=dr, window=window, scale=1.0,
                                      sink=torch.full((heads,), -4.0, device="cuda"))
            g = torch.Generator().manual_seed(pos + target)
            lat = torch.randn(pos + 1, w, generator=g, dtype=torch.float64) * 0.1
            lat[:, r:off] = 0
            lat[:, off + dr:] = 0
            q = torch.randn(2, heads, w, generator=g, dtype=torch.float64) * 0.1
            u = torch.nn.functional.normalize(torch.randn(w, generator=g, dtype=torch.float64), dim=0)
            u[r:off] = 0
            u[off + dr:] = 0
            q[1], lat[pos - target] = u * 5, u * 5
            q, lat = q.to(dtype).double(), lat.to(dtype).double()
            table = torch.zeros(2, 10, dtype=torch.int32)
            table[1, :9] = torch.randperm(9, generator=g) + 1
            cache = torch.full((10, bs, w), 3.0, dtype=torch.float64)
            for j in range(pos + 1):
                cache[table[1, j // bs], j % bs] = lat[j]
            cache[:, :, r:off] = 0
            cache[:, :, off + dr:] = 0
            out = torch.full((2, heads, r), 9.0, dtype=dtype, device="cuda")
            args = (dev(q, dtype), dev(cache, dtype), m, torch.tensor([-1, pos], dtype=torch.int32, device="cuda"), table.cuda(), bs)
            K.latent_decode(*args, out)
            outs = [out]
            m.dim, m.vdim = 8, 8
            assert K.latent_decode_tc_ok(m, bs)
            for splits in (1, 2, 3) if dtype == torch.bfloat16 else ():
                outs.append(torch.full((2, heads, r), 9.0, dtype=dtype, device="cuda"))
                scratch = torch.full((2, heads * splits * r), 5.0, device="cuda")
                K.latent_decode_tc(*args, outs[-1], scratch, torch.full((2, heads * splits * 2), 5.0, device="cuda"), splits)
            a = max(0, pos - window + 1)
            s = q[1] @ lat[a:].T
            p = s.exp() / (s.exp().sum(-1, keepdim=True) + torch.exp(torch.tensor(-4.0, dtype=torch.float64)))
            want = p @ lat[a:, :r]
            for out in outs:
                got = out[1].double().cpu()
                assert (got - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max(), (heads, pos, target)
                near = (got - lat[pos - target, :r]).abs().max() < 0.1 * lat[pos - target, :r].abs().max()
                assert bool(near) == (target < window)


@pytest.mark.parametrize("heads,r,dr,bs,window", [(5, 128, 64, 64, None), (32, 512, 64, 64, 300), (40, 96, 8, 16, 129), (64, 72, 40, 32, 128),
                                                  (100, 256, 32, 128, None), (2, 8, 8, 8, 1)])
def test_tensor_core_decode_attention(heads, r, dr, bs, window):
    """Ragged slots (idle ones included), several tiles and splits, scores large enough to move the reference maximum."""
    from trl_b200.ops import cuda_mixers as K

    lens = [0, 700, -1, 127, 128, 5, 300]
    B, off = len(lens), K.latent_row(r, dr)[0]
    w = K.latent_row(r, dr)[1]
    g = torch.Generator().manual_seed(heads)
    m = types.SimpleNamespace(heads=heads, kv_rank=r, rot_dim=dr, dim=8, vdim=8, window=window, scale=0.3,
                              sink=torch.randn(heads, generator=g).cuda())
    pages = -(-701 // bs)
    table = (torch.randperm(B * pages, generator=g) + 1).view(B, pages).int()
    cache = torch.randn(B * pages + 1, bs, w, generator=g, dtype=torch.float64)
    cache[:, :, r:off] = 0
    cache[:, :, off + dr:] = 0
    q = torch.randn(B, heads, w, generator=g, dtype=torch.float64) * (2.0 / w ** 0.5) * 8
    q[:, :, r:off] = 0
    q[:, :, off + dr:] = 0
    cache, q = cache.bfloat16().double(), q.bfloat16().double()
    assert K.latent_decode_tc_ok(m, bs)
    for splits in (1, 3):
        out = torch.zeros(B, heads, r, dtype=torch.bfloat16, device="cuda")
        K.latent_decode_tc(dev(q, torch.bfloat16), dev(cache, torch.bfloat16), m, torch.tensor(lens, dtype=torch.int32, device="cuda"),
                           table.cuda(), bs, out, torch.full((B, heads * splits * r), 5.0, device="cuda"),
                           torch.full((B, heads * splits * 2), 5.0, device="cuda"), splits)
        for b, pos in enumerate(lens):
            if pos < 0:
                assert not out[b].any()
                continue
            rows = torch.cat([cache[int(x)] for x in table[b]])[max(0, pos - window + 1) if window else 0:pos + 1]
            s = q[b] @ rows.T * m.scale
            top = torch.maximum(s.amax(-1), m.sink.double().cpu())
            e = (s - top[:, None]).exp()
            want = e @ rows[:, :r] / (e.sum(-1) + (m.sink.double().cpu() - top).exp())[:, None]
            assert (out[b].double().cpu() - want).abs().max() < 1e-2 * max(1.0, float(want.abs().max())), (b, splits)


@pytest.mark.parametrize("B", [1, 17, 64, 128, 130])
@pytest.mark.parametrize("H,M,Kd", [(3, 128, 64), (2, 200, 40), (1, 16, 520)])
@pytest.mark.parametrize("w_mn", [False, True])
def test_head_gemm(B, H, M, Kd, w_mn):
    from trl_b200.ops import cuda_mixers as K

    g = torch.Generator().manual_seed(B + M)
    x = torch.randn(B, H, Kd + 8, generator=g).bfloat16().cuda()
    w = torch.randn(*((H, Kd, M) if w_mn else (H, M, Kd)), generator=g).bfloat16().cuda()
    sc = torch.rand(B, H, generator=g).cuda()
    y = torch.zeros(B, H, M + 24, dtype=torch.bfloat16, device="cuda")
    K.head_gemm(x, w, y, w_mn=w_mn, scale=sc)
    want = torch.einsum("bhk,hkm->bhm" if w_mn else "bhk,hmk->bhm", x[..., :Kd].double(), w.double()) * sc.double()[..., None]
    assert torch.allclose(y[..., :M].double(), want, rtol=1e-2, atol=1e-2 * Kd ** 0.5)
    assert not y[..., M:].any()


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("n", [1, 3])
def test_greedy_generation_through_the_engine(n, graph):
    """More requests than slots: the scheduler admits, shares prompt pages and states, retires and admits again."""
    from trl_b200.rollout.engine import make_engine

    m, t = model("odd", torch.float32)
    eng = make_engine(m, max_num_seqs=4, max_model_len=64, block_size=8, poll_every=3, use_cuda_graph=graph)
    prompts = [U.tokens(k, 203, 20 + k) for k in (5, 16, 1, 23)]
    for _ in range(2):
        outs = eng.generate(prompts, SamplingParams(n=n, max_tokens=9, greedy=True))
        for i, p in enumerate(prompts):
            seq = list(p)
            want = greedy(tuple(p))
            for o in outs[i * n:(i + 1) * n]:
                assert o.token_ids == want and o.finish_reason == "length"


@functools.lru_cache(maxsize=None)
def greedy(prompt):
    _, t = U.make(U.ODD)
    seq = list(prompt)
    for _ in range(9):
        seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_bf16_generation_follows_the_fed_tokens():
    """Tokens and log-probs of a sampled bf16 run are those of the same tokens fed through the cache."""
    from trl_b200.rollout.engine import make_engine

    m, _ = model("tiles", torch.bfloat16)
    eng = make_engine(m, max_num_seqs=3, max_model_len=128)
    prompts = [U.tokens(k, 203, k) for k in (30, 7, 64, 2)]
    outs = eng.generate(prompts, SamplingParams(n=2, max_tokens=20, temperature=1.0, seed=5))
    for o in outs:
        f = feed("tiles", torch.bfloat16, slots=2, max_len=128)
        toks = o.prompt_ids + o.token_ids
        lg = f.step([("x", toks[:-1], list(range(len(o.prompt_ids) - 1, len(toks) - 1)))])[0]
        lp = torch.log_softmax(lg, -1).cpu().gather(1, torch.tensor(o.token_ids)[:, None])[:, 0]
        assert (lp - torch.tensor(o.logprobs)).abs().max() < 0.12


def test_gradients_are_refused():
    m, _ = U.make(U.ONES, torch.bfloat16, "cuda")
    m.requires_grad_(True)
    with pytest.raises(NotImplementedError, match="inference only"):
        m(torch.tensor([[1, 2, 3]], device="cuda"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_command(tmp_path, dtype):
    """bin/trace_run in a process of its own: unequal requests, requests that end, logits written in the order asked for."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    m, t = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path / "m"))
    (tmp_path / "out").mkdir()
    a, wa = wanted("odd", 70, 1)
    b, wb = wanted("odd", 70, 2)
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
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4").copy()).view(-1, 203)
        assert U.rel(got, w) < TOL[getattr(torch, dtype)]
