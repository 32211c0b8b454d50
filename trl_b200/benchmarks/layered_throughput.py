"""Prompt and decode throughput of a layered design beside the closest flat decoder of the same width, depth and
parameter count (random weights, bf16, one GPU), through the serving engine.

    python -m trl_b200.benchmarks.layered_throughput [--design zorelorn|povusun|suposun|gerupel] [--sizes small,base] [--kernels]

Prompt: packed prompts through the engine's prompt forward into its cache.  Decode: replays of the captured step (CUDA
graph, sampler included) with every slot at the given context.  CUDA events after warm-up; the weights of a step are
larger than L2.  ``--kernels`` times the mixers' kernels alone, L2 flushed in between, against the measured peaks."""
from __future__ import annotations

import argparse
import json
import os

import torch

# width, heads (attention of every kind), ff; Zorelorn: query latent, mLSTM heads, pairs of layers; Povusun: side input, quads;
# Suposun: experts of every second layer, of which a token runs `top` of width `eff` (ff = top x eff), quads; Gerupel: heads of the
# recurrent half (128 x 128), experts of every layer, layers, of which the third and fourth run twice
SIZES = {"zorelorn": {"small": dict(width=2048, heads=16, q_rank=768, ff=8192, mheads=4, pairs=4),
                      "base": dict(width=4096, heads=32, q_rank=1536, ff=16384, mheads=8, pairs=4)},
         "povusun": {"small": dict(width=2048, heads=16, ff=6144, side=256, quads=2),
                     "base": dict(width=4096, heads=32, ff=12288, side=256, quads=2)},
         "suposun": {"small": dict(width=2048, heads=16, ff=4096, eff=1024, experts=48, top=4, quads=2),
                     "base": dict(width=4096, heads=32, ff=8192, eff=2048, experts=32, top=4, quads=2)},
         "gerupel": {"small": dict(width=2048, heads=16, rheads=16, ff=4096, eff=1024, experts=32, top=4, layers=6),
                     "base": dict(width=4096, heads=32, rheads=32, ff=8192, eff=2048, experts=24, top=4, layers=6)}}
VOCAB = 32768


def zorelorn_config(width, heads, q_rank, ff, mheads, pairs, window=1024):
    att = dict(type="latent_attention", mlp=dict(kind="dense", ff=ff),
               mixer=dict(heads=heads, dim=128, rot_dim=64, vdim=128, q_rank=q_rank, kv_rank=512, scale=192 ** -0.5,
                          mask=dict(size=window), rot=dict(base=1e4, dims=64, scaling=dict(factor=4.0, original=4096,
                                                                                          fast=32.0, slow=1.0))))
    rec = dict(type="mlstm", mlp=dict(kind="dense", ff=ff), mixer=dict(heads=mheads, dim=256, vdim=512, gate_cap=15.0))
    return dict(architecture="Zorelorn", vocab=VOCAB, width=width, norm=dict(eps=1e-6), embedding=dict(scale=1.0),
                layers=[att, rec] * pairs)


def povusun_config(width, heads, ff, side, quads):
    mlp = dict(kind="dense", ff=ff, limit=7.0)
    att = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0, q_temp=dict(coef=0.1, every=1024))
    lat = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=128, vdim=128, kv_rank=512, scale=128 ** -0.5))
    rec = dict(type="rglru", mlp=mlp, mixer=dict(width=width, blocks=width // 256, conv=4))
    layers = []
    for i in range(quads):  # every second attention layer reads the cache of the one before
        own = dict(att, kv_from=4 * (i - 1)) if i % 2 else att
        layers += [dict(type="attention", mlp=mlp, mixer=own), rec, lat, rec]
    return dict(architecture="Povusun", vocab=VOCAB, width=width, norm=dict(eps=1e-6), token_side=dict(dim=side), layers=layers)


def suposun_config(width, heads, ff, eff, experts, top, quads, window=512):
    dense, moe = dict(kind="dense", ff=ff), dict(kind="moe", expert=dict(ff=eff, limit=7.0), router=dict(experts=experts, top=top))
    rot = dict(base=5e5, dims=64, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))
    near = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, mask=dict(size=window, keep_first=4), rot=rot)
    far = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, rot=dict(base=1e6, dims=128))
    layers = []
    for i in range(quads):  # the last layer of every second four reads the cache of the one four layers before
        own = dict(far, kv_from=4 * i - 1) if i % 2 else far
        layers += [dict(type="attention", mixer=near, mlp=m) for m in (dense, moe, dense)] + [dict(type="attention_2", mixer=own, mlp=moe)]
    return dict(architecture="Suposun", vocab=VOCAB, width=width, norm=dict(eps=1e-6), logit_scale=0.5, layers=layers,
                embedding=dict(scale=1.0, bigram=dict(buckets=8191, mul_prev=131, mul_cur=7)))


def gerupel_config(width, heads, rheads, ff, eff, experts, top, layers, window=512, pool=16):
    rot = dict(base=5e5, dims=128, scaling=dict(factor=8.0, original=8192, low=1.0, high=4.0))
    left = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=window, pool=pool), rot=rot)
    layer = dict(type="parallel", mixer=dict(left=left, right=dict(heads=rheads, dim=128, vdim=128), left_scale=0.9, right_scale=0.7),
                 mlp=dict(kind="moe", expert=dict(ff=eff), router=dict(experts=experts, top=top, scale=1.5)))
    return dict(architecture="Gerupel", vocab=VOCAB, width=width, norm=dict(eps=1e-6), residual_mult=0.8, layers=[layer] * layers,
                loop=dict(start=2, stop=4, times=2) if layers > 3 else None)


CONFIGS = {"zorelorn": zorelorn_config, "povusun": povusun_config, "suposun": suposun_config, "gerupel": gerupel_config}


def layered_config(design, s):
    return CONFIGS[design](**s)


def flat_config(s, depth, target, tied):
    """Flat decoder of the same width and depth brought to ``target`` parameters: of the Llama type by the width of its
    feed-forward, or, where the layered design has experts, of the Qwen3-MoE type with experts in every layer by their number."""
    from ..models.configuration import ModelArch

    if "experts" in s:
        kw = dict(model_type="qwen3_moe", vocab_size=VOCAB, hidden_size=s["width"], num_hidden_layers=depth, intermediate_size=s["ff"],
                  num_attention_heads=s["width"] // 128, num_key_value_heads=max(1, s["width"] // 512), head_dim=128, rope_theta=5e5,
                  tie_word_embeddings=tied, moe_intermediate_size=s["eff"], num_experts_per_tok=s["top"])
        one, two = (ModelArch(num_experts=n, **kw).num_parameters() for n in (s["top"], s["top"] + 1))
        return ModelArch(num_experts=s["top"] + max(0, round((target - one) / (two - one))), **kw)
    kw = dict(model_type="llama", vocab_size=VOCAB, hidden_size=s["width"], num_hidden_layers=depth,
              num_attention_heads=s["width"] // 128, num_key_value_heads=max(1, s["width"] // 512), head_dim=128,
              rope_theta=5e5, tie_word_embeddings=tied)
    rest = target - ModelArch(intermediate_size=0, **kw).num_parameters()
    return ModelArch(intermediate_size=max(256, rest // (kw["num_hidden_layers"] * 3 * s["width"]) // 256 * 256), **kw)


def timed(fn, iters, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


@torch.no_grad()
def measure(model, batch, prompt, n_prompts, iters=10):
    from ..ops import cuda as K
    from ..rollout.engine import make_engine
    from ..rollout.sampling import SamplingParams

    eng = make_engine(model, max_num_seqs=batch, max_model_len=prompt + 192)
    toks = [torch.randint(2, VOCAB, (prompt,)).tolist() for _ in range(n_prompts)]
    sp = SamplingParams(n=max(1, batch // n_prompts), max_tokens=64, seed=1)
    eng.generate(toks, sp)  # fills the cache and captures the decode graph
    bt = eng.block_table_host.numpy()
    for i, t in enumerate(toks):
        eng.sched.add(i, len(t), 64, i)
    owners = [(slot, toks[rid]) for rid, slot, _, _ in eng.sched.admit(bt)]
    eng.block_table.copy_(eng.block_table_host)
    n0 = K.LAUNCHES[0]
    ms_prompt = timed(lambda: eng._prefill_all(owners), iters)
    launches = K.LAUNCHES[0] - n0
    for slot, _ in owners:
        eng.sched.retire(slot, slot)
    eng.block_table.copy_(torch.arange(eng.block_table.numel(), device=eng.dev).view_as(eng.block_table).remainder(eng.num_blocks))

    def step():
        eng._graph.replay()

    eng.n_gen.zero_()
    eng.finished.zero_()
    eng.seq_lens.fill_(prompt)
    ms_step = timed(step, 40)
    K.check_status()
    return dict(prompt_tok_s=round(n_prompts * prompt / ms_prompt * 1e3), prompt_ms=round(ms_prompt, 3),
                decode_tok_s=round(batch / ms_step * 1e3), decode_ms=round(ms_step, 4), own_prompt_launches=launches)


def run(sizes=("small", "base"), batch=64, prompt=1024, n_prompts=8, design="zorelorn"):
    from ..models.configuration import ModelArch
    from ..models.hf_io import build_model

    out = []
    for name in sizes:
        s = SIZES[design][name]
        arch = ModelArch.from_hf_dict(layered_config(design, s))
        depth = arch.num_hidden_layers
        # tables of side inputs and token pairs are looked up, not multiplied with: they do not count as size
        tables = VOCAB * depth * arch.side_dim + (arch.pairs["buckets"] + 1 if arch.pairs else 0) * arch.hidden_size
        n = arch.num_parameters() - tables
        flat = flat_config(s, depth, n, arch.tie_word_embeddings)
        row = dict(design=design, size=name, layers=depth, width=s["width"], batch=batch, prompt=f"{n_prompts}x{prompt}",
                   decode_context=prompt)
        for key, cfg in (("layered", arch), ("flat", flat)):
            torch.manual_seed(0)
            model = build_model(cfg, dtype=torch.bfloat16, device="cuda").eval().requires_grad_(False)
            params = sum(p.numel() for p in model.parameters()) - (tables if key == "layered" else 0)
            row[key] = dict(params_m=round(params / 1e6), **measure(model, batch, prompt, n_prompts))
            del model
            torch.cuda.empty_cache()
        row["prompt_ratio"] = round(row["layered"]["prompt_tok_s"] / row["flat"]["prompt_tok_s"], 3)
        row["decode_ratio"] = round(row["layered"]["decode_tok_s"] / row["flat"]["decode_tok_s"], 3)
        out.append(row)
    return out


def peaks():
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


class KernelTimer:
    """Times kernels alone (cold L2): median time and the fraction of the roofline, which is the larger of bytes / measured
    copy bandwidth and operations / measured bf16 GEMM throughput."""

    def __init__(self, iters=20):
        self.iters, self.rows = iters, []
        self.bw, self.fl = peaks()
        # larger than L2, and long enough that the host has launched everything of an iteration before the first event
        self.flush = torch.empty(2 << 30, dtype=torch.uint8, device="cuda")

    def __call__(self, name, fn, nbytes, flops=0.0):
        for _ in range(3):
            fn()
        ev = []
        for _ in range(self.iters):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            ev.append((a, b))
        torch.cuda.synchronize()
        us = sorted(a.elapsed_time(b) * 1e3 for a, b in ev)[self.iters // 2]
        roof = max(nbytes / self.bw, flops / self.fl) * 1e6
        self.rows.append(dict(kernel=name, us=round(us, 1), roof_us=round(roof, 2), frac=round(roof / us, 3)))


def kernel_table(size="base", batch=64, prompt=1024, n_prompts=8, iters=20, design="zorelorn"):
    """Time of every mixer kernel alone beside the like kernels of the flat decoder."""
    from ..models.configuration import ModelArch
    from ..models.hf_io import build_model
    from ..ops import cuda as K
    from ..rollout.engine import make_engine

    s = dict(SIZES[design][size], **{"zorelorn": dict(pairs=1), "gerupel": dict(layers=1)}.get(design, dict(quads=1)))
    kernels = {"zorelorn": zorelorn_kernels, "povusun": povusun_kernels, "suposun": suposun_kernels, "gerupel": gerupel_kernels}[design]
    model = build_model(ModelArch.from_hf_dict(layered_config(design, s)), dtype=torch.bfloat16, device="cuda").eval().requires_grad_(False)
    eng = make_engine(model, max_num_seqs=batch, max_model_len=prompt + 64)
    row = KernelTimer(iters)
    kernels(s, model, eng, batch, prompt, n_prompts, row)
    flat_kernels(s, batch, prompt, n_prompts, row)
    K.check_status()
    return row.rows


def paged_context(eng, prompt):
    """Every slot at the given context, its pages spread over the cache."""
    eng.seq_lens.fill_(prompt)
    eng.block_table.copy_(torch.arange(eng.block_table.numel(), device=eng.dev).view_as(eng.block_table).remainder(eng.num_blocks))


@torch.no_grad()
def povusun_kernels(s, model, eng, batch, prompt, n_prompts, row):
    from ..models.decoder import SeqCtx
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    at, rg, la = (model.layers[i].mixer for i in range(3))
    T, W, dev, bf, B = n_prompts * prompt, s["width"], "cuda", torch.bfloat16, batch
    ctx = SeqCtx.from_lengths([prompt] * n_prompts, dev)
    h = torch.randn(T, W, device=dev, dtype=bf)
    x, d, nrm = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev), model.norm
    pairs = n_prompts * prompt * (prompt + 1) / 2
    row("prompt norm of output + residual + norm", lambda: KM.rms_residual(x, d, nrm.weight, nrm.weight, nrm.eps, bf), T * W * 14)
    y = mx.linear(h, at.w_in)
    temp = at.temperature.table(prompt, dev)
    kv = at.kv_heads * (at.dim + at.vdim)
    where = eng.slots[0].prompt_target(eng._page_writer(torch.arange(n_prompts, device=dev, dtype=torch.int32).repeat_interleave(prompt), ctx, None))
    paged_context(eng, prompt)
    row("prompt attention preparation + cache", lambda: KM.attn_prep(y, at, ctx.positions, temp, **where),
        T * 2 * (2 * (at.heads + at.kv_heads) * at.dim + at.kv_heads * at.vdim + kv))
    q, k, v, g = y.split(at.parts, 1)
    row("prompt grouped attention (capped, gated)", lambda: KM.mixer_attn(q, k, v, heads=at.heads, kv_heads=at.kv_heads, scale=at.scale, cap=at.cap,
                                                                          gate_logits=g, ctx=ctx),
        T * 2 * (y.shape[1] + at.heads * at.vdim), 2 * pairs * at.heads * (at.dim + at.vdim))
    row("prompt grouped attention without cap", lambda: KM.mixer_attn(q, k, v, heads=at.heads, kv_heads=at.kv_heads, scale=at.scale,
                                                                      gate_logits=g, ctx=ctx),
        T * 2 * (y.shape[1] + at.heads * at.vdim), 2 * pairs * at.heads * (at.dim + at.vdim))
    del y, q, k, v, g
    acc = mx.linear_f32(h, la.w_in[la.q_rows:])
    lw = KM.latent_row(la.kv_rank, 0)[1]
    lat = torch.zeros(T, lw, device=dev, dtype=bf)
    row("prompt latent preparation", lambda: KM.latent_prep(acc, la, ctx.positions, None, lat=lat), T * (acc.shape[1] * 4 + lw * 2))
    KM.latent_prep(acc, la, ctx.positions, None, lat=lat)
    q, ukv = mx.linear(h, la.w_in[: la.q_rows]), mx.linear(lat[:, : la.kv_rank], la.ukv)
    row("prompt latent attention", lambda: mx.latent_prompt_attention(q, ukv, lat, la, ctx, None),
        (q.numel() + ukv.numel() + T * la.heads * la.vdim) * 2, 2 * pairs * la.heads * (la.dim + la.vdim))
    del q, ukv, acc
    yx = mx.linear(h, rg.w_in)
    gy, gx = yx.chunk(2, 1)
    C, wb = rg.width, rg.width // rg.blocks
    row("prompt convolution", lambda: KM.conv_prompt(gx, rg, ctx), T * C * 4)
    u = KM.conv_prompt(gx, rg, ctx)
    row("prompt rglru (gates + scan + output)", lambda: KM.rglru_prompt_tc(u, gy, rg, ctx), T * C * 6 + rg.gates.numel() * 2, 4 * T * C * wb)
    del yx, gy, gx, u
    z = torch.randn(T, 2 * s["ff"], device=dev, dtype=bf)
    mlp, side = model.layers[0].mlp, model.layers[0].side
    row("prompt clamped unit", lambda: KM.clamped_glu(z, *mlp.glu), z.numel() * 3)
    del z
    zs, ids = torch.randn(T, side.dim, device=dev, dtype=bf), torch.randint(0, VOCAB, (T,), device=dev)
    row("prompt side gate", lambda: KM.side_gate(zs, ids, model.side_embed, 0), T * side.dim * 6)

    a, r, l = eng.slots[0], eng.slots[1], eng.slots[2]
    hb, xb, db = torch.randn(B, W, device=dev, dtype=bf), torch.randn(B, W, device=dev), torch.randn(B, W, device=dev)
    row("decode norm of output + residual + norm", lambda: KM.rms_residual(xb, db, nrm.weight, nrm.weight, nrm.eps, bf, clear=True, out=hb), B * W * 18)
    row("decode gemm input attention", lambda: K.decode_gemm(hb, at.w_in, y32=a.acc_in), at.w_in.numel() * 2)
    row("decode attention preparation + cache", a.prepare, a.acc_in.numel() * 10)
    row("decode grouped attention (capped, gated)", a.attend,
        B * (prompt + 1) * kv * 2 + (a.q.numel() + 2 * a.o.numel()) * 2, 2 * B * (prompt + 1) * at.heads * (at.dim + at.vdim))
    row("decode latent preparation", lambda: KM.latent_prep(l.acc_prep, la, eng.seq_lens, None, clear=True, cache=l.cache,
                                                            block_table=eng.block_table, block_size=eng.block_size), B * la.kv_rank * 10)
    row("decode absorb", l.absorb, la.uk.numel() * 2 + l.acc_q.numel() * 8 + l.q_lat.numel() * 2, 2 * B * la.heads * la.dim * la.kv_rank)
    row("decode latent attention", l.attend, B * (prompt + 1) * lw * 2 + (l.q_lat.numel() + l.o_lat.numel()) * 2,
        2 * B * (prompt + 1) * la.heads * (lw + la.kv_rank))
    row("decode expand", l.expand, la.uv.numel() * 2 + (l.o_lat.numel() + l.o.numel()) * 2, 2 * B * la.heads * la.vdim * la.kv_rank)
    row("decode convolution", r.convolve, B * C * (8 + 8 * (rg.taps - 1) + 2))
    row("decode rglru (gates + step + output)", r.recur, B * C * (2 + 8 + 8 + 2) + rg.gates.numel() * 2, 4 * B * C * wb)
    row("decode gate/up + clamped unit", lambda: eng.mlp_act(hb, mlp), mlp.gate_up.numel() * 2)
    row("decode side gate gemm", lambda: eng.gemm(hb, side.gate, eng.sums("side", side.dim)), side.gate.numel() * 2)
    row("decode side gate", lambda: KM.side_gate(eng.sums("side", side.dim), eng.next_input, model.side_embed, 0, clear=True), B * side.dim * 12)


@torch.no_grad()
def suposun_kernels(s, model, eng, batch, prompt, n_prompts, row):
    from ..models.decoder import SeqCtx
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    near, far, glu, moe = model.layers[0].mixer, model.layers[3].mixer, model.layers[0].mlp, model.layers[1].mlp
    T, W, dev, bf, B = n_prompts * prompt, s["width"], "cuda", torch.bfloat16, batch
    ctx = SeqCtx.from_lengths([prompt] * n_prompts, dev)
    h, post = torch.randn(T, W, device=dev, dtype=bf), model.layers[0].norm1b
    x, d = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
    slots = torch.arange(n_prompts, device=dev, dtype=torch.int32).repeat_interleave(prompt)
    pages = eng._page_writer(slots, ctx, None)
    paged_context(eng, prompt)
    ids, p = torch.randint(0, VOCAB, (T,), device=dev), model.config.pairs
    row("prompt embedding + pair embedding", lambda: KM.embed_pairs(ids, model.embed_tokens, 1.0, model.pair_embed, p["mul_prev"], p["mul_cur"], ctx.positions),
        T * W * 8)
    row("prompt norm of output + layer scale + residual", lambda: KM.rms_residual(x, d, post.weight, None, post.eps, bf, shift=1.0, post_scale=post.scale), T * W * 14)

    def qkv(m, li, name):
        y = mx.linear(h, m.w_in)
        keys = None if m.values else torch.empty(T, m.kv_heads * m.dim, device=dev, dtype=bf)
        gate = torch.empty(T, m.heads, device=dev) if m.gate else None
        table = m.rope.table(prompt, dev)
        kv = m.kv_heads * (m.dim + m.vdim)
        # in place: queries (and keys) read and written, values read, pages written; keys apart: read once, written twice and copied
        moved = 2 * m.heads * m.dim + (2 * m.kv_heads * m.dim + m.kv_heads * m.vdim if m.values else 2 * m.kv_heads * m.dim) + kv
        row(f"prompt preparation of {name}", lambda: KM.attn_prep(y, m, ctx.positions, None, table=table, k=keys, head_gate=gate, **m.prep,
                                                                  **eng.slots[li].prompt_target(pages)), T * 2 * moved)
        q, k, v, g = y[:, : sum(m.parts)].split(m.parts, 1)
        return (q, k, v, None) if m.values else (q, keys, k, gate)

    def attend(m, q, k, v, g, name, window, **kw):
        win = min(window or prompt, prompt)
        pairs = n_prompts * (win * (win + 1) / 2 + (prompt - win) * win)
        row(name, lambda: KM.mixer_attn(q, k, v, heads=m.heads, kv_heads=m.kv_heads, scale=m.scale, window=window, gate=g, ctx=ctx, **kw),
            T * 2 * (q.shape[1] + k.shape[1] + v.shape[1] + m.heads * m.vdim), 2 * pairs * m.heads * (m.dim + m.vdim))

    t = qkv(near, 0, "attention (keys as values)")
    attend(near, *t, "prompt windowed attention (capped, sink, gated)", near.window, keep=near.keep, cap=near.cap, sink=near.sink)
    attend(near, *t, "prompt windowed attention without cap", near.window, keep=near.keep, sink=near.sink)
    attend(near, *t, "prompt attention without window (capped, sink, gated)", None, cap=near.cap, sink=near.sink)
    t = qkv(far, 3, "attention_2 (norms over all heads)")
    attend(far, *t, "prompt attention_2", None)
    del t
    z = torch.randn(T, 2 * s["ff"], device=dev, dtype=bf)
    row("prompt GELU unit", lambda: KM.gelu_glu(z), z.numel() * 3)
    del z
    prompt_expert_kernels(moe, h, row)

    a, r = eng.slots[0], eng.slots[3]
    hb, xb, db = torch.randn(B, W, device=dev, dtype=bf), torch.randn(B, W, device=dev), torch.randn(B, W, device=dev)
    row("decode embedding + pair embedding", lambda: KM.embed_pairs(eng.next_input, model.embed_tokens, 1.0, model.pair_embed, p["mul_prev"], p["mul_cur"],
                                                                    eng.seq_lens, prev=eng.last_token, decode=True, out=xb), B * W * 8)
    row("decode norm of output + layer scale + residual", lambda: KM.rms_residual(xb, db, post.weight, None, post.eps, bf, clear=True, out=hb, shift=1.0,
                                                                                 post_scale=post.scale), B * W * 18)
    kv = near.kv_heads * 256
    row("decode gemm input attention", lambda: K.decode_gemm(hb, a.w_in, y32=a.acc_in), a.w_in.numel() * 2)
    row("decode preparation of attention + cache", a.prepare, a.acc_in.numel() * 10)
    row("decode gemm input attention_2", lambda: K.decode_gemm(hb, r.w_in, y32=r.acc_in), r.w_in.numel() * 2)
    row("decode preparation of attention_2 + cache", r.prepare, r.acc_in.numel() * 10)
    seen = min(prompt + 1, near.window + near.keep)
    row("decode windowed attention (capped, sink, gated)", a.attend, B * seen * kv * 2 + 4 * a.q.numel(), 2 * B * seen * near.heads * 256)
    row("decode attention_2", r.attend, B * (prompt + 1) * kv * 2 + 4 * r.q.numel(), 2 * B * (prompt + 1) * far.heads * 256)
    row("decode gate/up + GELU unit", lambda: eng.mlp_act(hb, glu), glu.gate_up.numel() * 2)
    decode_expert_kernels(eng, moe, hb, db, row)


@torch.no_grad()
def prompt_expert_kernels(moe, h, row):
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    E, top, n = moe.n, moe.top, moe.ff
    T, W = h.shape
    R = T * top
    zr = mx.linear_f32(h, moe.router)
    row("prompt router choice", lambda: KM.moe_route(zr, moe.correction, top, **moe.routing), T * (E * 4 + top * 12))
    choice, rank, weight, counts = KM.moe_route(zr, moe.correction, top, **moe.routing)
    row("prompt gather by expert", lambda: KM.moe_gather(h, choice, rank, counts), T * W * 2 + R * W * 2)
    xs, at, offsets = KM.moe_gather(h, choice, rank, counts)
    row("prompt experts gate/up + gated unit", lambda: K.grouped_gemm(xs, moe.gate_up, offsets, n, clamped_glu=moe.glu),
        moe.gate_up.numel() * 2 + R * (W + n) * 2, 4 * R * W * n)
    act = K.grouped_gemm(xs, moe.gate_up, offsets, n, clamped_glu=moe.glu)
    row("prompt experts down", lambda: K.grouped_gemm(act, moe.down, offsets, W), moe.down.numel() * 2 + R * (W + n) * 2, 2 * R * W * n)
    ys = K.grouped_gemm(act, moe.down, offsets, W)
    row("prompt weighted sum", lambda: KM.moe_sum(ys, at, weight), R * W * 2 + T * W * 4)
    row("prompt experts, all of it", lambda: mx.experts(moe, h), moe.gate_up.numel() * 3 + T * W * 6, 6 * R * W * n)


@torch.no_grad()
def decode_expert_kernels(eng, moe, hb, db, row):
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    (B, W), E, top, n = hb.shape, moe.n, moe.top, moe.ff
    zb = torch.zeros(B, E, device=hb.device)
    row("decode router product", lambda: K.decode_gemm(hb, moe.router, y32=zb), moe.router.numel() * 2)
    zb = mx.linear_f32(hb, moe.router)
    row("decode router choice", lambda: KM.moe_route(zb, moe.correction, top, positions=eng.seq_lens, **moe.routing), B * (E * 4 + top * 12))
    choice, rank, weight, counts = KM.moe_route(zb, moe.correction, top, **moe.routing)
    row("decode gather by expert", lambda: KM.moe_gather(hb, choice, rank, counts), B * W * 2 * (1 + top))
    xs, at, offsets = KM.moe_gather(hb, choice, rank, counts)
    used = int((counts > 0).sum())
    row("decode experts gate/up + gated unit", lambda: K.grouped_gemm(xs, moe.gate_up, offsets, n, clamped_glu=moe.glu), used * 4 * W * n)
    act = K.grouped_gemm(xs, moe.gate_up, offsets, n, clamped_glu=moe.glu)
    row("decode experts down", lambda: K.grouped_gemm(act, moe.down, offsets, W), used * 2 * W * n)
    ys = K.grouped_gemm(act, moe.down, offsets, W)
    row("decode weighted sum", lambda: KM.moe_sum(ys, at, weight, out=db), B * W * (2 * top + 4))
    row("decode experts, all of it", lambda: eng.experts(hb, moe, db), used * 6 * W * n)


@torch.no_grad()
def gerupel_kernels(s, model, eng, batch, prompt, n_prompts, row):
    from ..models.decoder import SeqCtx
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    m, moe, layer = model.layers[0].mixer, model.layers[0].mlp, model.layers[0]
    at, rg = m.left, m.right
    T, W, dev, bf, B = n_prompts * prompt, s["width"], "cuda", torch.bfloat16, batch
    ctx = SeqCtx.from_lengths([prompt] * n_prompts, dev)
    h = torch.randn(T, W, device=dev, dtype=bf)
    x, d = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
    of_seq = torch.arange(n_prompts, device=dev, dtype=torch.int32)
    target = eng.slots[0].prompt_target(eng._page_writer(of_seq.repeat_interleave(prompt), ctx, of_seq))
    paged_context(eng, prompt)
    ids = torch.randint(0, VOCAB, (T,), device=dev)
    row("prompt embedding + norm", lambda: KM.embed_normed(ids, model.embed_tokens, 1.0, model.embed_norm.weight, 1e-6), T * W * 6)
    ys = mx.experts(moe, h, summed=False)
    row("prompt experts' sum + residual + both norms", lambda: KM.rms_residual(x, (d, ys), None, layer.norm1.weight, 1e-6, bf, w2=layer.norm2.weight, mult=0.8),
        T * W * (16 + 2 * moe.top))
    del ys
    y, z = mx.linear(h, m.w_in[: m.rows]), mx.linear_f32(h, m.w_in[m.rows:])
    o = torch.empty(T, m.o.shape[1], device=dev, dtype=bf)
    ya, yr, (q, k, v, _) = y[:, : at.rows], y[:, at.rows:], y[:, : at.rows].split(at.parts, 1)
    where = {key: t for key, t in target["left"].items() if key != "pools"}
    kv = at.kv_heads * (at.dim + at.vdim)
    row("prompt preparation of attention", lambda: KM.attn_prep(ya, at, ctx.positions, None, table=at.rope.table(prompt, dev), **at.prep, **where),
        T * 2 * (2 * (at.heads + at.kv_heads) * at.dim + at.kv_heads * at.vdim + kv))
    row("prompt means of blocks", lambda: KM.pool_blocks(k, v, ctx.cu_seqlens, at.pool, **target["left"]["pools"]), T * kv * 2 * (1 + 2 / at.pool))
    blocks = KM.pool_blocks(k, v, ctx.cu_seqlens, at.pool)
    i = torch.arange(prompt, dtype=torch.float64)
    pairs = n_prompts * float((torch.clamp(i + 1, max=at.window) + torch.floor(torch.clamp(i + 1 - at.window, min=0) / at.pool)).sum())
    row("prompt windowed attention with blocks (sink)", lambda: KM.mixer_attn(q, k, v, heads=at.heads, kv_heads=at.kv_heads, scale=at.scale, **at.sight, pool=at.pool,
                                                                             blocks=blocks, ctx=ctx, out=o[:, : at.out_width], out_scale=0.9),
        T * 2 * (at.rows + at.out_width), 2 * pairs * at.heads * (at.dim + at.vdim))
    row("prompt hgrn2 (states + outputs + norm per head)", lambda: mx.hgrn2_rows(rg, yr, z, ctx, target["right"], out=o[:, at.out_width:], scale=0.7),
        T * rg.heads * (rg.dim * 6 + rg.vdim * 4) + n_prompts * rg.heads * rg.dim * rg.vdim * 4,
        2 * T * rg.heads * (2 * rg.dim * rg.vdim + 64 * (rg.dim + rg.vdim)))
    del y, z, o, ya, yr, q, k, v
    prompt_expert_kernels(moe, h, row)

    a = eng.slots[0]
    hb, xb, db = torch.randn(B, W, device=dev, dtype=bf), torch.randn(B, W, device=dev), torch.randn(B, W, device=dev)
    row("decode embedding + norm", lambda: KM.embed_normed(eng.next_input, model.embed_tokens, 1.0, model.embed_norm.weight, 1e-6, out=xb), B * W * 6)
    rows = eng.experts(hb, moe)
    row("decode experts' sum + residual + both norms", lambda: KM.rms_residual(xb, (db, rows), None, layer.norm1.weight, 1e-6, bf, clear=True, out=hb,
                                                                              w2=layer.norm2.weight, out2=eng._h2, mult=0.8), B * W * (20 + 2 * moe.top))
    hb = torch.randn(B, W, device=dev, dtype=bf)
    row("decode gemm input", lambda: K.decode_gemm(hb, m.w_in, y32=a.acc_in), m.w_in.numel() * 2)
    row("decode preparation of attention + cache", a.left.prepare, a.left.acc_in.numel() * 10)
    seen = min(prompt + 1, at.window) + max(0, prompt + 1 - at.window) // at.pool
    row("decode windowed attention with blocks (sink)", a.left.attend, B * seen * kv * 2 + 4 * a.left.q.numel(), 2 * B * seen * at.heads * (at.dim + at.vdim))
    row("decode hgrn2 step + norm", a.right.mix, a.right.state.numel() * 8 + B * sum(rg.parts) * 8 + a.right.y.numel() * 2)
    row("decode gemm output", lambda: K.decode_gemm(a.o, m.o, y32=eng._acc), m.o.numel() * 2)
    decode_expert_kernels(eng, moe, hb, db, row)


@torch.no_grad()
def zorelorn_kernels(s, model, eng, batch, prompt, n_prompts, row):
    from ..models.decoder import SeqCtx
    from ..ops import cuda as K
    from ..ops import cuda_mixers as KM
    from ..ops import mixers as mx

    la, ml = model.layers[0].mixer, model.layers[1].mixer
    T, W, dev, bf = n_prompts * prompt, s["width"], "cuda", torch.bfloat16
    ctx = SeqCtx.from_lengths([prompt] * n_prompts, dev)
    h = torch.randn(T, W, device=dev, dtype=bf)
    x, d = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
    nrm = model.norm
    row("prompt dynamic_tanh + residual", lambda: KM.dynamic_tanh(x, d, nrm.alpha, nrm.weight, nrm.bias, bf), T * W * 14)
    acc = mx.linear_f32(h, la.w_in)
    kr, lw = KM.latent_row(la.kv_rank, la.rot_dim)
    lat = torch.zeros(T, lw, device=dev, dtype=bf)
    table = la.rope.table(prompt, dev)
    row("prompt latent_prep", lambda: KM.latent_prep(acc, la, ctx.positions, table, lat=lat),
        T * (acc.shape[1] * 4 + (la.q_rank + lw) * 2 + la.heads * 4))
    cq, gate = KM.latent_prep(acc, la, ctx.positions, table, lat=lat)
    q, kv = mx.linear(cq, la.uq), mx.linear(lat[:, : la.kv_rank], la.ukv)
    row("prompt rotate_q", lambda: KM.rotate_q(q, la, ctx.positions, table), T * la.heads * la.rot_dim * 4)
    win = min(la.window or prompt, prompt)
    pairs = n_prompts * (win * (win + 1) / 2 + (prompt - win) * win)
    row("prompt latent attention", lambda: mx.latent_prompt_attention(q, kv, lat, la, ctx, gate),
        (q.numel() + kv.numel() + lat.numel() + T * la.heads * la.vdim) * 2,
        2 * pairs * la.heads * (la.dim + la.rot_dim + la.vdim))
    y = mx.linear(h, ml.w_in[: ml.gate_row])
    z = mx.linear_f32(h, ml.w_in[ml.gate_row:])
    ig, fg = KM.mlstm_gates(z, ml.gate_bias, ml.cap, ml.heads)
    row("prompt mlstm_gates", lambda: KM.mlstm_gates(z, ml.gate_bias, ml.cap, ml.heads), z.numel() * 8)
    qkv = ml.heads * (2 * ml.dim + ml.vdim)
    chunks = T // 128
    row("prompt mlstm chunk (scan + states + outputs)", lambda: KM.mlstm_chunk(y, ml, ig, fg, ctx.cu_seqlens),
        T * (qkv * 2 + ml.heads * ml.vdim * 4),
        2 * T * ml.heads * (2 * ml.dim * ml.vdim + 64 * (ml.dim + ml.vdim)))
    o32 = KM.mlstm_chunk(y, ml, ig, fg, ctx.cu_seqlens)
    yo = torch.empty(T, ml.heads * ml.vdim, device=dev, dtype=bf)
    row("prompt mlstm_out", lambda: KM.mlstm_out(o32, y[:, qkv:], ml, yo), o32.numel() * 8)
    up = torch.randn(T, s["ff"], device=dev, dtype=bf)
    row("prompt gelu", lambda: KM.gelu_erf(up), up.numel() * 4)
    del up, y, q, kv, o32

    paged_context(eng, prompt)
    a, r, B = eng.slots[0], eng.slots[1], batch
    hb = torch.randn(B, W, device=dev, dtype=bf)
    xb, db = torch.randn(B, W, device=dev), torch.randn(B, W, device=dev)
    row("decode dynamic_tanh + residual", lambda: KM.dynamic_tanh(xb, db, nrm.alpha, nrm.weight, nrm.bias, bf, clear=True, out=hb), B * W * 18)
    row("decode gemm input latent", lambda: K.decode_gemm(hb, la.w_in, y32=a.acc_in), la.w_in.numel() * 2)
    row("decode latent_prep", lambda: KM.latent_prep(a.acc_in, la, eng.seq_lens, a.table, clear=True, cq=a.cq, gate=a.gate,
                                                     cache=a.cache, block_table=eng.block_table, block_size=eng.block_size),
        B * la.w_in.shape[0] * 8)
    row("decode gemm query up", lambda: K.decode_gemm(a.cq, la.uq, y32=a.acc_q), la.uq.numel() * 2)
    row("decode absorb", a.absorb,
        la.uk.numel() * 2 + a.acc_q.numel() * 8 + a.q_lat.numel() * 2, 2 * B * la.heads * la.dim * la.kv_rank)
    n = min(prompt + 1, la.window or prompt + 1)
    row("decode latent attention", a.attend,
        B * n * lw * 2 + (a.q_lat.numel() + a.o_lat.numel()) * 2, 2 * B * n * la.heads * (lw + la.kv_rank))
    row("decode expand", a.expand, la.uv.numel() * 2 + (a.o_lat.numel() + a.o.numel()) * 2,
        2 * B * la.heads * la.vdim * la.kv_rank)
    row("decode gemm input mlstm", lambda: K.decode_gemm(hb, ml.w_in, y32=r.acc_in), ml.w_in.numel() * 2)
    row("decode mlstm_step", lambda: KM.mlstm_step(r.acc_in, ml, eng.seq_lens, r.state, r.o32),
        r.state[0].numel() * 8 + r.acc_in.numel() * 4 + r.o32.numel() * 4)
    row("decode mlstm_out", lambda: KM.mlstm_out(r.o32, r.acc_in[:, qkv:], ml, r.y, clear=r.acc_in), r.acc_in.numel() * 4 + r.o32.numel() * 8)
    mlp = model.layers[0].mlp
    row("decode up + gelu", lambda: eng.mlp_act(hb, mlp), mlp.up.numel() * 2)


def flat_kernels(s, batch, prompt, n_prompts, row):
    """The like kernels of the flat decoder, timed the same way."""
    from ..ops import cuda as K

    dev, bf, T, W = "cuda", torch.bfloat16, n_prompts * prompt, s["width"]
    Hq, Hk, D = W // 128, max(1, W // 512), 128
    q, k, v = (torch.randn(T, n, D, device=dev, dtype=bf) for n in (Hq, Hk, Hk))
    cu = torch.arange(0, T + 1, prompt, dtype=torch.int32, device=dev)
    pairs = n_prompts * prompt * (prompt + 1) / 2
    row("flat: prompt flash attention", lambda: K.fa_varlen_fwd(q, k, v, cu, cu), (2 * q.numel() + 2 * k.numel()) * 2, 4 * pairs * Hq * D)
    res, dl, w = (torch.randn(T, W, device=dev, dtype=bf), torch.randn(T, W, device=dev, dtype=bf), torch.ones(W, device=dev, dtype=bf))
    row("flat: prompt add + rmsnorm", lambda: K.add_rmsnorm_infer(res, dl, w, 1e-5), T * W * 8)
    gu = torch.randn(T, 2 * s["ff"], device=dev, dtype=bf)
    row("flat: prompt swiglu", lambda: K.swiglu_infer(gu), gu.numel() * 3)
    pages = batch * (prompt // 64 + 1)
    kc = torch.randn(pages, 64, Hk, D, device=dev, dtype=bf)
    vc = torch.randn(pages, Hk, D, 64, device=dev, dtype=bf)
    bt = torch.arange(pages, dtype=torch.int32, device=dev).view(batch, -1)
    sl = torch.full((batch,), prompt - 1, dtype=torch.int32, device=dev)
    splits = max(1, min(8, 148 // (batch * Hk)))
    po = torch.empty(batch * Hq * splits * D, device=dev)
    pm = torch.empty(batch * Hq * splits * 2, device=dev)
    qd, od = torch.randn(batch, Hq, D, device=dev, dtype=bf), torch.empty(batch, Hq, D, device=dev, dtype=bf)
    row("flat: decode attention", lambda: K.paged_decode_attn_tc(qd, kc, vc, sl, None, bt, D ** -0.5, splits, po, pm, od),
        batch * prompt * Hk * D * 4, 4 * batch * prompt * Hq * D)
    x, acc = torch.randn(batch, W, device=dev, dtype=bf), torch.zeros(batch, W, device=dev)
    row("flat: decode add + rmsnorm", lambda: K.add_rmsnorm_f32_infer(x, acc, w, 1e-5), batch * W * 14)
    qkv_w = torch.randn((Hq + 2 * Hk) * D, W, device=dev, dtype=bf)
    aq = torch.zeros(batch, qkv_w.shape[0], device=dev)
    row("flat: decode gemm qkv", lambda: K.decode_gemm(x, qkv_w, y32=aq), qkv_w.numel() * 2)
    row("flat: decode rope + kv write", lambda: K.rope_kv_write_f32(aq, None, None, None, 1e-5, sl, None, bt, 64, qd, kc, vc, Hq, Hk, D, 5e5,
                                                                    v_transposed=True), aq.numel() * 10)
    gw = torch.randn(2 * s["ff"], W, device=dev, dtype=bf)
    act = torch.empty(batch, s["ff"], device=dev, dtype=bf)
    row("flat: decode gate/up + swiglu", lambda: K.decode_gemm(x, gw, out=act, swiglu=True), gw.numel() * 2)
    if "experts" in s:
        flat_moe_kernels(s, batch, T, row)


def flat_moe_kernels(s, batch, T, row):
    from ..ops import cuda as K
    from ..ops import functional as F_

    dev, bf, W, n, E, top = "cuda", torch.bfloat16, s["width"], s["eff"], s["experts"], s["top"]
    router, gu, down = (torch.randn(*sh, device=dev, dtype=bf) * 0.02 for sh in ((E, W), (E, 2 * n, W), (E, W, n)))
    for name, rows in (("prompt", T), ("decode", batch)):
        R = rows * top
        h, xs, act = (torch.randn(r, c, device=dev, dtype=bf) for r, c in ((rows, W), (R, W), (R, n)))
        counts = torch.bincount(torch.randint(0, E, (R,), device=dev), minlength=E)
        offsets = torch.cat([counts.new_zeros(1), counts.cumsum(0)]).int()
        used = int((counts > 0).sum())
        row(f"flat: {name} experts gate/up + swiglu", lambda: K.grouped_gemm(xs, gu, offsets, n, swiglu=True), used * 4 * W * n + R * (W + n) * 2, 4 * R * W * n)
        row(f"flat: {name} experts down", lambda: K.grouped_gemm(act, down, offsets, W), used * 2 * W * n + R * (W + n) * 2, 2 * R * W * n)
        row(f"flat: {name} experts, all of it", lambda: F_.moe_mlp(h, router, gu, down, top, True), used * 6 * W * n + rows * W * 4, 6 * R * W * n)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", choices=sorted(SIZES), default="zorelorn")
    ap.add_argument("--sizes", default="small,base")
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--prompt", type=int, default=1024)
    ap.add_argument("--prompts", type=int, default=8)
    ap.add_argument("--kernels", action="store_true")
    a = ap.parse_args()
    if a.kernels:
        for r in kernel_table(a.sizes.split(",")[-1], a.batch, a.prompt, a.prompts, design=a.design):
            print(json.dumps(r))
        return
    for r in run(a.sizes.split(","), a.batch, a.prompt, a.prompts, a.design):
        print(json.dumps(r))


if __name__ == "__main__":
    main()
