"""Suposun on CPU: configuration, checkpoint names, the CPU path of every mechanism against the plain restatement, training,
generation through the eager generator and the server."""
import json
import math

import pytest
import torch

import suposun_reference as ref
import suposun_util as U
from trl_b200.models import SeqCtx, load_model, preset
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model
from trl_b200.models.layered import LayeredLM, RmsNormAboutZero, layered_kinds
from trl_b200.ops.mixers import RotarySpec
from trl_b200.oracle import mixers as om
from trl_b200.rollout.engine import EagerGenerator
from trl_b200.rollout.sampling import SamplingParams

f64 = torch.float64


@pytest.mark.parametrize("dims,base,scaling", [(2, 10.0, None), (24, 3e3, None), (32, 1e5, U.yarn(4.0, 300, 32.0, 1.0)), (14, 1e3, U.yarn()),
                                               (8, 50.0, U.yarn(1.0, 40, 2.0, 0.1)), (64, 1e6, U.yarn(16.0, 4096, 32.0, 1.0))])
@pytest.mark.parametrize("halves", [False, True])
def test_rotation(dims, base, scaling, halves):
    t = RotarySpec(dims, base, scaling).table(3000, "cpu").double()
    x = torch.randn(4, 3, dims, dtype=f64)
    for p in (0, 1, 77, 2999):
        turn = om.rotate_halves if halves else om.rotate_pairs
        got = turn(x, t[p, :, 0].expand(4, -1), t[p, :, 1].expand(4, -1))
        want = ref.rotate(x, p, dict(dims=dims, base=base, scaling=scaling), halves)
        assert torch.allclose(got, want, atol=1e-6)
    if scaling:
        assert ref.frequencies(dims, base, scaling)[1] == pytest.approx(0.1 * math.log(scaling["factor"]) + 1)


def test_visible_tokens():
    """The edges of the window and of the kept tokens, spelled out."""
    m = dict(size=3, keep_first=2)
    assert ref.visible(0, m) == [0] and ref.visible(4, m) == [0, 1, 2, 3, 4] and ref.visible(5, m) == [0, 1, 3, 4, 5]
    assert ref.visible(9, m) == [0, 1, 7, 8, 9] and ref.visible(9, dict(size=1)) == [9] and ref.visible(3) == [0, 1, 2, 3]


@pytest.mark.parametrize("H,G", [(6, 3), (4, 4), (5, 1)])
@pytest.mark.parametrize("cap", [None, 1.5])
@pytest.mark.parametrize("mask", [None, dict(size=4), dict(size=1, keep_first=3), dict(size=3, keep_first=1), dict(size=50, keep_first=60)])
def test_attention_mask_cap_and_sink(H, G, cap, mask):
    q, k, v = (torch.randn(17, n, d, dtype=f64) * 2 for n, d in ((H, 6), (G, 6), (G, 4)))
    for sink in (None, torch.randn(H, dtype=f64) + 1):
        got = om.sink_window_attention(q, k, v, 0.4, (mask or {}).get("size"), sink, torch.tensor([0, 5, 17]), cap, (mask or {}).get("keep_first", 0))
        for a, b in ((0, 5), (5, 17)):
            assert torch.allclose(got[a:b], ref.attend(q[a:b], k[a:b], v[a:b], 0.4, cap, mask, sink))


def test_the_sink_counts_once_and_unscaled():
    """One key of score zero beside a sink of logarithm three: a quarter of the value comes out."""
    q, k, v = torch.zeros(1, 1, 4, dtype=f64), torch.randn(1, 1, 4, dtype=f64), torch.randn(1, 1, 4, dtype=f64)
    sink = torch.tensor([math.log(3.0)], dtype=f64)
    for f in (lambda: om.sink_window_attention(q, k, v, 7.0, None, sink, torch.tensor([0, 1]), 0.5), lambda: ref.attend(q, k, v, 7.0, 0.5, None, sink)):
        assert torch.allclose(f(), v / 4)


@pytest.mark.parametrize("spec", [dict(mul_prev=29, mul_cur=11, buckets=101), dict(mul_prev=1, mul_cur=1, buckets=1), dict(mul_prev=0, mul_cur=5, buckets=7),
                                  dict(mul_prev=99991, mul_cur=65537, buckets=100003)])
def test_pair_rows(spec):
    ids = torch.tensor([5, 9, 9, 0, 12, 60000])
    pos = torch.tensor([0, 1, 2, 0, 1, 2])
    got = om.pair_rows(ids, pos, **spec).tolist()
    prev = [None, 5, 9, None, 0, 12]
    assert got == [ref.bigram_row(p, int(c), **spec) for p, c in zip(prev, ids)]


@pytest.mark.parametrize("E,top", [(1, 1), (5, 5), (9, 1), (16, 3)])
def test_routing_and_experts(E, top):
    z, c = torch.randn(20, E, dtype=f64) * 2, torch.randn(E, dtype=f64)
    idx, w = om.route(z, c, top)
    for t in range(20):
        want = ref.route(z[t], torch.eye(E, dtype=f64), c, top)
        assert idx[t].tolist() == [e for e, _ in want] and torch.allclose(w[t], torch.stack([s for _, s in want]))
    # a correction decides who is chosen and leaves the weights alone
    c = torch.zeros(E, dtype=f64)
    c[E - 1] = 10.0
    idx, w = om.route(z, c, 1)
    assert (idx == E - 1).all() and torch.allclose(w[:, 0], torch.sigmoid(z[:, E - 1]))


def test_units_and_norms():
    h, g, u, d = torch.randn(9, 5, dtype=f64) * 3, torch.randn(7, 5, dtype=f64), torch.randn(7, 5, dtype=f64), torch.randn(5, 7, dtype=f64)
    assert torch.allclose(om.gelu_glu(h @ torch.cat([g, u]).T) @ d.T, ref.dense_mlp(h, dict(gate=g, up=u, down=d)))
    assert torch.allclose(om.clamped_glu(h @ torch.cat([g, u]).T, 0.9, 1.702, 1.0) @ d.T, ref.expert(h, g, u, d, 0.9))
    x, w, p, s = torch.randn(9, 5, dtype=f64), torch.randn(5, dtype=f64), torch.randn(5, dtype=f64), torch.randn(5, dtype=f64)
    y, r = om.rms_residual(x, h, p, w, 1e-3, shift=1.0, post_scale=s, gain=0.3)
    assert torch.allclose(r, x + ref.norm_about_zero(h, p, 1e-3) * s) and torch.allclose(y, ref.norm_about_zero(r, w, 1e-3) * 0.3)


@pytest.mark.parametrize("cfg", [U.ODD, U.TILES, U.ONES, U.PLAIN])
def test_model_matches_restatement(cfg):
    m, t = U.make(cfg)
    a, b = U.tokens(31, cfg["vocab"], 1), U.tokens(44, cfg["vocab"], 2)
    got = m(torch.tensor([a + b]), position_ids=torch.tensor([list(range(31)) + list(range(44))])).logits[0]
    assert U.rel(got[:31], U.logits(cfg, t, a)) < 2e-5
    assert U.rel(got[31:], U.logits(cfg, t, b)) < 2e-5


def test_residual_stream_after_every_layer():
    """The stream with its pending addition, layer by layer, against the restatement."""
    m, t = U.make(U.ODD)
    toks, want = U.tokens(17, 193, 5), []
    ref.forward(U.ODD, t, toks, want)
    ctx = SeqCtx.from_lengths([17], "cpu")
    ctx.shared = dict.fromkeys(m.config.lenders)
    ids = torch.tensor(toks)
    x, delta, post = m.embed(ids, ctx), None, None
    for li, layer in enumerate(m.layers):
        x, delta, post = layer(x, delta, post, ctx, li, ids)
        assert isinstance(post, RmsNormAboutZero)
        s = post.stream(x, torch.float32, delta, post)[1]
        assert torch.allclose(s.double(), want[li], atol=2e-4), li


def test_borrowing_layers():
    m, _ = U.make(U.ODD)
    names = set(m.named_tensors())
    assert m.config.lenders == {1} and {"l3.mix.q", "l3.mix.q.norm", "l1.mix.k.norm"} <= names
    assert not {"l3.mix.k", "l3.mix.v", "l5.mix.k.norm", "l0.mix.v", "l1.mix.g", "l1.mix.sink", "head"} & names
    toks = torch.tensor([U.tokens(9, 193)])
    before = m(toks).logits
    with torch.no_grad():  # the lender's values change, nothing of the borrowers does
        m.layers[1].mixer.w_in[72:] *= -1
        m.layers[1].mixer.o.zero_()
    first = m(toks).logits
    with torch.no_grad():
        m.layers[1].mixer.w_in[72:] *= -1
    assert not torch.allclose(m(toks).logits, first) and not torch.allclose(before, first)


def test_checkpoint_round_trip(tmp_path):
    m, t = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path))
    d = json.load(open(tmp_path / "config.json"))
    assert d["layers"][3]["mixer"]["kv_from"] == 1 and d["embedding"]["bigram"]["buckets"] == 97 and d["logit_scale"] == 0.7
    assert layered_kinds(str(tmp_path)) == {"attention", "attention_2", "moe"}
    again = load_model(str(tmp_path), dtype=torch.bfloat16)
    assert isinstance(again, LayeredLM) and again.config.num_hidden_layers == 8
    for name, x in again.named_tensors().items():
        assert torch.equal(x.double(), t[name]), name
    from safetensors.torch import load_file

    sd = load_file(str(tmp_path / "model.safetensors"))
    assert sd["l0.mlp.e6.gate"].shape == (17, 76) and sd["l0.mix.g"].shape == (6, 76) and sd["bigram"].shape == (98, 76)
    assert sd["l1.mix.q.norm"].shape == (48,) and sd["l0.mix.q.norm"].shape == (20,) and "l7.norm2" not in sd
    del sd["l1.ls1"]
    with pytest.raises(KeyError, match="l1.ls1"):
        again.load_named_tensors(sd)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "same kind"), (lambda c: c["layers"][5]["mixer"].update(kv_from=3), "of its own"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=27), "vdim differs"), (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "not supported"),
    (lambda c: c["layers"][0].update(type="nothing"), "not registered")])
def test_config_errors(change, message):
    bad = json.loads(json.dumps(U.ODD))
    change(bad)
    with pytest.raises(ValueError, match=message):
        ModelArch.from_hf_dict(bad)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "have its size|have their size"), (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "rotated"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key/value heads")])
def test_model_errors(change, message):
    bad = json.loads(json.dumps(U.ODD))
    change(bad)
    with pytest.raises(ValueError, match=message):
        build_model(ModelArch.from_hf_dict(bad))


def test_other_designs_have_no_experts():
    with pytest.raises(ValueError, match="not supported"):
        ModelArch.from_hf_dict(dict(architecture="Povusun", vocab=9, width=8, norm=dict(eps=1e-5),
                                    layers=[dict(type="rglru", mixer=dict(width=8, blocks=1, conv=2), mlp=U.moe(8, 2, 1))]))


def test_preset_trains_on_cpu():
    m = build_model(preset("tiny-suposun"))
    ids = torch.randint(0, 1024, (2, 40))
    loss = m(ids, labels=ids).loss
    loss.backward()
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for n, p in m.named_parameters() if not n.endswith("correction"))
    assert m.config.num_parameters() == sum(p.numel() for p in m.parameters())
    m.resize_token_embeddings(1030)
    assert m.lm_head_weight.shape[0] == 1030 and m(ids + 6).logits.shape[-1] == 1030


def test_greedy_generation():
    m, t = U.make(U.ODD)
    prompts = [U.tokens(6, 193, 3), U.tokens(19, 193, 4)]
    outs = EagerGenerator(m).generate(prompts, SamplingParams(max_tokens=6, greedy=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(6):
            seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
        assert o.token_ids == seq[len(p):]


def test_server_serves_a_checkpoint(tmp_path):
    from trl_b200.scripts.rollout_serve import ServeArguments, WorkerPool

    m, t = U.make(U.PLAIN)
    m.save_pretrained(str(tmp_path))
    pool = WorkerPool(ServeArguments(model=str(tmp_path), max_model_len=64))
    try:
        prompt = U.tokens(7, 193, 9)
        out = pool.generate([prompt], {"max_tokens": 3, "generation_kwargs": {"greedy": True}})
        seq = list(prompt)
        for _ in range(3):
            seq.append(int(U.logits(U.PLAIN, t, seq)[-1].argmax()))
        assert out[0][1] == seq[7:]
    finally:
        pool.close()
