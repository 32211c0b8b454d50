"""Gerupel on CPU: configuration, checkpoint names, the CPU path of every mechanism against the plain restatement, training,
generation through the eager generator and the server."""
import json
import math

import pytest
import torch

import gerupel_reference as ref
import gerupel_util as U
from trl_b200.models import SeqCtx, load_model, preset
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model
from trl_b200.models.layered import LayeredLM, RmsNorm, layered_kinds
from trl_b200.ops import mixers as mx
from trl_b200.oracle import mixers as om
from trl_b200.rollout.engine import EagerGenerator
from trl_b200.rollout.sampling import SamplingParams

f64 = torch.float64


@pytest.mark.parametrize("dims,base,scaling", [(2, 10.0, None), (24, 3e3, None), (32, 1e5, U.llama3(8.0, 1.0, 4.0, 2000)), (14, 1e3, U.llama3()), (8, 50.0, U.llama3(1.0)),
                                               (64, 1e6, U.llama3(16.0, 1.0, 4.0, 8192)), (16, 100.0, U.llama3(4.0, 1.0, 2.0, 5000)), (16, 1e7, U.llama3(4.0, 30.0, 40.0, 20))])
def test_rotation(dims, base, scaling):
    t = mx.RotarySpec(dims, base, scaling).table(3000, "cpu").double()
    x = torch.randn(4, 3, dims + 3, dtype=f64)
    for p in (0, 1, 77, 2999):
        got = torch.cat([om.rotate_halves(x[..., :dims], t[p, :, 0].expand(4, -1), t[p, :, 1].expand(4, -1)), x[..., dims:]], -1)
        assert torch.allclose(got, ref.rotate(x, p, dict(dims=dims, base=base, scaling=scaling)), atol=1e-6)


def test_frequency_scaling():
    """Short wavelengths stay, long ones are slowed down by the whole factor, one half-way by the mean of both."""
    s = U.llama3(8.0, 1.0, 3.0, 200)
    base = 10000.0
    f, g = ref.frequencies(64, base), ref.frequencies(64, base, s)
    turns = [200 * x / (2 * math.pi) for x in f]
    assert any(t > 3 for t in turns) and any(1 < t < 3 for t in turns) and any(t < 1 for t in turns)
    for a, b, t in zip(f, g, turns):
        share = min(max((t - 1) / 2, 0), 1)
        assert b == pytest.approx(share * a + (1 - share) * a / 8)
    assert torch.allclose(mx.RotarySpec(64, base, s).frequencies(), torch.tensor(g, dtype=f64))


def test_sight():
    """The edges of the window and of the blocks, spelled out: tokens that left the window wait for their block to be complete
    outside of it."""
    m = dict(size=3, pool=2)
    assert ref.sight(0, m) == ([0], []) and ref.sight(2, m) == ([0, 1, 2], []) and ref.sight(3, m) == ([1, 2, 3], [])
    assert ref.sight(4, m) == ([2, 3, 4], [0]) and ref.sight(5, m) == ([3, 4, 5], [0]) and ref.sight(6, m) == ([4, 5, 6], [0, 1])
    assert ref.sight(2, dict(size=1, pool=1)) == ([2], [0, 1]) and ref.sight(9, dict(size=1, pool=20)) == ([9], [])
    assert ref.sight(3) == ([0, 1, 2, 3], []) and ref.sight(3, dict(size=2)) == ([2, 3], [])


@pytest.mark.parametrize("H,G", [(6, 3), (4, 4), (5, 1)])
@pytest.mark.parametrize("mask", [None, dict(size=4, pool=2), dict(size=1, pool=1), dict(size=3, pool=5), dict(size=2, pool=3), dict(size=50, pool=2)])
def test_attention_over_window_and_blocks(H, G, mask):
    q, k, v = (torch.randn(26, n, d, dtype=f64) * 2 for n, d in ((H, 6), (G, 6), (G, 4)))
    temp = torch.randn(H, dtype=f64) + 1
    m = mask or {}
    got = om.sink_window_attention(q * temp[:, None], k, v, 0.4, m.get("size"), torch.zeros(H), torch.tensor([0, 5, 26]), pool=m.get("pool", 0))
    for a, b in ((0, 5), (5, 26)):
        for t in range(b - a):
            assert torch.allclose(got[a + t], ref.attend_one(q[a + t], k[a:b], v[a:b], 0.4, temp, mask, t)), t


def test_one_in_the_denominator():
    """One key of score zero: half of its value comes out; of score log 3: three quarters."""
    q, k, v = torch.ones(1, 4, dtype=f64), torch.zeros(1, 1, 4, dtype=f64), torch.randn(1, 1, 4, dtype=f64)
    for key, share in ((0.0, 0.5), (math.log(3.0), 0.75)):
        k[0, 0, 0] = key
        assert torch.allclose(ref.attend_one(q, k, v, 1.0, torch.ones(1), None, 0), v[0] * share)
        assert torch.allclose(om.sink_window_attention(q[None], k, v, 1.0, None, torch.zeros(1), torch.tensor([0, 1]))[0], v[0] * share)


def test_recurrence():
    q, f, v = torch.randn(19, 3, 5, dtype=f64), torch.rand(19, 3, 5, dtype=f64), torch.randn(19, 3, 4, dtype=f64)
    f[4] = 0.0  # everything is replaced
    f[9] = 1.0  # nothing is written
    got = om.hgrn2_scan(q, f, v, torch.tensor([0, 7, 19]))
    assert torch.allclose(got[:7], ref.recurrence(q[:7], f[:7], v[:7])[0]) and torch.allclose(got[7:], ref.recurrence(q[7:], f[7:], v[7:])[0])
    assert torch.allclose(ref.recurrence(q[:5], f[:5], v[:5])[0][4], q[4].sum(-1, keepdim=True) * v[4])
    # closed form: what token j wrote has been multiplied by all later gates
    want = sum((q[6] * (1 - f[j]) * f[j + 1:7].prod(0)).sum(-1, keepdim=True) * v[j] for j in range(7))
    assert torch.allclose(got[6], want)


def test_forget_gate_bounds():
    z, low = torch.tensor([-50.0, 0.0, 50.0], dtype=f64), torch.tensor([0.25], dtype=f64)
    assert torch.allclose(ref.forget(z, low), torch.tensor([0.25, 0.625, 1.0], dtype=f64))


@pytest.mark.parametrize("E,top", [(1, 1), (5, 5), (9, 1), (16, 3)])
def test_routing(E, top):
    z = torch.randn(20, E, dtype=f64) * 2
    idx, w = om.route(z, None, top, True, "softmax", 2.5)
    for t in range(20):
        want = ref.route(z[t], top, 2.5)
        assert idx[t].tolist() == [e for e, _ in want] and torch.allclose(w[t], torch.stack([s for _, s in want]))
    assert torch.allclose(w.sum(-1), torch.full((20,), 2.5, dtype=f64))


def test_norms_around_the_stream():
    x, a, b, first, w, w2, step = (torch.randn(*s, dtype=f64) for s in ((9, 5), (9, 5), (9, 5), (9, 5), (5,), (5,), (5,)))
    (y, y2), r = om.rms_residual(x, (a, b), None, w, 1e-3, mult=0.3, anchor=first, bump=step, w2=w2)
    want = x + 0.3 * (a + b) + first + step
    assert torch.allclose(r, want) and torch.allclose(y, ref.norm(want, w, 1e-3)) and torch.allclose(y2, ref.norm(want, w2, 1e-3))
    y, r = om.rms_residual(x, None, None, w, 1e-3, bump=step)
    assert torch.allclose(r, x + step) and torch.allclose(y, ref.norm(x + step, w, 1e-3))


@pytest.mark.parametrize("cfg", [U.ODD, U.TILES, U.ONES, U.PLAIN])
def test_model_matches_restatement(cfg):
    m, t = U.make(cfg)
    a, b = U.tokens(31, cfg["vocab"], 1), U.tokens(60, cfg["vocab"], 2)
    got = m(torch.tensor([a + b]), position_ids=torch.tensor([list(range(31)) + list(range(60))])).logits[0]
    assert U.rel(got[:31], U.logits(cfg, t, a)) < 3e-5
    assert U.rel(got[31:], U.logits(cfg, t, b)) < 3e-5


def test_residual_stream_after_every_layer_run():
    """The stream with its pending additions, run by run, against the restatement."""
    m, t = U.make(U.ODD)
    toks, want = U.tokens(17, 193, 5), []
    ref.forward(U.ODD, t, toks, want)
    assert len(want) == m.config.num_hidden_layers == len(m.layers) == 8
    ctx = SeqCtx.from_lengths([17], "cpu")
    ctx.shared = {}
    ids = torch.tensor(toks)
    x, delta, post = m.embed(ids), None, None
    first = x.clone()
    for li, layer in enumerate(m.layers):
        x, delta, post = layer(x, delta, post, ctx, li, ids, enter=m.entrance(li, first))
        s = RmsNorm.stream(x, torch.float32, delta, post, mult=layer.mult)[1]
        assert torch.allclose(s.double(), want[li], atol=2e-4), li


def test_loops():
    """Order of the runs, what enters them, and whose tensors they use."""
    c = ModelArch.from_hf_dict(U.ODD)
    assert [s.index for s in c.layers] == [0, 1, 2, 1, 2, 1, 2, 3] and [s.enters for s in c.layers] == [None, 0, None, 1, None, 2, None, None]
    m = build_model(c)
    assert m.layers[3] is m.layers[1] and m.layers[6] is m.layers[2] and m.layers[7] is not m.layers[0]
    names = set(m.named_tensors())
    assert {"l3.mix.right.norm", "l2.mlp.e4.down", "loop.step", "embed.norm"} <= names and not any(n.startswith(("l4.", "l7.")) for n in names)
    assert m.loop_step.shape == (3, 76) and not {"l1.norm2", "l1.mlp.router", "head", "l0.mix.left.sink"} & names
    first = torch.zeros(1, 76)
    assert m.entrance(0, first) == {} and m.entrance(1, first)["anchor"] is None and m.entrance(3, first)["anchor"] is first
    assert torch.equal(m.entrance(5, first)["bump"], m.loop_step[2])
    # a loop of one pass adds its step all the same
    one, t = U.make(U.ONES)
    toks = torch.tensor([[1, 5, 3]])
    before = one(toks).logits
    one.loop_step.data += 1.0
    assert not torch.allclose(one(toks).logits, before)


def test_checkpoint_round_trip(tmp_path):
    m, t = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path))
    d = json.load(open(tmp_path / "config.json"))
    assert len(d["layers"]) == 4 and d["loop"] == dict(start=1, stop=3, times=3) and d["layers"][0]["mixer"]["left"]["mask"] == dict(size=7, pool=3)
    assert layered_kinds(str(tmp_path)) == {"parallel", "attention", "hgrn2", "moe"}
    again = load_model(str(tmp_path), dtype=torch.bfloat16)
    assert isinstance(again, LayeredLM) and again.config.num_hidden_layers == 8
    for name, x in again.named_tensors().items():
        assert torch.equal(x.double(), t[name]), name
    from safetensors.torch import load_file

    sd = load_file(str(tmp_path / "model.safetensors"))
    assert set(sd) == set(t)
    assert sd["l0.mlp.e6.gate"].shape == (17, 76) and sd["l0.mix.left.o"].shape == (76, 168) and sd["l0.mix.right.o"].shape == (76, 30)
    assert sd["l1.mix.right.f"].shape == (5, 76) and sd["l1.mix.right.norm"].shape == (33,) and sd["l2.mix.left.temp"].shape == (4,)
    del sd["l1.mix.right.lower"]
    with pytest.raises(KeyError, match="l1.mix.right.lower"):
        again.load_named_tensors(sd)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["loop"].update(stop=5), "loop over layers"), (lambda c: c["loop"].update(times=0), "loop over layers"), (lambda c: c["loop"].update(start=3), "loop over layers"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "not supported"), (lambda c: c["layers"][0].update(type="nothing"), "not registered")])
def test_config_errors(change, message):
    bad = json.loads(json.dumps(U.ODD))
    change(bad)
    with pytest.raises(ValueError, match=message):
        ModelArch.from_hf_dict(bad)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=22), "rotated"), (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"), (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=1), "pooled")])
def test_model_errors(change, message):
    bad = json.loads(json.dumps(U.ODD))
    change(bad)
    with pytest.raises(ValueError, match=message):
        build_model(ModelArch.from_hf_dict(bad))


def test_mixers_serve_other_designs():
    """The recurrent mixer alone, in a design with norms around its sublayers, against its restatement."""
    cfg = dict(architecture="Povusun", vocab=50, width=24, norm=dict(eps=1e-4), layers=[dict(type="hgrn2", mixer=dict(heads=2, dim=6, vdim=10), mlp=None)])
    m = build_model(ModelArch.from_hf_dict(cfg)).double()
    mixer, h = m.layers[0].mixer, torch.randn(9, 24)
    for p in mixer.parameters():
        p.data.normal_()
    w = {k[3:]: t.detach().double() for k, t in mixer.tensors("xx.").items()}
    w["lower"] = mixer.lower.data.copy_(mixer.lower.data.sigmoid()).double()
    got = mixer(h, SeqCtx.from_lengths([9], "cpu"), 0)
    assert torch.allclose(got.double(), ref.linear_attention(h.double(), w, dict(heads=2, dim=6, vdim=10), 1e-4), atol=1e-4)


def test_preset_trains_on_cpu():
    m = build_model(preset("tiny-gerupel"))
    ids = torch.randint(0, 1024, (2, 40))
    loss = m(ids, labels=ids).loss
    loss.backward()
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for p in m.parameters())
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
