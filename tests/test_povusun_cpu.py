"""Povusun on CPU: configuration, checkpoint names, the CPU path of every mechanism against the plain restatement, training,
generation through the eager generator and the server."""
import json

import pytest
import torch

import povusun_reference as ref
import povusun_util as U
from trl_b200.models import SeqCtx, load_model, preset
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model
from trl_b200.models.layered import LayeredLM
from trl_b200.ops.mixers import TemperatureSpec
from trl_b200.oracle import mixers as om
from trl_b200.rollout.engine import EagerGenerator
from trl_b200.rollout.sampling import SamplingParams

f64 = torch.float64


@pytest.mark.parametrize("coef,every", [(0.3, 5), (1.7, 1), (0.0, 9), (0.25, 1000)])
def test_temperature_table(coef, every):
    t = TemperatureSpec(coef, every).table(2100, "cpu")
    for p in (0, 1, every - 2, every - 1, every, 2 * every - 2, 2 * every - 1, 999, 2099):
        if 0 <= p < 2100:
            assert float(t[p]) == pytest.approx(ref.temperature(p, coef, every), rel=1e-7)
    assert float(t[0]) == 1.0 or every == 1


@pytest.mark.parametrize("H,G", [(6, 3), (4, 4), (5, 1)])
@pytest.mark.parametrize("cap", [None, 1.5])
def test_grouped_attention(H, G, cap):
    q, k, v = (torch.randn(12, n, d, dtype=f64) * 2 for n, d in ((H, 6), (G, 6), (G, 4)))
    got = om.sink_window_attention(q, k, v, 0.4, None, None, torch.tensor([0, 5, 12]), cap)
    for a, b in ((0, 5), (5, 12)):
        assert torch.allclose(got[a:b], ref.grouped_attention(q[a:b], k[a:b], v[a:b], 0.4, cap))


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution(taps):
    x, w, b = torch.randn(11, 3, dtype=f64), torch.randn(3, taps, dtype=f64), torch.randn(3, dtype=f64)
    got = om.causal_conv(x, w, b, torch.tensor([0, 2, 11]))
    for i, j in ((0, 2), (2, 11)):
        assert torch.allclose(got[i:j], ref.causal_conv(x[i:j], w, b))


def test_recurrence():
    T, C = 37, 4
    u, r, i, lam = torch.randn(T, C, dtype=f64), torch.rand(T, C, dtype=f64), torch.rand(T, C, dtype=f64), torch.tensor([-9.0, -2.0, 0.0, 3.0], dtype=f64)
    log_a = -8 * r * torch.nn.functional.softplus(lam)
    got = om.linear_recurrence(log_a.exp(), torch.sqrt(-torch.expm1(2 * log_a)) * i * u, torch.tensor([0, 1, 18, T]))
    for a, b in ((0, 1), (1, 18), (18, T)):
        assert torch.allclose(got[a:b], ref.rglru_recurrence(u[a:b], r[a:b], i[a:b], lam))


def test_clamped_unit_and_norms():
    h, g, u, d = torch.randn(9, 5, dtype=f64) * 3, torch.randn(7, 5, dtype=f64), torch.randn(7, 5, dtype=f64), torch.randn(5, 7, dtype=f64)
    got = om.clamped_glu(h @ torch.cat([g, u]).T, 1.3, 1.702, 1.0) @ d.T
    assert torch.allclose(got, ref.clamped_glu(h, g, u, d, 1.3))
    x, w, p = torch.randn(9, 5, dtype=f64), torch.randn(5, dtype=f64), torch.randn(5, dtype=f64)
    y, s = om.rms_residual(x, h, p, w, 1e-3)
    assert torch.allclose(s, x + ref.rms_norm(h, p, 1e-3)) and torch.allclose(y, ref.rms_norm(s, w, 1e-3))
    assert torch.equal(om.rms_residual(x, None, None, None, 1e-3)[0], x)


@pytest.mark.parametrize("cfg", [U.ODD, U.TILES, U.ONES])
def test_model_matches_restatement(cfg):
    m, t = U.make(cfg)
    a, b = U.tokens(31, cfg["vocab"], 1), U.tokens(44, cfg["vocab"], 2)
    got = m(torch.tensor([a + b]), position_ids=torch.tensor([list(range(31)) + list(range(44))])).logits[0]
    assert U.rel(got[:31], U.logits(cfg, t, a)) < 2e-5
    assert U.rel(got[31:], U.logits(cfg, t, b)) < 2e-5


def test_residual_stream_after_every_layer():
    """The stream with its pending addition, layer by layer, against the restatement."""
    m, t = U.make(U.ODD)
    toks, want = U.tokens(17, 197, 5), []
    ref.forward(U.ODD, t, toks, want)
    ctx = SeqCtx.from_lengths([17], "cpu")
    ctx.shared = dict.fromkeys(m.config.lenders)
    ids = torch.tensor(toks)
    x, delta, post = m.embed(ids), None, None
    for li, layer in enumerate(m.layers):
        x, delta, post = layer(x, delta, post, ctx, li, ids, m.side_embed)
        s = om.rms_residual(x, delta, None if post is None else post.weight, None, 1e-5)[1]
        assert torch.allclose(s.double(), want[li], atol=2e-4), li


def test_borrowing_layers():
    m, _ = U.make(U.ODD)
    names = set(m.named_tensors())
    assert m.config.lenders == {1} and "l3.mix.q" in names and not {"l3.mix.k", "l3.mix.v", "l6.mix.k", "head"} & names
    assert m.lm_head is None and m.lm_head_weight is m.embed_tokens
    # a change of the lender's keys reaches the borrower
    toks = torch.tensor([U.tokens(9, 197)])
    before = m(toks).logits
    kept = m.layers[3].mixer.w_in.clone()
    with torch.no_grad():
        m.layers[1].mixer.w_in[120:180] *= -1
    assert torch.equal(m.layers[3].mixer.w_in, kept) and not torch.allclose(m(toks).logits, before)


def test_checkpoint_round_trip(tmp_path):
    m, t = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json"))["layers"][3]["mixer"]["kv_from"] == 1
    again = load_model(str(tmp_path), dtype=torch.bfloat16)
    assert isinstance(again, LayeredLM) and again.config.num_hidden_layers == 9
    for name, x in again.named_tensors().items():
        assert torch.equal(x.double(), t[name]), name
    from safetensors.torch import load_file

    sd = load_file(str(tmp_path / "model.safetensors"))
    assert sd["l0.mix.ra"].shape == (4, 15, 15) and sd["l0.mix.ra.b"].shape == (4, 15) and sd["l0.mix.conv"].shape == (60, 3)
    del sd["l1.norm1b"]
    with pytest.raises(KeyError, match="l1.norm1b"):
        again.load_named_tensors(sd)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][3]["mixer"].update(kv_from=4), "kv_from"), (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "same kind"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=3), "of its own"), (lambda c: c["layers"][3]["mixer"].update(vdim=27), "vdim differs"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "not supported"), (lambda c: c["layers"][0].update(type="nothing"), "not registered")])
def test_config_errors(change, message):
    bad = json.loads(json.dumps(U.ODD))
    change(bad)
    with pytest.raises(ValueError, match=message):
        ModelArch.from_hf_dict(bad)


def test_preset_trains_on_cpu():
    m = build_model(preset("tiny-povusun"))
    ids = torch.randint(0, 1024, (2, 24))
    loss = m(ids, labels=ids).loss
    loss.backward()
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for p in m.parameters())
    assert m.config.num_parameters() == sum(p.numel() for p in m.parameters())
    m.resize_token_embeddings(1030)
    assert m.side_embed.shape[0] == m.lm_head_weight.shape[0] == 1030
    assert m(ids + 6).logits.shape[-1] == 1030


def test_greedy_generation():
    m, t = U.make(U.ODD)
    prompts = [U.tokens(6, 197, 3), U.tokens(19, 197, 4)]
    outs = EagerGenerator(m).generate(prompts, SamplingParams(max_tokens=6, greedy=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(6):
            seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
        assert o.token_ids == seq[len(p):]


def test_server_serves_a_checkpoint(tmp_path):
    from trl_b200.scripts.rollout_serve import ServeArguments, WorkerPool

    m, t = U.make(U.ONES)
    m.save_pretrained(str(tmp_path))
    pool = WorkerPool(ServeArguments(model=str(tmp_path), max_model_len=64))
    try:
        prompt = U.tokens(7, 13, 9)
        out = pool.generate([prompt], {"max_tokens": 3, "generation_kwargs": {"greedy": True}})
        seq = list(prompt)
        for _ in range(3):
            seq.append(int(U.logits(U.ONES, t, seq)[-1].argmax()))
        assert out[0][1] == seq[7:]
    finally:
        pool.close()
