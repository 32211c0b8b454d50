"""Zorelorn on CPU: configuration, checkpoint names, the CPU path of every mechanism against the plain restatement,
generation through the eager generator, and the scheduler's growing sequences."""
import json
import math

import numpy as np
import pytest
import torch

import zorelorn_reference as ref
import zorelorn_util as U
from trl_b200.models import SeqCtx, load_model, preset
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model
from trl_b200.models.layered import LayeredLM
from trl_b200.ops.mixers import RotarySpec
from trl_b200.oracle import mixers as om
from trl_b200.rollout.engine import EagerGenerator
from trl_b200.rollout.sampling import SamplingParams


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 5000.0, None), (64, 7e5, dict(factor=5.0, original=2048, fast=24.0, slow=2.0)),
    (2, 100.0, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)), (32, 1e4, dict(factor=1.0, original=64, fast=4.0, slow=4.0)),
    (48, 2e5, dict(factor=40.0, original=100000, fast=64.0, slow=0.25))])
def test_rotary_table(dims, base, scaling):
    spec = RotarySpec(dims, base, scaling)
    f, mag = ref.yarn_frequencies(dims, base, scaling)
    assert torch.allclose(spec.frequencies(), torch.tensor(f, dtype=torch.float64), rtol=1e-12)
    assert spec.magnitude == pytest.approx(mag)
    t = spec.table(700, "cpu")
    for p in (0, 1, 255, 256, 699):
        for i in range(dims // 2):
            assert float(t[p, i, 0]) == pytest.approx(mag * math.cos(p * f[i]), abs=1e-6)
            assert float(t[p, i, 1]) == pytest.approx(mag * math.sin(p * f[i]), abs=1e-6)


def test_rotation_pairs_neighbours():
    x = torch.randn(5, 3, 8, dtype=torch.float64)
    f = [0.7, 0.2, 0.05, 0.01]
    ang = torch.arange(5, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    got = om.rotate_pairs(x, ang.cos() * 1.3, ang.sin() * 1.3)
    assert torch.allclose(got, ref.rotate_interleaved(x, range(5), f, 1.3))


@pytest.mark.parametrize("window", [1, 2, 7, None])
def test_attention_window_and_sink(window):
    q, k, v = (torch.randn(12, 2, d, dtype=torch.float64) * 2 for d in (6, 6, 4))
    sink = torch.tensor([3.0, -1.0], dtype=torch.float64)
    cu = torch.tensor([0, 5, 12])
    got = om.sink_window_attention(q, k, v, 0.4, window, sink, cu)
    for a, b in ((0, 5), (5, 12)):
        assert torch.allclose(got[a:b], ref.sink_window_attention(q[a:b], k[a:b], v[a:b], 0.4, window, sink))


def test_mlstm_parallel_form():
    T, H = 23, 2
    q, k, v = (torch.randn(T, H, d, dtype=torch.float64) for d in (5, 5, 3))
    ig, z = 6 * torch.randn(T, H, dtype=torch.float64), 4 * torch.randn(T, H, dtype=torch.float64)
    fg = torch.nn.functional.logsigmoid(z)
    got = om.mlstm_parallel(q, k, v, ig, fg, torch.tensor([0, 1, 9, T]))
    for a, b in ((0, 1), (1, 9), (9, T)):
        assert torch.allclose(got[a:b], ref.mlstm_recurrence(q[a:b], k[a:b], v[a:b], ig[a:b], fg[a:b]))


@pytest.mark.parametrize("cfg", [U.ODD, U.TILES, U.ONES])
def test_model_matches_restatement(cfg):
    m, t = U.make(cfg)
    a, b = U.tokens(31, cfg["vocab"], 1), U.tokens(44, cfg["vocab"], 2)
    got = m(torch.tensor([a + b]), position_ids=torch.tensor([list(range(31)) + list(range(44))])).logits[0]
    assert U.rel(got[:31], U.logits(cfg, t, a)) < 2e-5
    assert U.rel(got[31:], U.logits(cfg, t, b)) < 2e-5


def test_borrowed_weights_are_one_set_of_parameters():
    m, _ = U.make(U.ODD)
    assert m.layers[3] is m.layers[1] and m.layers[5] is m.layers[1] and m.layers[4] is m.layers[0]
    assert m.layers[2] is not m.layers[1]
    assert {n.split(".")[0] for n in m.named_tensors()} == {"embed", "head", "final", "l0", "l1", "l2", "l6"}


def test_checkpoint_round_trip(tmp_path):
    m, t = U.make(U.ODD, torch.bfloat16)
    m.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json"))["layers"][3]["weights_of"] == 1
    again = load_model(str(tmp_path), dtype=torch.bfloat16)
    assert isinstance(again, LayeredLM) and again.config.num_hidden_layers == 7
    for name, x in again.named_tensors().items():
        assert torch.equal(x.double(), t[name]), name
    from safetensors.torch import load_file

    sd = load_file(str(tmp_path / "model.safetensors"))
    del sd["l2.mix.sink"]
    with pytest.raises(KeyError, match="l2.mix.sink"):
        again.load_named_tensors(sd)


def test_config_errors():
    bad = json.loads(json.dumps(U.ODD))
    bad["layers"][3]["mixer"]["vdim"] += 1
    with pytest.raises(ValueError, match="described differently"):
        ModelArch.from_hf_dict(bad)
    bad = json.loads(json.dumps(U.ODD))
    bad["layers"][0]["type"] = "nothing"
    with pytest.raises(ValueError, match="not registered"):
        ModelArch.from_hf_dict(bad)
    bad = json.loads(json.dumps(U.ODD))
    bad["layers"][1]["weights_of"] = 4
    with pytest.raises(ValueError, match="earlier layer"):
        ModelArch.from_hf_dict(bad)
    with pytest.raises(ValueError, match="not registered"):
        ModelArch.from_hf_dict(dict(U.ODD, architecture="Unknown"))


def test_preset_trains_on_cpu():
    m = build_model(preset("tiny-zorelorn"))
    ids = torch.randint(0, 1024, (2, 24))
    loss = m(ids, labels=ids).loss
    loss.backward()
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for p in m.parameters())
    assert m.config.num_parameters() == sum(p.numel() for p in m.parameters())


def test_greedy_generation():
    m, t = U.make(U.ODD)
    prompts = [U.tokens(6, 203, 3), U.tokens(19, 203, 4)]
    outs = EagerGenerator(m).generate(prompts, SamplingParams(max_tokens=6, greedy=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(6):
            seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
        assert o.token_ids == seq[len(p):]


def test_packed_context_lengths():
    m, _ = U.make(U.ONES)
    ctx = SeqCtx.from_lengths([1, 4, 2], "cpu")
    h = m.forward_hidden(torch.tensor(U.tokens(7, 11)), ctx)
    alone = m.forward_hidden(torch.tensor(U.tokens(7, 11)[1:5]), SeqCtx.from_lengths([4], "cpu"))
    assert torch.allclose(h[1:5], alone, atol=1e-6)


def test_scheduler_grows_and_reuses_pages():
    from trl_b200._native import host_runtime

    rt = host_runtime()
    if rt is None:
        pytest.skip("host library not built")
    bt = np.zeros((3, 8), dtype=np.int32)
    s = rt.scheduler(3, 6, 4, 8)
    s.add(0, 5, 0, 0)
    s.add(1, 4, 0, 1)
    admitted = {rid: slot for rid, slot, _, _ in s.admit(bt)}
    assert s.num_free_blocks == 3
    a, b = admitted[0], admitted[1]
    assert s.grow(a, 8, bt) == 0 and s.grow(a, 9, bt) == 1 and s.grow(b, 5, bt) == 1
    used = list(bt[a, :3]) + list(bt[b, :2])
    assert len(set(used)) == 5
    assert s.grow(b, 9, bt) == 1
    with pytest.raises(RuntimeError, match="full"):
        s.grow(a, 13, bt)
    with pytest.raises(ValueError):
        s.grow(2, 4, bt)
    s.retire(a, 0)
    assert s.num_free_blocks == 3
    assert s.grow(b, 24, bt) == 3 and len(set(bt[b, :6])) == 6
    with pytest.raises(ValueError):
        s.grow(b, 33, bt)


def test_server_serves_a_checkpoint_without_tokenizer(tmp_path):
    from trl_b200.scripts.rollout_serve import ServeArguments, WorkerPool

    m, t = U.make(U.ODD)
    m.save_pretrained(str(tmp_path))
    pool = WorkerPool(ServeArguments(model=str(tmp_path), max_model_len=64))
    try:
        assert pool.tok is None
        prompt = U.tokens(7, 203, 9)
        out = pool.generate([prompt], {"max_tokens": 3, "generation_kwargs": {"greedy": True}})
        seq = list(prompt)
        for _ in range(3):
            seq.append(int(U.logits(U.ODD, t, seq)[-1].argmax()))
        assert out[0][1] == seq[7:]
    finally:
        pool.close()


def test_replay_command_needs_the_documented_arguments():
    from trl_b200.scripts.trace_run import main

    with pytest.raises(SystemExit):
        main(["--model", "x"])
