"""Small random Zorelorn models for the tests, beside their restatement in zorelorn_reference.py."""
import torch

import zorelorn_reference as ref
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model


def latent(heads=3, dim=24, rot=16, vdim=40, q_rank=36, kv_rank=44, window=17, base=5000.0, scale=0.17,
           scaling=dict(factor=3.0, original=64, fast=8.0, slow=1.0), **rest):
    return dict(type="latent_attention",
                mixer=dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                           mask=dict(size=window) if window else None,
                           rot=dict(base=base, dims=rot, **({"scaling": dict(scaling)} if scaling else {}))),
                mlp=rest.pop("mlp", None), **rest)


def mlstm(heads=5, dim=20, vdim=28, cap=9.0, **rest):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), mlp=rest.pop("mlp", None), **rest)


def ff(n):
    return dict(kind="dense", ff=n)


def config(layers, width=88, vocab=203, eps=1e-5, scale=3.0):
    return dict(architecture="Zorelorn", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                layers=[{k: v for k, v in l.items()} for l in layers])


# sizes that fit no vector width, a feed-forward on either mixer, shared weights of both mixers, two windows
ODD = config([mlstm(mlp=ff(50)), latent(), latent(heads=1, dim=9, rot=2, vdim=5, q_rank=1, kv_rank=7, window=3, mlp=ff(31)),
              latent(weights_of=1), mlstm(weights_of=0, mlp=ff(50)), latent(weights_of=3), mlstm(heads=1, dim=7, vdim=3)])
# sizes that the tensor-core kernels take: several boxes per head, rotated part longer than the rest, window over tiles
TILES = config([latent(heads=2, dim=72, rot=64, vdim=136, q_rank=64, kv_rank=48, window=150, mlp=ff(96)),
                mlstm(heads=2, dim=64, vdim=96), latent(heads=4, dim=16, rot=32, vdim=24, q_rank=40, kv_rank=24, window=40),
                mlstm(heads=3, dim=128, vdim=128, cap=12.0, mlp=ff(64)),
                latent(heads=2, dim=128, rot=64, vdim=128, q_rank=32, kv_rank=128, window=None, scaling=None)], width=160)
# one head of everything
ONES = config([latent(heads=1, dim=8, rot=8, vdim=8, q_rank=8, kv_rank=8, window=1), mlstm(heads=1, dim=1, vdim=1, mlp=ff(8))],
              width=8, vocab=11, scale=1.0)


def make(cfg, dtype=torch.float32, device=None, seed=0, gain=1.0):
    """Model with every tensor random (bf16-representable), plus the same tensors in float64 by checkpoint name."""
    m = build_model(ModelArch.from_hf_dict(cfg), dtype=dtype, device=device).eval().requires_grad_(False)
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, t in m.named_tensors().items():
        z = torch.randn(t.shape, generator=g, dtype=torch.float64)
        leaf = name.split(".")[-1]
        if name.endswith((".alpha",)):
            z = 0.5 + 0.1 * z
        elif t.ndim >= 2:
            z = z * gain / t.shape[1] ** 0.5 * (3.0 if leaf in ("i", "f") else 1.0)
        elif name.endswith("f.b"):
            z = z + 2.0
        elif leaf in ("norm1", "norm2", "norm"):
            z = 1.0 + 0.2 * z
        z = z.bfloat16().double()
        t.copy_(z)
        tensors[name] = z
    return m, tensors


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel(got, want):
    """Worst row error of centred logits over the typical size of a row."""
    got, want = got.double().cpu(), want.double()
    d = (got - want) - (got - want).mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.var(-1).mean().sqrt())


def logits(cfg, tensors, toks):
    return ref.forward(cfg, tensors, toks)
