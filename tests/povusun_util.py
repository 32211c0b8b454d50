"""Small random Povusun models for the tests, beside their restatement in povusun_reference.py."""
import torch

import povusun_reference as ref
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model


def attention(heads=6, kv_heads=3, dim=20, vdim=28, scale=0.3, softcap=4.0, q_temp=(0.4, 7), mlp=None, **mixer):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, **mixer)
    if softcap:
        m["softcap"] = softcap
    if q_temp:
        m["q_temp"] = dict(coef=q_temp[0], every=q_temp[1])
    return dict(type="attention", mixer=m, mlp=mlp)


def latent(heads=5, dim=12, vdim=20, kv_rank=28, scale=0.3, mlp=None):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=scale), mlp=mlp)


def rglru(width=60, blocks=4, conv=4, mlp=None):
    return dict(type="rglru", mixer=dict(width=width, blocks=blocks, conv=conv), mlp=mlp)


def ff(n, limit=0.7):
    return dict(kind="dense", ff=n, limit=limit)


def config(layers, width=84, vocab=197, eps=1e-5, side=12):
    c = dict(architecture="Povusun", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if side:
        c["token_side"] = dict(dim=side)
    return c


# sizes that fit no vector width, layers without a feed-forward, two borrowers of one cache, several convolution lengths
ODD = config([rglru(conv=3, mlp=ff(50)), attention(mlp=ff(31, 2.5)), latent(mlp=ff(40)), attention(kv_from=1, scale=0.2, q_temp=(0.9, 3)),
              rglru(width=33, blocks=1, conv=1), attention(heads=3, kv_heads=3, dim=9, vdim=5, softcap=None, q_temp=None, mlp=ff(17)),
              attention(kv_from=1, softcap=1.5, q_temp=None, mlp=ff(9)), latent(heads=1, dim=7, vdim=3, kv_rank=5), rglru(width=14, blocks=7, conv=6)],
             side=11)
# sizes that the tensor-core kernels take: several boxes per head, groups of 10 and of 1, blocks over one channel tile
TILES = config([attention(heads=20, kv_heads=2, dim=72, vdim=136, scale=0.15, softcap=20.0, q_temp=(0.3, 40), mlp=ff(96)),
                rglru(width=272, blocks=2, conv=4, mlp=ff(72, 1.5)), latent(heads=3, dim=40, vdim=72, kv_rank=136, scale=0.2, mlp=ff(64)),
                attention(heads=20, kv_heads=2, dim=72, vdim=136, scale=0.1, softcap=None, q_temp=None, kv_from=0, mlp=ff(40, 3.0)),
                attention(heads=2, kv_heads=2, dim=24, vdim=16, scale=0.4, q_temp=(0.2, 1)), rglru(width=96, blocks=4, conv=2, mlp=ff(160)),
                latent(heads=4, dim=128, vdim=128, kv_rank=64, scale=0.09)], width=160, side=40)
# one of everything, no token input
ONES = config([attention(heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0), latent(heads=1, dim=8, vdim=8, kv_rank=8), rglru(width=8, blocks=1, conv=2, mlp=ff(8))],
              width=8, vocab=13, side=0)


def make(cfg, dtype=torch.float32, device=None, seed=0):
    """Model with every tensor random (bf16-representable), plus the same tensors in float64 by checkpoint name."""
    m = build_model(ModelArch.from_hf_dict(cfg), dtype=dtype, device=device).eval().requires_grad_(False)
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, t in sorted(m.named_tensors().items()):
        z = torch.randn(t.shape, generator=g, dtype=torch.float64)
        leaf = name.split(".")[-1]
        if leaf in ("ra", "ri"):
            z = 2 * z / t.shape[-1] ** 0.5
        elif leaf == "conv":
            z = z / t.shape[1] ** 0.5
        elif name in ("embed", "side.embed"):
            z = z * 0.5 if name == "embed" else z
        elif t.ndim >= 2 and leaf != "b":
            z = z / t.shape[1] ** 0.5
        elif leaf == "lam":
            z = -3 + 2 * z  # from slow to fast decay
        elif leaf in ("norm1", "norm2", "norm1b", "norm2b", "norm"):
            z = 1.0 + 0.2 * z
        else:
            z = 0.3 * z
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
