"""Small random Gerupel models for the tests, beside their restatement in gerupel_reference.py."""
import copy

import torch

import gerupel_reference as ref
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model


def llama3(factor=4.0, low=0.5, high=3.0, original=50):
    return dict(factor=factor, low=low, high=high, original=original)


def left(heads=6, kv_heads=2, dim=20, vdim=28, scale=0.3, mask=(7, 3), rot=(8, 5e2), scaling=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if mask:
        m["mask"] = dict(size=mask[0], pool=mask[1])
    if rot:
        m["rot"] = dict(base=rot[1], dims=rot[0])
        if scaling:
            m["rot"]["scaling"] = scaling
    return m


def right(heads=3, dim=18, vdim=10):
    return dict(heads=heads, dim=dim, vdim=vdim)


def moe(n, experts, top, scale=1.7):
    return dict(kind="moe", expert=dict(ff=n), router=dict(experts=experts, top=top, scale=scale))


def layer(l=None, r=None, mlp=None, scales=(0.9, 0.6)):
    return dict(type="parallel", mixer=dict(left=l or left(), right=r or right(), left_scale=scales[0], right_scale=scales[1]), mlp=mlp)


def config(layers, width=76, vocab=193, eps=1e-4, mult=0.6, loop=None):
    c = dict(architecture="Gerupel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers, residual_mult=mult)
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# sizes that fit no vector width, a layer without a feed-forward, a loop in the middle, windows of one and of many tokens, blocks of one
# token, smaller, equal to and larger than the window, a part, the whole and nothing of a head rotated, keys smaller and larger than values
ODD = config([layer(left(scaling=llama3()), mlp=moe(17, 7, 3)), layer(left(heads=5, kv_heads=5, dim=9, vdim=5, mask=(1, 1), rot=(6, 40.0)), right(1, 5, 33)),
              layer(left(heads=4, kv_heads=1, dim=14, vdim=6, mask=(4, 9), rot=(14, 1e3)), right(5, 7, 3), moe(9, 5, 5, 0.4), (1.0, 1.0)),
              layer(left(mask=(5, 5), rot=None), right(2, 40, 20), moe(20, 4, 1), (-0.5, 1.3))], loop=(1, 3, 3))
# sizes that the tensor-core kernels take: several boxes per head, groups of 10 and of 1, windows inside, over and far below a tile, more than
# a tile of blocks, states of one and of several tiles, experts wider and narrower than a tile
TILES = config([layer(left(20, 2, 72, 136, 0.12, (40, 1), (24, 3e3), llama3(2.0, 1.0, 4.0, 100)), right(4, 64, 128), moe(40, 6, 2)),
                layer(left(6, 2, 56, 72, 0.13, (130, 12), (56, 9e4)), right(2, 128, 72), moe(136, 3, 2)),
                layer(left(4, 1, 128, 128, 0.09, (24, 16), (64, 2e5)), right(3, 40, 24), moe(64, 4, 3))], width=160, vocab=200, loop=(0, 2, 2))
# one of everything
ONES = config([layer(left(1, 1, 8, 8, 1.0, (1, 1), (2, 7.0)), right(1, 8, 8), moe(8, 1, 1, 1.0), (1.0, 1.0))], width=8, vocab=13, mult=1.0, loop=(0, 1, 1))
# no loop, no window, no rotation
PLAIN = config([layer(left(mask=None, rot=None), mlp=moe(24, 4, 2)) for _ in range(2)], width=40, mult=1.0)


def every_expert(cfg):
    """The same model with every expert chosen: a choice that hangs on rounding says nothing about a kernel."""
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        if l["mlp"]:
            l["mlp"]["router"]["top"] = l["mlp"]["router"]["experts"]
    return cfg


def make(cfg, dtype=torch.float32, device=None, seed=0):
    """Model with every tensor random (bf16-representable), plus the same tensors in float64 by checkpoint name."""
    m = build_model(ModelArch.from_hf_dict(cfg), dtype=dtype, device=device).eval().requires_grad_(False)
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, t in sorted(m.named_tensors().items()):
        z = torch.randn(t.shape, generator=g, dtype=torch.float64)
        leaf = name.split(".")[-1]
        if name == "loop.step":
            z = z * 0.5
        elif leaf == "router":
            z = 1.5 * z / t.shape[1] ** 0.5
        elif t.ndim >= 2 and name != "embed":
            z = z / t.shape[1] ** 0.5
        elif leaf == "temp":
            z = 1.0 + 0.5 * z
        elif leaf == "lower":  # none, some, and much that is never forgotten
            z = torch.sigmoid(2 * z) * (z > -0.5)
        elif leaf == "b":      # from almost nothing to almost everything kept
            z = 1.0 + 3.0 * z
        elif name != "embed":
            z = 1.0 + 0.3 * z  # norms
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
