"""Small random Suposun models for the tests, beside their restatement in suposun_reference.py."""
import torch

import suposun_reference as ref
from trl_b200.models.configuration import ModelArch
from trl_b200.models.hf_io import build_model


def yarn(factor=3.0, original=60, fast=6.0, slow=0.5):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def attention(heads=6, kv_heads=2, dim=20, scale=0.4, softcap=5.0, mask=(9, 2), rot=(8, 5e2), scaling=None, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale)
    if softcap:
        m["softcap"] = softcap
    if mask:
        m["mask"] = dict(size=mask[0], keep_first=mask[1])
    if rot:
        m["rot"] = dict(base=rot[1], dims=rot[0])
        if scaling:
            m["rot"]["scaling"] = scaling
    return dict(type="attention", mixer=m, mlp=mlp)


def attention_2(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.35, rot=(12, 2e3), mlp=None, **mixer):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, **mixer)
    if rot:
        m["rot"] = dict(base=rot[1], dims=rot[0])
    return dict(type="attention_2", mixer=m, mlp=mlp)


def ff(n):
    return dict(kind="dense", ff=n)


def moe(n, experts, top, limit=1.1):
    return dict(kind="moe", expert=dict(ff=n, limit=limit), router=dict(experts=experts, top=top))


def config(layers, width=76, vocab=193, eps=1e-4, scale=3.0, pairs=(97, 13, 5), logit_scale=0.7):
    c = dict(architecture="Suposun", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers, embedding=dict(scale=scale),
             logit_scale=logit_scale)
    if pairs:
        c["embedding"]["bigram"] = dict(buckets=pairs[0], mul_prev=pairs[1], mul_cur=pairs[2])
    return c


# sizes that fit no vector width, layers without a feed-forward, two borrowers of one cache (with other scales), windows of one and
# of many tokens with and without kept ones, a part and the whole of a head rotated, values of another size than keys
ODD = config([attention(mlp=moe(17, 7, 3)), attention_2(mlp=ff(31)), attention(heads=5, kv_heads=5, dim=9, mask=(1, 3), rot=(6, 40.0), softcap=2.0),
              attention_2(kv_from=1, scale=0.2, mlp=moe(9, 5, 5, 0.6)), attention(heads=3, kv_heads=1, dim=14, mask=(25, 0), rot=(14, 1e3), scaling=yarn(), mlp=ff(50)),
              attention_2(kv_from=1, scale=0.5, mlp=ff(18)), attention(mask=None, softcap=None, rot=(2, 10.0), mlp=moe(20, 4, 1)),
              attention_2(heads=3, kv_heads=3, dim=7, vdim=7, rot=(4, 3e2))])
# sizes that the tensor-core kernels take: several boxes per head, groups of 10 and of 1, windows inside, over and far below a tile,
# kept tokens over more than a tile, experts wider and narrower than a tile
TILES = config([attention(heads=20, kv_heads=2, dim=72, scale=0.12, softcap=8.0, mask=(40, 3), rot=(24, 3e3), scaling=yarn(2.0, 100), mlp=moe(40, 6, 2)),
                attention_2(heads=6, kv_heads=2, dim=56, vdim=136, scale=0.13, rot=(56, 9e4), mlp=ff(96)),
                attention(heads=4, kv_heads=1, dim=128, scale=0.09, softcap=30.0, mask=(200, 130), rot=(64, 2e5), mlp=ff(160)),
                attention_2(heads=6, kv_heads=2, dim=56, vdim=136, scale=0.2, rot=(56, 9e4), kv_from=1, mlp=moe(136, 12, 4, 2.0)),
                attention(heads=3, kv_heads=3, dim=16, scale=0.3, softcap=3.0, mask=(130, 1), rot=(16, 50.0), mlp=moe(64, 3, 3)),
                attention_2(heads=8, kv_heads=8, dim=40, vdim=24, scale=0.2, rot=(40, 1e6))], width=160, vocab=200)
# one of everything
ONES = config([attention(heads=1, kv_heads=1, dim=8, mask=(1, 1), rot=(8, 7.0), mlp=moe(8, 1, 1)), attention_2(heads=1, kv_heads=1, dim=8, vdim=8, rot=(2, 9.0), mlp=ff(8))],
              width=8, vocab=13, scale=1.0, pairs=(1, 1, 1), logit_scale=1.0)
# neither pairs of tokens nor rotation nor experts
PLAIN = config([attention(rot=None, mask=None, mlp=ff(24)), attention_2(rot=None, mlp=ff(24))], width=40, pairs=None, scale=2.0)


def make(cfg, dtype=torch.float32, device=None, seed=0, clear=False):
    """Model with every tensor random (bf16-representable), plus the same tensors in float64 by checkpoint name.  ``clear``:
    corrections far apart, so that rounding cannot change which experts are chosen (their weights still vary)."""
    m = build_model(ModelArch.from_hf_dict(cfg), dtype=dtype, device=device).eval().requires_grad_(False)
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, t in sorted(m.named_tensors().items()):
        z = torch.randn(t.shape, generator=g, dtype=torch.float64)
        leaf = name.split(".")[-1]
        if name in ("embed", "bigram"):
            z = z * 0.5
        elif leaf == "router":
            z = 1.5 * z / t.shape[1] ** 0.5
        elif leaf == "correction":
            z = 2.0 * z.argsort() if clear else 0.4 * z
        elif t.ndim >= 2:
            z = z / t.shape[1] ** 0.5
        elif leaf == "norm" and ".mix." in name:
            z = 1.0 + 0.3 * z
        elif leaf in ("ls1", "ls2"):
            z = 0.8 + 0.3 * z
        elif leaf == "sink":
            z = 1.0 + z
        else:
            z = 0.3 * z  # norms about zero
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
