"""Decoders described layer by layer.

The flat families of :mod:`trl_b200.models.configuration` repeat one block.  A *layered* design instead lists its
layers in ``config.json``, each with a mixer (kind and sizes) and a feed-forward (or none); a layer may run with
another layer's weights, or attend to another layer's keys and values.  :data:`DESIGNS` registers what a design fixes
(norm and where it stands, feed-forward, head); everything else is read from the file.  A mixer is a module here
(parameters, tensor names, prompt forward) with its kernels in ``csrc/`` and its decode state in
``rollout/layered_engine.py``; registering another kind in :data:`MIXERS` makes it available to every layered design.

Designs
    Zorelorn    embeddings times a constant, Dynamic-Tanh norms, ``latent_attention`` (multi-head latent attention with
                YaRN rotary part, sliding window, softmax sink, per-head output gate) and ``mlstm`` (matrix memory with
                exponential gates) mixers, erf-GELU feed-forward.
    Povusun     RMS norms before and after every sublayer, ``attention`` (grouped queries, unit-rms queries and keys, query
                temperature by position, capped scores, per-element output gate; a layer may read another one's cache),
                ``latent_attention`` (without positions, queries straight from the input) and ``rglru`` (short convolution
                and real-gated linear recurrence) mixers, clamped gated feed-forward, a per-token input of every layer,
                tied head.
    Suposun     RMS norms (weights about zero) and layer scales on the sublayers' outputs only, a table of token pairs beside the
                embedding, ``attention`` (the projected keys are the values; weighted norms per head, YaRN rotation, window with
                kept first tokens, capped scores, softmax sink, gate per head) and ``attention_2`` (norms over all heads, rotated
                halves; a layer may read another one's cache) mixers, GELU-gated or expert feed-forward, tied head with a scale.
    Gerupel     mixer and feed-forward side by side behind a norm each, the residual sum times a constant, a run of layers
                repeated with the embedding added again, a norm on the embedding, ``parallel`` mixers (``attention`` over a window
                and pooled blocks before it, Llama-3 frequency scaling, factor per head, one in the softmax denominator, beside
                ``hgrn2``: linear attention whose forget gate also writes), experts chosen by softmax, tied head.

The residual stream, norms, gates and recurrent states are fp32 whatever the model dtype.
"""
from __future__ import annotations

import copy
import dataclasses
import json
import math
import os
from dataclasses import dataclass, field
from typing import Any

import torch
import torch.nn as nn

from ..ops import mixers as mx
from .configuration import ModelArch
from .decoder import CausalLM, SeqCtx


@dataclass(frozen=True)
class AttentionStyle:
    """What a design fixes about a grouped-query attention mixer."""

    norm: bool = True            # queries and keys over their rms
    norm_weight: bool = False    # times a weight
    whole_norm: bool = False     # that norm over all heads at once instead of per head
    halves: bool = False         # rotated pairs (i, i + dims / 2) instead of (2 i, 2 i + 1)
    values: bool = True          # a projection of values; without it the projected keys serve as values
    sink: bool = False           # exp(sink) in the softmax denominator
    sink_one: bool = False       # the same with exp(sink) = 1 for every head
    temp: bool = False           # scores times a number per head
    gate: str | None = "element"  # sigmoid gates per "element" or per "head" of the output


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models."""

    norm: str
    mlp: str | None              # dense feed-forward
    moe: str | None = None       # feed-forward of kind 'moe'
    beside: bool = False         # mixer and feed-forward read the same stream, each through its norm, and are added together
    embed_norm: bool = False     # a norm on the embedding
    sides: tuple = ()            # mixer 'parallel': the kinds of its left and its right half
    pre_norm: bool = True        # a norm on the input of every sublayer; without it the sublayers read the stream itself
    post_norm: bool = False      # a norm on the output of every sublayer, before it is added
    layer_scale: bool = False    # that norm's result times a vector
    latent_sink: bool = False    # latent_attention: exp(sink) in the softmax denominator
    latent_gate: bool = False    # latent_attention: sigmoid gate per head
    attention: dict = field(default_factory=dict)  # AttentionStyle by mixer kind, where it is not the default one
    tied_head: bool = False


DESIGNS: dict[str, Design] = {
    "Zorelorn": Design(norm="dynamic_tanh", mlp="gelu", latent_sink=True, latent_gate=True),
    "Povusun": Design(norm="rms", mlp="clamped_glu", post_norm=True, tied_head=True),
    "Suposun": Design(norm="rms_about_zero", mlp="gelu_glu", moe="clamped_glu_experts", pre_norm=False, post_norm=True, layer_scale=True,
                      tied_head=True,
                      attention={"attention": AttentionStyle(norm_weight=True, values=False, sink=True, gate="head"),
                                 "attention_2": AttentionStyle(norm_weight=True, whole_norm=True, halves=True, gate=None)}),
    "Gerupel": Design(norm="rms", mlp=None, moe="softmax_experts", beside=True, embed_norm=True, sides=("attention", "hgrn2"), tied_head=True,
                      attention={"attention": AttentionStyle(norm=False, halves=True, sink_one=True, temp=True, gate=None)}),
}


@dataclass
class LayerSpec:
    """One layer run.  ``owner``: place of the run whose tensors this one runs with (itself, usually); ``index``: entry of the
    layer list; ``enters``: number of the loop's pass that begins in front of it."""

    kind: str
    mixer: dict
    mlp: dict | None
    owner: int
    index: int
    enters: int | None = None

    @property
    def ff(self) -> int:
        return 0 if self.mlp is None else int((self.mlp.get("expert") or self.mlp)["ff"])

    @property
    def key(self):
        return (self.kind, json.dumps(self.mixer, sort_keys=True), json.dumps(self.mlp, sort_keys=True))


@dataclass
class LayeredArch(ModelArch):
    design: str = ""
    layers: list = field(default_factory=list)  # [LayerSpec], in the order of computation: a loop is unrolled
    passes: int = 0  # of the loop (0: none)
    residual_mult: float = 1.0  # what sublayer outputs are multiplied by when they are added
    side_dim: int = 0  # per-token input of every layer: elements per layer (0: none)
    pairs: dict | None = None  # table of token pairs: mul_prev, mul_cur, buckets
    logit_scale: float = 1.0
    source: dict = field(default_factory=dict)  # the config.json this came from

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "LayeredArch":
        name = d["architecture"]
        if name not in DESIGNS:
            raise ValueError(f"architecture={name!r} is not registered; layered designs: {sorted(DESIGNS)}")
        specs: list[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not registered; known: {sorted(MIXERS)}")
            mlp = e.get("mlp")
            if mlp is not None and not dict(dense=DESIGNS[name].mlp, moe=DESIGNS[name].moe).get(mlp.get("kind", "dense")):
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind', 'dense')!r} is not supported")
            owner = i
            if e.get("weights_of") is not None:
                j = int(e["weights_of"])
                if not 0 <= j < i:
                    raise ValueError(f"layer {i}: weights_of={j} must name an earlier layer")
                owner = specs[j].owner
            s = LayerSpec(e["type"], dict(e["mixer"]), None if mlp is None else dict(mlp), owner, i)
            _check_lender(specs, s, i)
            if owner != i and s.key != specs[owner].key:
                raise ValueError(f"layer {i} runs with the weights of layer {owner} but is described differently")
            specs.append(s)
        loop = d.get("loop")
        if loop:
            specs = _unrolled(specs, int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        design = DESIGNS[name]
        embedding = d.get("embedding") or {}
        heads = max((h.get("heads", 1) for s in specs for h in (s.mixer, s.mixer.get("left") or {}, s.mixer.get("right") or {})), default=1)
        return cls(model_type=name.lower(), design=name, vocab_size=d["vocab"], hidden_size=d["width"],
                   intermediate_size=max((s.ff for s in specs), default=0), num_hidden_layers=len(specs),
                   num_attention_heads=heads, num_key_value_heads=heads, rms_norm_eps=float(d["norm"]["eps"]),
                   embed_scale=float(embedding.get("scale", 1.0)), layers=specs, source=copy.deepcopy(d),
                   passes=int(loop["times"]) if loop else 0, residual_mult=float(d.get("residual_mult", 1.0)),
                   pairs=dict(embedding["bigram"]) if embedding.get("bigram") else None, logit_scale=float(d.get("logit_scale", 1.0)),
                   side_dim=int((d.get("token_side") or {}).get("dim", 0)), tie_word_embeddings=design.tied_head,
                   attention_bias=False, qk_norm=False, pad_token_id=d.get("pad_token_id"),
                   bos_token_id=d.get("bos_token_id"), eos_token_id=d.get("eos_token_id"))

    def to_hf_dict(self) -> dict[str, Any]:
        d = copy.deepcopy(self.source)
        d["vocab"] = self.vocab_size
        for k in ("pad_token_id", "bos_token_id", "eos_token_id"):
            if getattr(self, k) is not None:
                d[k] = getattr(self, k)
        return d

    @property
    def architectures(self) -> list[str]:
        return [self.design]

    def num_parameters(self, exclude_embeddings: bool = False) -> int:
        m = LayeredLM(self, device="meta", init=False)
        n = sum(p.numel() for p in m.parameters())
        return n - ((1 if self.tie_word_embeddings else 2) * self.vocab_size * self.hidden_size if exclude_embeddings else 0)

    @property
    def lenders(self) -> set:
        """Layers whose keys and values others borrow."""
        return {s.mixer["kv_from"] for s in self.layers if s.mixer.get("kv_from") is not None}


def _unrolled(specs: list, start: int, stop: int, times: int) -> list:
    """Layer runs of a list whose entries ``start`` .. ``stop`` - 1 run ``times`` times in a row with the same weights."""
    if not 0 <= start < stop <= len(specs) or times < 1:
        raise ValueError(f"loop over layers {start} .. {stop - 1} of {len(specs)}, {times} times")
    if any(s.mixer.get("kv_from") is not None for s in specs):
        raise ValueError("a loop together with layers that read another one's keys and values")
    out, first = [], {}
    for t in range(times):
        out += [(s, t if s.index == start else None) for s in specs[start:stop]]
    out = [(s, None) for s in specs[:start]] + out + [(s, None) for s in specs[stop:]]
    for place, (s, _) in enumerate(out):
        first.setdefault(s.index, place)
    return [dataclasses.replace(s, owner=first[s.owner], enters=t) for s, t in out]


def _check_lender(specs: list, s: LayerSpec, i: int):
    j = s.mixer.get("kv_from")
    if j is None:
        return
    if not 0 <= j < i or specs[j].kind != s.kind or specs[j].mixer.get("kv_from") is not None:
        raise ValueError(f"layer {i}: kv_from={j} must name an earlier layer of the same kind with keys and values of its own")
    for k in ("heads", "kv_heads", "dim", "vdim"):
        if specs[j].mixer[k] != s.mixer[k]:
            raise ValueError(f"layer {i}: {k} differs from that of layer {j}, whose keys and values it reads")


def _vec(n=None, fill=0.0, device=None):
    """Small per-channel parameters are fp32 in every model dtype: the kernels read them as such."""
    shape = () if n is None else (n,)
    return nn.Parameter(torch.full(shape, float(fill), dtype=torch.float32, device=device))


class DynamicTanh(nn.Module):
    """``tanh(alpha x) w + b``: a norm without statistics."""

    def __init__(self, cfg: LayeredArch, device=None, **kw):
        super().__init__()
        if kw or cfg.residual_mult != 1.0:
            raise NotImplementedError(f"Dynamic Tanh with {sorted(kw) or 'residual_mult'}")
        n = cfg.hidden_size
        self.weight, self.bias, self.alpha = _vec(n, 1.0, device), _vec(n, 0.0, device), _vec(None, 0.5, device)

    def tensors(self, name):
        return {name: self.weight, name + ".b": self.bias, name + ".alpha": self.alpha}

    def forward(self, x, out_dtype, delta=None, post=None, **kw):
        """x [T, H] fp32 -> (norm of the stream in ``out_dtype``, the stream).  ``delta``, when given, is added to the stream
        first (in place on CUDA), normalised by ``post`` when that is given.  ``clear`` (delta is zeroed) and ``out`` are for
        the decode step."""
        if post is not None:
            raise NotImplementedError("Dynamic Tanh around a sublayer's output")
        return mx.dynamic_tanh(x, delta, self.alpha, self.weight, self.bias, out_dtype, **kw)


class RmsNorm(nn.Module):
    """``x / sqrt(mean(x^2) + eps) w gain``; as a norm of a sublayer's output it may carry that sublayer's ``scale`` vector."""

    shift = 0.0  # added to the weight

    def __init__(self, cfg: LayeredArch, device=None, gain: float = 1.0, scale: bool = False):
        super().__init__()
        self.weight, self.eps, self.gain, self.mult = _vec(cfg.hidden_size, 1.0 - self.shift, device), cfg.rms_norm_eps, gain, cfg.residual_mult
        self.scale = _vec(cfg.hidden_size, 1.0, device) if scale else None

    def tensors(self, name):
        return {name: self.weight}

    def forward(self, x, out_dtype, delta=None, post=None, **kw):
        return mx.rms_residual(x, delta, w=self.weight, eps=self.eps, out_dtype=out_dtype, shift=self.shift, gain=self.gain,
                               mult=self.mult, **_weights(post), **kw)

    @staticmethod
    def stream(x, out_dtype, delta, post, mult=1.0, **kw):
        """The stream itself after the addition of ``delta`` (normed by ``post``), in ``out_dtype``, and in fp32."""
        eps, shift = (0.0, 0.0) if post is None else (post.eps, post.shift)
        return mx.rms_residual(x, delta, w=None, eps=eps, out_dtype=out_dtype, shift=shift, mult=mult, **_weights(post), **kw)


class RmsNormAboutZero(RmsNorm):
    """:class:`RmsNorm` with the weight stored as its distance from one."""

    shift = 1.0


def _weights(post):
    return dict(post=None) if post is None else dict(post=post.weight, post_scale=post.scale)


NORMS = {"dynamic_tanh": DynamicTanh, "rms": RmsNorm, "rms_about_zero": RmsNormAboutZero}


class LatentAttention(nn.Module):
    """Multi-head latent attention: keys and values of all heads are linear in one latent per token (plus one rotated
    key part shared by the heads), and only those are cached.  Queries come through a latent of their own (``q_rank``) or
    straight from the layer input.  In memory the projections that read the layer input are one matrix (query latent or
    queries | key/value latent | rotated key | gate), as are the key and value up-projections."""

    kind = "latent_attention"

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        design = DESIGNS[cfg.design]
        self.eps, self.gated = cfg.rms_norm_eps, design.latent_gate
        self.heads, self.dim, self.rot_dim, self.vdim = m["heads"], m["dim"], m.get("rot_dim", 0), m["vdim"]
        self.q_rank, self.kv_rank = m.get("q_rank", 0), m["kv_rank"]
        self.scale = float(m["scale"])
        mask = m.get("mask") or {}
        self.window = int(mask["size"]) if mask.get("size") else None
        self.rope = None
        if self.rot_dim:
            rot = m["rot"]
            if rot["dims"] != self.rot_dim or self.rot_dim % 2:
                raise ValueError("latent_attention rotates its whole rot_dim part, in pairs")
            self.rope = mx.RotarySpec(self.rot_dim, float(rot["base"]), rot.get("scaling"))
        h, q = cfg.hidden_size, self.heads * (self.dim + self.rot_dim)
        self.q_rows = self.q_rank or q  # first rows of w_in
        self.w_in = nn.Parameter(torch.empty(self.q_rows + self.kv_rank + self.rot_dim + (self.heads if self.gated else 0), h, **kw))
        self.uq = nn.Parameter(torch.empty(q, self.q_rank, **kw)) if self.q_rank else None
        self.ukv = nn.Parameter(torch.empty(self.heads * (self.dim + self.vdim), self.kv_rank, **kw))
        self.o = nn.Parameter(torch.empty(h, self.heads * self.vdim, **kw))
        self.q_norm = _vec(self.q_rank, 1.0, device) if self.q_rank else None
        self.kv_norm = _vec(self.kv_rank, 1.0, device)
        self.sink = _vec(self.heads, 0.0, device) if design.latent_sink else None

    @property
    def uk(self):
        return self.ukv[: self.heads * self.dim]

    @property
    def uv(self):
        return self.ukv[self.heads * self.dim:]

    def tensors(self, p):
        a, b = self.q_rows, self.q_rows + self.kv_rank + self.rot_dim
        out = ({p + "dq": self.w_in[:a], p + "dq.norm": self.q_norm, p + "uq": self.uq} if self.q_rank else {p + "q": self.w_in[:a]})
        out.update({p + "dkv": self.w_in[a:b], p + "dkv.norm": self.kv_norm, p + "uk": self.uk, p + "uv": self.uv})
        if self.sink is not None:
            out[p + "sink"] = self.sink
        if self.gated:
            out[p + "g"] = self.w_in[b:]
        out[p + "o"] = self.o
        return out

    def forward(self, h, ctx: SeqCtx, li: int):
        """[T, H] normed input -> [T, H] fp32 block output (packed prompts)."""
        return mx.latent_attention(self, h, ctx, li)


class MLstm(nn.Module):
    """Matrix-memory recurrence with exponential input and sigmoid forget gates, stabilised by a running maximum.  The
    projections that read the layer input are one matrix (query | key | value | output gate | input gate | forget
    gate)."""

    kind = "mlstm"

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.eps = cfg.rms_norm_eps
        self.heads, self.dim, self.vdim, self.cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
        h = cfg.hidden_size
        self.w_in = nn.Parameter(torch.empty(self.gate_row + 2 * self.heads, h, **kw))
        self.o = nn.Parameter(torch.empty(h, self.heads * self.vdim, **kw))
        self.norm = _vec(self.heads * self.vdim, 1.0, device)
        self.gate_bias = _vec(2 * self.heads, 0.0, device)

    @property
    def gate_row(self):
        """First row of the input / forget gate projections in ``w_in``."""
        return 2 * self.heads * (self.dim + self.vdim)

    def tensors(self, p):
        H, qd, vd = self.heads, self.heads * self.dim, self.heads * self.vdim
        r = self.gate_row
        return {p + "q": self.w_in[:qd], p + "k": self.w_in[qd:2 * qd], p + "v": self.w_in[2 * qd:2 * qd + vd],
                p + "g": self.w_in[2 * qd + vd:r], p + "o": self.o, p + "norm": self.norm,
                p + "i": self.w_in[r:r + H], p + "i.b": self.gate_bias[:H],
                p + "f": self.w_in[r + H:], p + "f.b": self.gate_bias[H:]}

    def forward(self, h, ctx: SeqCtx, li: int):
        return mx.mlstm(self, h, ctx, li)


class GroupedAttention(nn.Module):
    """Grouped-query attention: queries and keys over their rms, optionally rotated, queries optionally times a temperature that
    grows with the position or times a number per head, scores optionally capped by tanh, over all earlier keys or a window and
    the first tokens or the means of the key blocks before it, the output optionally times sigmoid gates that read the layer input
    (what of it a design has: :class:`AttentionStyle` and the layer's sizes).  With ``kv_from`` the layer has no keys and values
    of its own and reads those of another layer.  The projections are one matrix (query | key | value | gate, with gates per head
    filled up to whole 16-byte rows); a ``part`` of another mixer leaves both projections to that one."""

    kind = "attention"
    f32_rows = 0  # rows of the input projection whose fp32 sums are needed

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device, part: bool = False):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        style = DESIGNS[cfg.design].attention.get(self.kind, AttentionStyle())
        self.eps, self.dtype = cfg.rms_norm_eps, dtype
        self.heads, self.kv_heads, self.dim, self.vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads over {self.kv_heads} key/value heads")
        self.scale = float(m["scale"])
        self.cap = float(m["softcap"]) if m.get("softcap") else None
        t = m.get("q_temp")
        self.temperature = mx.TemperatureSpec(t["coef"], t["every"]) if t else None
        mask, rot = m.get("mask") or {}, m.get("rot")
        self.window = int(mask["size"]) if mask.get("size") else None
        self.keep = int(mask.get("keep_first") or 0)
        self.pool = int(mask.get("pool") or 0) if self.window else 0
        if self.pool and (self.keep or m.get("kv_from") is not None):
            raise ValueError("pooled blocks together with kept tokens or another layer's cache")
        self.rot, self.rope = (int(rot["dims"]), mx.RotarySpec(rot["dims"], float(rot["base"]), rot.get("scaling"))) if rot else (0, None)
        if self.rot % 2 or self.rot > self.dim:
            raise ValueError(f"{self.rot} rotated elements of {self.dim}")
        self.unit, self.whole_norm, self.halves, self.values, self.gate = style.norm, style.whole_norm, style.halves, style.values, style.gate
        if not self.values and self.vdim != self.dim:
            raise ValueError("values that are the keys have their size")
        self.kv_from = m.get("kv_from")
        own = self.kv_heads if self.kv_from is None else 0
        gates = {"element": self.heads * self.vdim, "head": self.heads, None: 0}[self.gate]
        self.parts = [self.heads * self.dim, own * self.dim, own * self.vdim if self.values else 0, gates]  # rows of w_in
        self.rows, self.out_width = sum(self.parts), self.heads * self.vdim
        h, fill = cfg.hidden_size, -self.rows % 8 if self.gate == "head" else 0
        if not part:
            self.w_in = nn.Parameter(torch.empty(self.rows + fill, h, **kw))
            if fill:
                self.w_in.data[-fill:].zero_()
            self.o = nn.Parameter(torch.empty(h, self.out_width, **kw))
        self.q_norm = self.k_norm = None
        if style.norm_weight:
            self.q_norm = _vec(self.heads * self.dim if self.whole_norm else self.dim, 1.0, device)
            if own:
                self.k_norm = _vec(own * self.dim if self.whole_norm else self.dim, 1.0, device)
        self.temp = _vec(self.heads, 1.0, device) if style.temp else None
        if style.sink_one:
            self.register_buffer("sink", torch.zeros(self.heads, dtype=torch.float32, device=device), persistent=False)
        else:
            self.sink = _vec(self.heads, 0.0, device) if style.sink else None
        self.sink_learned = style.sink

    @property
    def prep(self) -> dict:
        """How queries and keys are prepared (:func:`~trl_b200.ops.cuda_mixers.attn_prep`)."""
        return dict(q_norm=self.q_norm, k_norm=self.k_norm, unit=self.unit, whole_norm=self.whole_norm, q_head=self.temp, rot=self.rot,
                    halves=self.halves, values=self.values, gates=self.gate)

    @property
    def sight(self) -> dict:
        """What a query sees besides the earlier tokens' keys as they are."""
        return dict(window=self.window, keep=self.keep, sink=self.sink)

    def tensors(self, p, w_in=None, o=None):
        """``w_in``, ``o``: where a part's projections are."""
        q, k, v, g = (self.w_in[: self.rows] if w_in is None else w_in).split(self.parts)
        out = {p + "q": q, p + "o": self.o if o is None else o}
        if self.kv_from is None:
            out[p + "k"] = k
            if self.values:
                out[p + "v"] = v
        if self.gate:
            out[p + "g"] = g
        out.update({p + n: t for n, t in (("q.norm", self.q_norm), ("k.norm", self.k_norm), ("sink", self.sink if self.sink_learned else None),
                                          ("temp", self.temp)) if t is not None})
        return out

    def forward(self, h, ctx: SeqCtx, li: int):
        return mx.attention(self, h, ctx, li)


class GroupedAttention2(GroupedAttention):
    """The other grouped-query attention of a design that has two."""

    kind = "attention_2"


class RgLru(nn.Module):
    """Griffin's recurrent block: a GELU branch times a branch of a short causal convolution and a linear recurrence per
    channel whose decay and input gates are block-diagonal in the convolved input.  The projections are one matrix (GELU
    branch | recurrent branch), the gates' weights one tensor (recurrence gate, input gate)."""

    kind = "rglru"
    decay = 8.0  # log a = -decay * gate * softplus(lam)

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.eps = cfg.rms_norm_eps
        self.width, self.blocks, self.taps = m["width"], m["blocks"], m["conv"]
        if self.width % self.blocks:
            raise ValueError(f"{self.width} channels in {self.blocks} blocks")
        h, w, wb = cfg.hidden_size, self.width, self.width // self.blocks
        self.w_in = nn.Parameter(torch.empty(2 * w, h, **kw))
        self.gates = nn.Parameter(torch.empty(2, self.blocks, wb, wb, **kw))
        self.o = nn.Parameter(torch.empty(h, w, **kw))
        self.y_bias, self.x_bias, self.conv_bias, self.lam = (_vec(w, 0.0, device) for _ in range(4))
        f32 = dict(dtype=torch.float32, device=device)
        self.gate_bias = nn.Parameter(torch.zeros(2, w, **f32))
        self.conv = nn.Parameter(torch.zeros(w, self.taps, **f32))

    def tensors(self, p):
        w = self.width
        b = self.gate_bias.view(2, self.blocks, -1)
        return {p + "y": self.w_in[:w], p + "y.b": self.y_bias, p + "x": self.w_in[w:], p + "x.b": self.x_bias, p + "conv": self.conv,
                p + "conv.b": self.conv_bias, p + "ra": self.gates[0], p + "ra.b": b[0], p + "ri": self.gates[1], p + "ri.b": b[1],
                p + "lam": self.lam, p + "o": self.o}

    def forward(self, h, ctx: SeqCtx, li: int):
        return mx.rglru(self, h, ctx, li)


class HGrn2(nn.Module):
    """Linear attention in which one gate per head and channel forgets and writes: ``S = diag(f) S + (1 - f) v^T``, ``o = S^T q``
    with ``f`` between a learned lower bound and one, and an RMS norm per head on the result.  The projections are one matrix
    (query | value | forget gate); a ``part`` of another mixer leaves both projections to that one."""

    kind = "hgrn2"

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device, part: bool = False):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.eps, self.dtype = cfg.rms_norm_eps, dtype
        self.heads, self.dim, self.vdim = m["heads"], m["dim"], m["vdim"]
        qd, vd = self.heads * self.dim, self.heads * self.vdim
        self.parts, self.rows, self.f32_rows, self.out_width = [qd, vd, qd], qd + vd, qd, vd
        h = cfg.hidden_size
        if not part:
            self.w_in = nn.Parameter(torch.empty(sum(self.parts), h, **kw))
            self.o = nn.Parameter(torch.empty(h, vd, **kw))
        self.f_bias, self.lower, self.norm = _vec(qd, 0.0, device), _vec(qd, 0.0, device), _vec(self.vdim, 1.0, device)

    def tensors(self, p, w_in=None, o=None):
        """``w_in``, ``o``: where a part's projections are."""
        q, v, f = (self.w_in if w_in is None else w_in).split(self.parts)
        return {p + "q": q, p + "f": f, p + "f.b": self.f_bias, p + "lower": self.lower, p + "v": v, p + "norm": self.norm,
                p + "o": self.o if o is None else o}

    def forward(self, h, ctx: SeqCtx, li: int):
        return mx.hgrn2(self, h, ctx, li)


class ParallelMixers(nn.Module):
    """Two mixers side by side: ``left_scale left(x) + right_scale right(x)``.  Both input projections are one matrix (left's rows
    | right's rows | rows whose fp32 sums are needed), and so are both output projections; the scales go to the halves' results."""

    kind = "parallel"

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.left, self.right = (MIXERS[k](cfg, m[s], dtype, device, part=True) for k, s in zip(DESIGNS[cfg.design].sides, ("left", "right")))
        if self.left.f32_rows:
            raise ValueError("the half with fp32 projections is the right one")
        self.scales = (float(m["left_scale"]), float(m["right_scale"]))
        self.rows = self.left.rows + self.right.rows
        self.w_in = nn.Parameter(torch.empty(self.rows + self.right.f32_rows, cfg.hidden_size, **kw))
        self.o = nn.Parameter(torch.empty(cfg.hidden_size, self.left.out_width + self.right.out_width, **kw))

    def tensors(self, p):
        a, b = self.left.rows, self.left.out_width
        return {**self.left.tensors(p + "left.", self.w_in[:a], self.o[:, :b]), **self.right.tensors(p + "right.", self.w_in[a:], self.o[:, b:])}

    def forward(self, h, ctx: SeqCtx, li: int):
        return mx.parallel(self, h, ctx, li)


MIXERS = {c.kind: c for c in (LatentAttention, MLstm, GroupedAttention, GroupedAttention2, RgLru, HGrn2, ParallelMixers)}


class DenseMlp(nn.Module):
    """``down(act(up x))`` with the exact GELU.

    ``w_in`` is the first product's weight, ``fused`` names its activation to the weight-streaming product, ``act`` is that
    activation alone."""

    fused = dict(gelu=True)

    def __init__(self, cfg: LayeredArch, spec: dict, dtype, device):
        super().__init__()
        ff = int(spec["ff"])
        self.up = nn.Parameter(torch.empty(ff, cfg.hidden_size, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.empty(cfg.hidden_size, ff, dtype=dtype, device=device))

    @property
    def w_in(self):
        return self.up

    def tensors(self, p):
        return {p + "up": self.up, p + "down": self.down}

    def act(self, z, out=None):
        return mx.gelu_erf(z, out)

    def forward(self, h):
        return mx.linear_f32(self.act(mx.linear(h, self.w_in)), self.down)


class GeluGluMlp(DenseMlp):
    """``down(gelu_tanh(gate x) * up x)``.  Gate and up projections are one matrix."""

    fused = dict(gelu_glu=True)

    def __init__(self, cfg: LayeredArch, spec: dict, dtype, device):
        nn.Module.__init__(self)
        self.ff = int(spec["ff"])
        self.gate_up = nn.Parameter(torch.empty(2 * self.ff, cfg.hidden_size, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.empty(cfg.hidden_size, self.ff, dtype=dtype, device=device))

    @property
    def w_in(self):
        return self.gate_up

    def tensors(self, p):
        return {p + "gate": self.gate_up[: self.ff], p + "up": self.gate_up[self.ff:], p + "down": self.down}

    def act(self, z, out=None):
        return mx.gelu_glu(z, out)


class ClampedGluMlp(GeluGluMlp):
    """``down(g sigmoid(alpha g) (u + shift))`` with ``g = min(gate x, limit)`` and ``u = up x`` within +- limit."""

    alpha, shift = 1.702, 1.0

    def __init__(self, cfg: LayeredArch, spec: dict, dtype, device):
        super().__init__(cfg, spec, dtype, device)
        self.limit = float(spec["limit"])

    @property
    def glu(self):
        return self.limit, self.alpha, self.shift

    @property
    def fused(self):
        return dict(clamped_glu=self.glu)

    def act(self, z, out=None):
        return mx.clamped_glu(z, *self.glu, out=out)


class ExpertMlp(nn.Module):
    """Mixture of experts, each a clamped gated unit: a token runs the ``top`` experts of the largest sigmoid score plus
    correction and adds them up with their bare scores as weights.  The experts' matrices are stacked."""

    alpha, shift = 1.702, 1.0
    scores = "sigmoid"
    renormalize = False  # weights over their sum
    gain = 1.0           # of the weights

    def __init__(self, cfg: LayeredArch, spec: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.n, self.top = int(spec["router"]["experts"]), int(spec["router"]["top"])
        self.ff, self.limit = int(spec["expert"]["ff"]), float(spec["expert"].get("limit", math.inf))
        if not 1 <= self.top <= self.n <= 1024:
            raise ValueError(f"{self.top} of {self.n} experts (at most 1024)")
        h = cfg.hidden_size
        self.router = nn.Parameter(torch.empty(self.n, h, **kw))
        self.correction = _vec(self.n, 0.0, device) if self.scores == "sigmoid" else None
        self.gate_up = nn.Parameter(torch.empty(self.n, 2 * self.ff, h, **kw))
        self.down = nn.Parameter(torch.empty(self.n, h, self.ff, **kw))

    @property
    def glu(self):
        return self.limit, self.alpha, self.shift

    @property
    def routing(self) -> dict:
        return dict(scores=self.scores, renormalize=self.renormalize, gain=self.gain)

    def tensors(self, p):
        out = {p + "router": self.router}
        if self.correction is not None:
            out[p + "correction"] = self.correction
        for e in range(self.n):
            out.update({f"{p}e{e}.gate": self.gate_up[e, : self.ff], f"{p}e{e}.up": self.gate_up[e, self.ff:], f"{p}e{e}.down": self.down[e]})
        return out

    def forward(self, h, summed: bool = True):
        """``summed``: see :func:`~trl_b200.ops.mixers.experts`."""
        return mx.experts(self, h, summed=summed)


class SoftmaxExpertMlp(ExpertMlp):
    """Mixture of SiLU-gated units: the ``top`` experts of the largest softmax score, weighted with their scores over the sum of
    these, times a constant."""

    alpha, shift = 1.0, 0.0  # the clamped unit without its limit is the SiLU-gated one
    scores, renormalize = "softmax", True

    def __init__(self, cfg: LayeredArch, spec: dict, dtype, device):
        super().__init__(cfg, spec, dtype, device)
        self.gain = float(spec["router"].get("scale", 1.0))


MLPS = {"gelu": DenseMlp, "gelu_glu": GeluGluMlp, "clamped_glu": ClampedGluMlp, "clamped_glu_experts": ExpertMlp,
        "softmax_experts": SoftmaxExpertMlp}


class TokenSide(nn.Module):
    """A layer's own input from the token: ``proj(gelu_tanh(gate x) * e)``, e the layer's part of the token's row in a table
    shared by the layers; its output is normed before it is added."""

    def __init__(self, cfg: LayeredArch, dtype, device):
        super().__init__()
        self.dim = cfg.side_dim
        self.gate = nn.Parameter(torch.empty(self.dim, cfg.hidden_size, dtype=dtype, device=device))
        self.proj = nn.Parameter(torch.empty(cfg.hidden_size, self.dim, dtype=dtype, device=device))
        self.norm = RmsNorm(cfg, device)

    def tensors(self, p):
        return {p + "gate": self.gate, p + "proj": self.proj, **self.norm.tensors(p + "norm")}

    def forward(self, h, ids, table, li: int):
        return mx.side_input(h, ids, table, li * self.dim, self.gate, self.proj)


class LayeredBlock(nn.Module):
    """Mixer and (optional) feed-forward around an fp32 residual stream; depending on the design with a norm on each sublayer's
    input (norm1, norm2), on its output (norm1b, norm2b in memory), or both, and a per-token input after them.  With ``beside``
    both read the same stream, and what is pending after the layer are both outputs."""

    def __init__(self, cfg: LayeredArch, spec: LayerSpec, dtype, device):
        super().__init__()
        design = DESIGNS[cfg.design]
        norm, none = NORMS[design.norm], lambda *_, **__: None
        pre, post = norm if design.pre_norm else none, norm if design.post_norm else none
        scale = dict(scale=True) if design.layer_scale else {}
        self.norm1, self.norm1b = pre(cfg, device), post(cfg, device, **scale)
        self.mixer = MIXERS[spec.kind](cfg, spec.mixer, dtype, device)
        self.norm2 = self.norm2b = self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.norm2b = pre(cfg, device), post(cfg, device, **scale)
            self.mlp = MLPS[design.moe if spec.mlp.get("kind") == "moe" else design.mlp](cfg, spec.mlp, dtype, device)
        self.side = TokenSide(cfg, dtype, device) if cfg.side_dim else None
        self.dtype, self.mult, self.beside = dtype, cfg.residual_mult, design.beside
        self.lora = nn.ModuleDict()
        self.lora_enabled = True

    def proj_slices(self):
        return {}  # adapters target the projections of the flat families

    def tensors(self, p):
        out = self.mixer.tensors(p + "mix.")
        if self.mlp is not None:
            out.update(self.mlp.tensors(p + "mlp."))
        for i, pre, post in (("1", self.norm1, self.norm1b), ("2", self.norm2, self.norm2b)):
            if pre is not None:
                out.update(pre.tensors(f"{p}norm{i}"))
            if post is not None:
                out.update(post.tensors(f"{p}norm{i}" if pre is None else f"{p}norm{i}b"))
                if post.scale is not None:
                    out[f"{p}ls{i}"] = post.scale
        if self.side is not None:
            out.update(self.side.tensors(p + "side."))
        return out

    def read_mixer(self, x, delta, post, **kw):
        """What the mixer reads, and the stream after the addition of the pending ``delta``."""
        return self._read(self.norm1, x, delta, post, **kw)

    def read_mlp(self, x, delta, post, **kw):
        return self._read(self.norm2, x, delta, post, **kw)

    def read_both(self, x, delta, post, **kw):
        """What mixer and feed-forward read (one of the two without a feed-forward) of the same stream."""
        if self.mlp is not None:
            kw["w2"] = self.norm2.weight
        h, x = self.norm1(x, self.dtype, delta, post, **kw)
        return (h if self.mlp is not None else (h, None)), x

    def read_side(self, x, delta, post, **kw):
        return self._read(None, x, delta, post, **kw)

    def _read(self, norm, x, delta, post, **kw):
        if norm is None:
            return RmsNorm.stream(x, self.dtype, delta, post, mult=self.mult, **kw)
        return norm(x, self.dtype, delta, post, **kw)

    def forward(self, x, delta, post, ctx: SeqCtx, li: int, ids=None, side_table=None, enter=None):
        """(residual, sublayer output not yet added to it, norm of that output) -> the same triple after this layer: every
        addition rides on the norm that follows it.  ``enter``: what a loop adds to the stream in front of this layer."""
        enter = enter or {}
        if self.beside:
            (h, h2), x = self.read_both(x, delta, post, **enter)
            delta = self.mixer(h, ctx, li)
            return x, (delta if h2 is None else (delta, self.mlp(h2, summed=False))), None
        h, x = self.read_mixer(x, delta, post, **enter)
        delta, post = self.mixer(h, ctx, li), self.norm1b
        if self.mlp is not None:
            h, x = self.read_mlp(x, delta, post)
            delta, post = self.mlp(h), self.norm2b
        if self.side is not None:
            h, x = self.read_side(x, delta, post)
            delta, post = self.side(h, ids, side_table, li), self.side.norm
        return x, delta, post


class LayeredLM(CausalLM):
    """Decoder of a layered design behind the :class:`CausalLM` interface (trainers, servers, engines)."""

    is_layered = True
    serves_float32 = True

    def __init__(self, cfg: LayeredArch, dtype=torch.float32, device=None, init: bool = True):
        nn.Module.__init__(self)
        if cfg.num_labels:
            raise NotImplementedError("layered designs have no classification head")
        self.config = cfg
        self.embed_tokens = nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device))
        design = DESIGNS[cfg.design]
        if cfg.passes and design.norm == "dynamic_tanh":
            raise NotImplementedError("a loop over layers with Dynamic-Tanh norms")
        self.embed_norm = NORMS[design.norm](cfg, device) if design.embed_norm else None
        self.loop_step = nn.Parameter(torch.zeros(cfg.passes, cfg.hidden_size, dtype=torch.float32, device=device)) if cfg.passes else None
        blocks: list[LayeredBlock] = []
        for i, s in enumerate(cfg.layers):  # a layer that borrows weights IS its owner's block at another place
            blocks.append(blocks[s.owner] if s.owner != i else LayeredBlock(cfg, s, dtype, device))
        self.layers = nn.ModuleList(blocks)
        # the head's scale rides on the norm in front of it
        self.norm = NORMS[DESIGNS[cfg.design].norm](cfg, device, **(dict(gain=cfg.logit_scale) if cfg.logit_scale != 1.0 else {}))
        self.lm_head = None if cfg.tie_word_embeddings else nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device))
        self.side_embed = (nn.Parameter(torch.empty(cfg.vocab_size, cfg.side_dim * cfg.num_hidden_layers, dtype=dtype, device=device))
                           if cfg.side_dim else None)
        self.pair_embed = (nn.Parameter(torch.empty(cfg.pairs["buckets"] + 1, cfg.hidden_size, dtype=dtype, device=device))
                           if cfg.pairs else None)
        self.gradient_checkpointing = False
        self.name_or_path = ""
        self.generation_config = None
        self.warnings_issued = {}
        if init and str(device) != "meta":
            self.reset_parameters()

    @torch.no_grad()
    def reset_parameters(self, std: float = 0.02, generator: torch.Generator | None = None):
        for p in self.parameters():
            if p.ndim >= 2:
                p.normal_(0.0, std, generator=generator)

    def named_tensors(self) -> dict[str, torch.Tensor]:
        """Checkpoint name -> parameter or view into a fused parameter."""
        out = {"embed": self.embed_tokens}
        if self.embed_norm is not None:
            out.update(self.embed_norm.tensors("embed.norm"))
        if self.loop_step is not None:
            out["loop.step"] = self.loop_step
        if self.side_embed is not None:
            out["side.embed"] = self.side_embed
        if self.pair_embed is not None:
            out["bigram"] = self.pair_embed
        for i, (s, b) in enumerate(zip(self.config.layers, self.layers)):
            if s.owner == i:
                out.update(b.tensors(f"l{s.index}."))
        out.update(self.norm.tensors("final.norm"))
        if self.lm_head is not None:
            out["head"] = self.lm_head
        return out

    def resize_token_embeddings(self, new_size: int, pad_to_multiple_of: int | None = None):
        super().resize_token_embeddings(new_size, pad_to_multiple_of)
        if self.side_embed is not None and self.side_embed.shape[0] != self.config.vocab_size:
            old, n = self.side_embed, min(self.side_embed.shape[0], self.config.vocab_size)
            w = torch.empty(self.config.vocab_size, old.shape[1], dtype=old.dtype, device=old.device).normal_(0, 0.02)
            w[:n] = old.data[:n]
            self.side_embed = nn.Parameter(w)

    @torch.no_grad()
    def load_named_tensors(self, sd: dict[str, torch.Tensor], strict: bool = True) -> list[str]:
        mine = self.named_tensors()
        for name, dst in mine.items():
            if name not in sd:
                if strict:
                    raise KeyError(f"missing tensor {name} in checkpoint")
                continue
            if sd[name].shape != dst.shape:
                raise ValueError(f"{name}: {tuple(sd[name].shape)} in the checkpoint, {tuple(dst.shape)} by the config")
            dst.copy_(sd[name])
        return [k for k in sd if k not in mine]

    def embed(self, input_ids, ctx: SeqCtx | None = None):
        if self.embed_norm is not None:
            n = self.embed_norm
            return mx.embed_normed(input_ids.reshape(-1), self.embed_tokens, self.config.embed_scale, n.weight, n.eps, n.shift)
        if self.pair_embed is None:
            return mx.embed_scaled(input_ids, self.embed_tokens, self.config.embed_scale)
        if ctx is None:
            raise NotImplementedError("the embedding of this design depends on the tokens' positions in their sequences")
        where = ctx.kv.last_tokens() if ctx.kv is not None else {}
        return mx.embed_pairs(input_ids.reshape(-1), self.embed_tokens, self.config.embed_scale, self.pair_embed, self.config.pairs,
                              ctx.positions, where)

    def final_norm(self, x, delta=None, post=None):
        return self.norm(x, self.dtype, delta, post)[0]

    def forward_hidden(self, input_ids, ctx: SeqCtx, inputs_embeds=None):
        mx.check_can_run(self.embed_tokens)
        ctx = dataclasses.replace(ctx, shared=dict.fromkeys(self.config.lenders))
        ids = input_ids.reshape(-1)
        x, delta, post = (self.embed(input_ids, ctx) if inputs_embeds is None else inputs_embeds.float()), None, None
        first = x.clone() if self.config.passes > 1 else None  # the stream moves on in place
        for li, layer in enumerate(self.layers):
            x, delta, post = layer(x, delta, post, ctx, li, ids, self.side_embed, self.entrance(li, first))
        return self.final_norm(x, delta, post)

    def entrance(self, li: int, first) -> dict:
        """What the loop adds to the stream in front of layer run ``li``; ``first``: the embedding."""
        t = self.config.layers[li].enters
        return {} if t is None else dict(anchor=first if t > 0 else None, bump=self.loop_step[t])


def is_layered_dir(path: str) -> bool:
    f = os.path.join(path, "config.json")
    if not os.path.exists(f):
        return False
    with open(f) as fh:
        return json.load(fh).get("architecture") in DESIGNS


def layered_kinds(path: str) -> set:
    """Mixers and feed-forwards of a model directory whose kernels are built apart (csrc/build.py)."""
    with open(os.path.join(path, "config.json")) as fh:
        d = json.load(fh)
    layers = d["layers"]
    kinds = {e["type"] for e in layers} | {"moe" for e in layers if (e.get("mlp") or {}).get("kind") == "moe"}
    return kinds | (set(DESIGNS[d["architecture"]].sides) if "parallel" in kinds else set())
