"""Decoders described layer by layer.

The flat families of :mod:`trl_b200.models.configuration` repeat one block.  A *layered* design instead lists its
layers in ``config.json``, each with a mixer (kind and sizes) and a feed-forward (or none), and a layer may run with
another layer's weights.  :data:`DESIGNS` registers what a design fixes (norm, activation); everything else is read
from the file.  A mixer is a module here (parameters, tensor names, prompt forward) with its kernels in
``csrc/mixers.cu`` and its decode state in ``rollout/layered_engine.py``; registering another kind in :data:`MIXERS`
makes it available to every layered design.

Designs
    Zorelorn    embeddings times a constant, Dynamic-Tanh norms, ``latent_attention`` (multi-head latent attention with
                YaRN rotary part, sliding window, softmax sink, per-head output gate) and ``mlstm`` (matrix memory with
                exponential gates) mixers, erf-GELU feed-forward.

The residual stream, norms, gates and recurrent states are fp32 whatever the model dtype.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Any

import torch
import torch.nn as nn

from ..ops import mixers as mx
from .configuration import ModelArch
from .decoder import CausalLM, SeqCtx


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models."""

    norm: str = "dynamic_tanh"
    mlp_act: str = "gelu"


DESIGNS: dict[str, Design] = {"Zorelorn": Design()}


@dataclass
class LayerSpec:
    """One entry of the layer list.  ``owner``: index of the layer whose tensors this one runs with (itself, usually)."""

    kind: str
    mixer: dict
    ff: int | None
    owner: int

    @property
    def key(self):
        return (self.kind, json.dumps(self.mixer, sort_keys=True), self.ff)


@dataclass
class LayeredArch(ModelArch):
    design: str = ""
    layers: list = field(default_factory=list)  # [LayerSpec]
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
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not supported")
            owner = i
            if e.get("weights_of") is not None:
                j = int(e["weights_of"])
                if not 0 <= j < i:
                    raise ValueError(f"layer {i}: weights_of={j} must name an earlier layer")
                owner = specs[j].owner
            s = LayerSpec(e["type"], dict(e["mixer"]), None if mlp is None else int(mlp["ff"]), owner)
            if owner != i and s.key != specs[owner].key:
                raise ValueError(f"layer {i} runs with the weights of layer {owner} but is described differently")
            specs.append(s)
        heads = max((s.mixer.get("heads", 1) for s in specs), default=1)
        return cls(model_type=name.lower(), design=name, vocab_size=d["vocab"], hidden_size=d["width"],
                   intermediate_size=max((s.ff or 0 for s in specs), default=0), num_hidden_layers=len(specs),
                   num_attention_heads=heads, num_key_value_heads=heads, rms_norm_eps=float(d["norm"]["eps"]),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), layers=specs, source=copy.deepcopy(d),
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
        return n - (2 * self.vocab_size * self.hidden_size if exclude_embeddings else 0)


def _vec(n=None, fill=0.0, device=None):
    """Small per-channel parameters are fp32 in every model dtype: the kernels read them as such."""
    shape = () if n is None else (n,)
    return nn.Parameter(torch.full(shape, float(fill), dtype=torch.float32, device=device))


class DynamicTanh(nn.Module):
    """``tanh(alpha x) w + b``: a norm without statistics."""

    def __init__(self, n, device=None):
        super().__init__()
        self.weight, self.bias, self.alpha = _vec(n, 1.0, device), _vec(n, 0.0, device), _vec(None, 0.5, device)

    def tensors(self, name):
        return {name: self.weight, name + ".b": self.bias, name + ".alpha": self.alpha}

    def forward(self, x, out_dtype, delta=None):
        """x [T, H] fp32 (``delta``, when given, is added to it in place first) -> [T, H] ``out_dtype``."""
        return mx.dynamic_tanh(x, delta, self.alpha, self.weight, self.bias, out_dtype)


NORMS = {"dynamic_tanh": DynamicTanh}


class LatentAttention(nn.Module):
    """Multi-head latent attention: keys and values of all heads are linear in one latent per token (plus one rotated
    key part shared by the heads), and only those are cached.  In memory the projections that read the layer input are
    one matrix (query latent | key/value latent | rotated key | gate), as are the key and value up-projections."""

    kind = "latent_attention"

    def __init__(self, cfg: LayeredArch, m: dict, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.eps = cfg.rms_norm_eps
        self.heads, self.dim, self.rot_dim, self.vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        self.q_rank, self.kv_rank = m["q_rank"], m["kv_rank"]
        self.scale = float(m["scale"])
        mask = m.get("mask") or {}
        self.window = int(mask["size"]) if mask.get("size") else None
        rot = m["rot"]
        if rot["dims"] != self.rot_dim or self.rot_dim % 2:
            raise ValueError("latent_attention rotates its whole rot_dim part, in pairs")
        self.rope = mx.RotarySpec(self.rot_dim, float(rot["base"]), rot.get("scaling"))
        h = cfg.hidden_size
        self.w_in = nn.Parameter(torch.empty(self.q_rank + self.kv_rank + self.rot_dim + self.heads, h, **kw))
        self.uq = nn.Parameter(torch.empty(self.heads * (self.dim + self.rot_dim), self.q_rank, **kw))
        self.ukv = nn.Parameter(torch.empty(self.heads * (self.dim + self.vdim), self.kv_rank, **kw))
        self.o = nn.Parameter(torch.empty(h, self.heads * self.vdim, **kw))
        self.q_norm, self.kv_norm = _vec(self.q_rank, 1.0, device), _vec(self.kv_rank, 1.0, device)
        self.sink = _vec(self.heads, 0.0, device)

    @property
    def uk(self):
        return self.ukv[: self.heads * self.dim]

    @property
    def uv(self):
        return self.ukv[self.heads * self.dim:]

    def tensors(self, p):
        a, b = self.q_rank, self.q_rank + self.kv_rank + self.rot_dim
        return {p + "dq": self.w_in[:a], p + "dq.norm": self.q_norm, p + "uq": self.uq, p + "dkv": self.w_in[a:b],
                p + "dkv.norm": self.kv_norm, p + "uk": self.uk, p + "uv": self.uv, p + "sink": self.sink,
                p + "g": self.w_in[b:], p + "o": self.o}

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


MIXERS = {c.kind: c for c in (LatentAttention, MLstm)}


class DenseMlp(nn.Module):
    """``down(act(up x))`` with the exact GELU."""

    def __init__(self, cfg: LayeredArch, ff: int, dtype, device):
        super().__init__()
        self.up = nn.Parameter(torch.empty(ff, cfg.hidden_size, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.empty(cfg.hidden_size, ff, dtype=dtype, device=device))

    def tensors(self, p):
        return {p + "up": self.up, p + "down": self.down}

    def forward(self, h):
        return mx.linear_f32(mx.gelu_linear(h, self.up), self.down)


class LayeredBlock(nn.Module):
    """Pre-norm mixer and (optional) feed-forward around an fp32 residual stream."""

    def __init__(self, cfg: LayeredArch, spec: LayerSpec, dtype, device):
        super().__init__()
        norm = NORMS[DESIGNS[cfg.design].norm]
        self.norm1 = norm(cfg.hidden_size, device)
        self.mixer = MIXERS[spec.kind](cfg, spec.mixer, dtype, device)
        self.norm2 = norm(cfg.hidden_size, device) if spec.ff is not None else None
        self.mlp = DenseMlp(cfg, spec.ff, dtype, device) if spec.ff is not None else None
        self.dtype = dtype
        self.lora = nn.ModuleDict()
        self.lora_enabled = True

    def proj_slices(self):
        return {}  # adapters target the projections of the flat families

    def tensors(self, p):
        out = {**self.norm1.tensors(p + "norm1"), **self.mixer.tensors(p + "mix.")}
        if self.mlp is not None:
            out.update({**self.norm2.tensors(p + "norm2"), **self.mlp.tensors(p + "mlp.")})
        return out

    def forward(self, x, delta, ctx: SeqCtx, li: int):
        """(residual, block output not yet added to it) -> the same pair after this layer: every addition rides on the
        norm that follows it."""
        h, x = self.norm1(x, self.dtype, delta)
        delta = self.mixer(h, ctx, li)
        if self.mlp is not None:
            h, x = self.norm2(x, self.dtype, delta)
            delta = self.mlp(h)
        return x, delta


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
        blocks: list[LayeredBlock] = []
        for i, s in enumerate(cfg.layers):  # a layer that borrows weights IS its owner's block at another place
            blocks.append(blocks[s.owner] if s.owner != i else LayeredBlock(cfg, s, dtype, device))
        self.layers = nn.ModuleList(blocks)
        self.norm = NORMS[DESIGNS[cfg.design].norm](cfg.hidden_size, device)
        self.lm_head = nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device))
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
        for i, (s, b) in enumerate(zip(self.config.layers, self.layers)):
            if s.owner == i:
                out.update(b.tensors(f"l{i}."))
        out.update(self.norm.tensors("final.norm"))
        out["head"] = self.lm_head
        return out

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

    def embed(self, input_ids):
        return mx.embed_scaled(input_ids, self.embed_tokens, self.config.embed_scale)

    def final_norm(self, x, delta=None):
        return self.norm(x, self.dtype, delta)[0]

    def forward_hidden(self, input_ids, ctx: SeqCtx, inputs_embeds=None):
        mx.check_can_run(self.embed_tokens)
        x, delta = (self.embed(input_ids) if inputs_embeds is None else inputs_embeds.float()), None
        for li, layer in enumerate(self.layers):
            x, delta = layer(x, delta, ctx, li)
        return self.final_norm(x, delta)


def is_layered_dir(path: str) -> bool:
    f = os.path.join(path, "config.json")
    if not os.path.exists(f):
        return False
    with open(f) as fh:
        return json.load(fh).get("architecture") in DESIGNS
