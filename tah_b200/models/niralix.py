"""Niralix: a small decoder of attention, latent-attention and gated-linear-attention layers on hyper-connected residual streams.

This module reads the family's ``config.json`` into the specs of :mod:`tah_b200.models.layered` and says which tensors a
checkpoint has.  The mechanisms:

* several residual streams that every sublayer reads through one learned vector and writes through another, mixing the
  streams on the way; RMS norms in front of the sublayers with weights stored around zero;
* attention: grouped heads with separate q/k and v sizes, projection biases, rotary positions on part of a head (YaRN
  scaling), values mixed with those of the first attention layer that mixes;
* latent attention: queries through a latent, keys and values from one cached latent per token, a shared rotated key part, a
  softmax sink per head, a full-width output gate;
* gla: gated linear attention with a decay per key channel from a low-rank projection;
* feed-forward: SwiGLU, dense or a mixture of experts (softmax router, the score on the expert's output);
* the embedding table is the output projection, logits times ``logit_scale``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from tah_b200.models.layered import (AttentionSpec, ExpertSpec, GLASpec, LatentAttentionSpec, LayeredConfig, LayeredForCausalLM,
                                     LayerSpec, MixtureSpec, RotarySpec, SwiGLUSpec, YarnSpec, check_attention, check_rotary)


def _rotary(r: Optional[dict], interleaved: bool) -> Optional[RotarySpec]:
    if not r:
        return None
    y = r.get("scaling")
    return RotarySpec(dims=int(r["dims"]), base=float(r["base"]), interleaved=interleaved,
                      yarn=None if not y else YarnSpec(factor=float(y["factor"]), original=float(y["original"]), fast=float(y["fast"]),
                                                       slow=float(y["slow"])))


def _rotary_dict(r: RotarySpec) -> dict:
    d = dict(base=r.base, dims=r.dims)
    if r.yarn is not None:
        d["scaling"] = dict(factor=r.yarn.factor, original=r.yarn.original, fast=r.yarn.fast, slow=r.yarn.slow)
    return d


def _mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        return AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                             scale=float(m["scale"]), proj_bias=True, out_bias=True, rotary=_rotary(m.get("rot"), False),
                             v_mix=bool(m.get("v_mix")))
    if kind == "latent_attention":
        s = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                rotary=_rotary(m["rot"], True))
        check_rotary(i, s.rotary, s.rot_dim)
        if s.rotary.dims != s.rot_dim:
            raise ValueError(f"layer {i}: rotation of {s.rotary.dims} dims in a rotated part of {s.rot_dim}")
        return s
    if kind == "gla":
        s = GLASpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
        if not s.tau > 0:
            raise ValueError(f"layer {i}: decay exponent 1 / {s.tau}")
        return s
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def _feed_forward(i: int, m):
    if m is None:
        return None
    if m["kind"] == "dense":
        return SwiGLUSpec(int(m["ff"]))
    if m["kind"] == "moe":
        ff = MixtureSpec(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]),
                         expert=ExpertSpec(int(m["expert"]["ff"]), slope=1.0, offset=0.0), softmax=True, weight_output=True)
        if not 1 <= ff.top <= ff.experts:
            raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts")
        return ff
    raise ValueError(f"layer {i}: unknown feed-forward kind {m['kind']!r}")


@dataclass
class NiralixConfig(LayeredConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "NiralixConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            mixer = _mixer(i, e["type"], e["mixer"])
            if isinstance(mixer, AttentionSpec):
                check_attention(i, mixer, layers)
            layers.append(LayerSpec(mixer, _feed_forward(i, e.get("mlp"))))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=1.0, rms_norm_eps=float(d["norm"]["eps"]),
                   layers=layers, logit_scale=float(d["logit_scale"]), norm_offset=1.0, streams=int(d["streams"]), tied_head=True,
                   raw=dict(d))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m, f = l.mixer, l.ff
            if isinstance(m, AttentionSpec):
                mix = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, v_mix=m.v_mix)
                if m.rotary is not None:
                    mix["rot"] = _rotary_dict(m.rotary)
            elif isinstance(m, LatentAttentionSpec):
                mix = dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale,
                           rot=_rotary_dict(m.rotary))
            else:
                mix = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, tau=m.tau)
            if f is None:
                mlp = None
            elif isinstance(f, SwiGLUSpec):
                mlp = dict(kind="dense", ff=f.ff)
            else:
                mlp = dict(kind="moe", router=dict(experts=f.experts, top=f.top), expert=dict(ff=f.expert.ff))
            layers.append(dict(type=m.kind, mixer=mix, mlp=mlp))
        return dict(architecture="Niralix", vocab=self.vocab_size, width=self.hidden_size, streams=self.streams,
                    logit_scale=self.logit_scale, norm=dict(eps=self.rms_norm_eps), layers=layers)

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, V, S = self.hidden_size, self.vocab_size, self.streams
        out: Dict[str, Tuple[int, ...]] = {"embed": (V, W)}

        def unit(p, ff):
            out[p + "gate"] = out[p + "up"] = (ff, W)
            out[p + "down"] = (W, ff)

        for i, l in enumerate(self.layers):
            m, f, x, y = l.mixer, l.ff, f"l{i}.mix.", f"l{i}.mlp."
            for q in (1,) if f is None else (1, 2):
                out[f"l{i}.norm{q}"] = (W,)
                out[f"l{i}.hc{q}.in"] = out[f"l{i}.hc{q}.out"] = (S,)
                out[f"l{i}.hc{q}.mix"] = (S, S)
            if isinstance(m, AttentionSpec):
                for n, rows, cols in (("q", m.heads * m.dim, W), ("k", m.kv_heads * m.dim, W), ("v", m.kv_heads * m.vdim, W),
                                      ("o", W, m.heads * m.vdim)):
                    out[x + n], out[x + n + ".b"] = (rows, cols), (rows,)
                if m.v_mix:
                    out[x + "vmix"] = ()
            elif isinstance(m, LatentAttentionSpec):
                out[x + "dq"], out[x + "dq.norm"] = (m.q_rank, W), (m.q_rank,)
                out[x + "uq"] = (m.heads * (m.dim + m.rot_dim), m.q_rank)
                out[x + "dkv"], out[x + "dkv.norm"] = (m.kv_rank + m.rot_dim, W), (m.kv_rank,)
                out[x + "uk"], out[x + "uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
                out[x + "sink"], out[x + "g"], out[x + "o"] = (m.heads,), (m.heads * m.vdim, W), (W, m.heads * m.vdim)
            else:
                for n, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
                    out[x + n] = (rows, W)
                out[x + "o"], out[x + "norm"] = (W, m.heads * m.vdim), (m.vdim,)
                out[x + "a1"], out[x + "a2"], out[x + "a2.b"] = (m.rank, W), (m.heads * m.dim, m.rank), (m.heads * m.dim,)
            if isinstance(f, SwiGLUSpec):
                unit(y, f.ff)
            elif isinstance(f, MixtureSpec):
                for e in range(f.experts):
                    unit(f"{y}e{e}.", f.expert.ff)
                out[y + "router"] = (f.experts, W)
        out["final.norm"] = (W,)
        return out


class NiralixForCausalLM(LayeredForCausalLM):
    config_class = NiralixConfig

    @classmethod
    def _adapt(cls, cfg, tensors) -> None:
        for i, l in enumerate(cfg.layers):
            if isinstance(l.mixer, GLASpec):
                l.mixer.rank = int(tensors[f"l{i}.mix.a1"].shape[0])
            if l.ff is None:                             # what a checkpoint may still hold for the absent sublayer is unused
                for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix"):
                    tensors.pop(f"l{i}.{n}", None)

    @torch.no_grad()
    def init_random(self, seed: int = 0) -> "NiralixForCausalLM":
        """Random weights of sensible size (benchmarks, tests): unit-variance projections, norms of one, streams that stay apart."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for key, p in self.weights.items():
            parts = key.split("/")
            name, hc = parts[-1], parts[-2] if len(parts) > 1 else ""
            if hc.startswith("hc"):
                S = self.config.streams
                if name == "mix":
                    p.copy_(torch.eye(S) * 0.9 + 0.1 / S)
                else:
                    p.copy_(torch.linspace(0.5, 1.5, S) / (S if name == "in" else 1))
            elif name == "embed":
                p.normal_(generator=g)
            elif name in ("norm1", "norm2") or hc == "final":
                p.zero_()
            elif name == "norm":
                p.fill_(1.0)
            elif name == "vmix":
                p.fill_(0.3)
            elif key.endswith("a2/b"):
                p.fill_(2.0)
            elif p.dim() == 2:
                p.normal_(std=1.0 / math.sqrt(p.shape[1]), generator=g)
        return self


def niralix_preset(name: str) -> NiralixConfig:
    """Configurations for benchmarks with the layer sizes of the Qwen3-1.7B backbone: ``niralix-1.7b`` has dense layers only,
    ``niralix-moe`` 64 experts in every layer but the first, 8 of them per token.  In both, every group of four layers is two
    latent-attention layers, an attention layer and a gla layer."""
    def build(vocab, width, n, streams, attn, latent, gla, dense, moe=None):
        layers = []
        for i in range(n):
            kind, mix = (("attention", attn), ("latent_attention", latent), ("gla", gla), ("latent_attention", latent))[i % 4]
            mlp = dict(kind="dense", ff=dense) if moe is None or i == 0 else dict(kind="moe", **moe)
            layers.append(dict(type=kind, mixer=mix, mlp=mlp))
        return NiralixConfig.from_dict(dict(architecture="Niralix", vocab=vocab, width=width, streams=streams, logit_scale=0.5,
                                            norm=dict(eps=1e-6), layers=layers))

    yarn = dict(factor=4.0, original=4096, fast=32.0, slow=1.0)
    attn = dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, v_mix=True, rot=dict(dims=64, base=1e6, scaling=yarn))
    latent = dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512, scale=192 ** -0.5, rot=dict(dims=64, base=1e4))
    gla = dict(heads=8, dim=128, vdim=256, tau=16.0)
    if name == "niralix-1.7b":
        return build(151936, 2048, 28, 2, attn, latent, gla, 6144)
    if name == "niralix-moe":
        return build(151936, 2048, 28, 2, attn, latent, gla, 6144, dict(router=dict(experts=64, top=8), expert=dict(ff=768)))
    if name == "niralix-tiny":
        return build(300, 160, 4, 3, dict(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.2, v_mix=True, rot=dict(dims=20, base=5e3, scaling=yarn)),
                     dict(heads=3, dim=24, rot_dim=12, vdim=40, q_rank=56, kv_rank=48, scale=0.16, rot=dict(dims=12, base=2e3)),
                     dict(heads=5, dim=24, vdim=48, tau=9.0), 208, dict(router=dict(experts=5, top=2), expert=dict(ff=72)))
    raise KeyError(name)
