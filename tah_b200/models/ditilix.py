"""Ditilix: a small decoder whose layers run attention and feed-forward in parallel, most of them a mixture of experts.

This module reads the family's ``config.json`` into the specs of :mod:`tah_b200.models.layered` and says which tensors a
checkpoint has.  The mechanisms:

* sinusoidal positions added to the embedding; RMS norms over equal groups of the hidden vector;
* layer: one norm feeds the mixer and the feed-forward, their sum times ``residual_mult`` joins the residual stream;
* attention: grouped heads with separate q/k and v sizes, no biases and no rotation, a query temperature that grows with
  the logarithm of the position, a tanh cap on the scores, and optionally the keys and values of another layer;
* feed-forward: dense with the PolyNorm activation, or a mixture of clamped gated units (sigmoid router, the score on the
  expert's input, an optional gated shared expert);
* logits times ``logit_scale``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Tuple

import torch

from tah_b200.models.layered import (AttentionSpec, ExpertSpec, LayeredConfig, LayeredForCausalLM, LayerSpec, MixtureSpec,
                                     PolyNormSpec, check_attention)


def _number(v):
    """A number of config.json as it stands there (whole numbers stay whole)."""
    return int(v) if float(v) == int(v) else float(v)


def _attention(m: dict) -> AttentionSpec:
    t = m.get("q_temp")
    return AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         scale=float(m["scale"]), softcap=None if m.get("softcap") is None else float(m["softcap"]),
                         q_temp=None if t is None else (float(t["coef"]), _number(t["every"])),
                         kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))


def _expert(e: dict) -> ExpertSpec:
    return ExpertSpec(ff=int(e["ff"]), limit=float(e["limit"]))


def _feed_forward(i: int, m):
    if m is None:
        return None
    if m["kind"] == "dense":
        return PolyNormSpec(int(m["ff"]))
    if m["kind"] == "moe":
        ff = MixtureSpec(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), expert=_expert(m["expert"]),
                         shared=None if m.get("shared") is None else _expert(m["shared"]))
        if not 1 <= ff.top <= ff.experts:
            raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts")
        return ff
    raise ValueError(f"layer {i}: unknown feed-forward kind {m['kind']!r}")


@dataclass
class DitilixConfig(LayeredConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "DitilixConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mixer = _attention(e["mixer"])
            check_attention(i, mixer, layers)
            layers.append(LayerSpec(mixer, _feed_forward(i, e.get("mlp")), parallel=True))
        groups = int(d["norm"]["groups"])
        if groups < 1 or int(d["width"]) % groups:
            raise ValueError(f"a width of {d['width']} does not split into {groups} norm groups")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=1.0,
                   rms_norm_eps=float(d["norm"]["eps"]), layers=layers, norm_groups=groups, sinusoidal=True,
                   residual_mult=float(d["residual_mult"]), logit_scale=float(d["logit_scale"]), raw=dict(d))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m, f = l.mixer, l.ff
            mix = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale)
            if m.softcap is not None:
                mix["softcap"] = m.softcap
            if m.q_temp is not None:
                mix["q_temp"] = dict(coef=m.q_temp[0], every=m.q_temp[1])
            if m.kv_from is not None:
                mix["kv_from"] = m.kv_from
            if f is None:
                mlp = None
            elif isinstance(f, PolyNormSpec):
                mlp = dict(kind="dense", ff=f.ff)
            else:
                mlp = dict(kind="moe", router=dict(experts=f.experts, top=f.top), expert=dict(ff=f.expert.ff, limit=f.expert.limit))
                if f.shared is not None:
                    mlp["shared"] = dict(ff=f.shared.ff, limit=f.shared.limit)
            layers.append(dict(type=m.kind, mixer=mix, mlp=mlp))
        return dict(architecture="Ditilix", vocab=self.vocab_size, width=self.hidden_size, residual_mult=self.residual_mult,
                    logit_scale=self.logit_scale, norm=dict(eps=self.rms_norm_eps, groups=self.norm_groups), layers=layers)

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, V = self.hidden_size, self.vocab_size
        out: Dict[str, Tuple[int, ...]] = {"embed": (V, W)}

        def unit(p, ff):
            out[p + "gate"] = out[p + "up"] = (ff, W)
            out[p + "down"] = (W, ff)

        for i, l in enumerate(self.layers):
            m, f, x, y = l.mixer, l.ff, f"l{i}.mix.", f"l{i}.mlp."
            out[f"l{i}.norm1"] = (W,)
            out[x + "q"] = (m.heads * m.dim, W)
            if m.kv_from is None:
                out[x + "k"], out[x + "v"] = (m.kv_heads * m.dim, W), (m.kv_heads * m.vdim, W)
            out[x + "o"] = (W, m.heads * m.vdim)
            if isinstance(f, PolyNormSpec):
                out[y + "up"], out[y + "down"], out[y + "act"] = (f.ff, W), (W, f.ff), (4,)
            elif isinstance(f, MixtureSpec):
                for e in range(f.experts):
                    unit(f"{y}e{e}.", f.expert.ff)
                out[y + "router"] = (f.experts, W)
                if f.shared is not None:
                    unit(y + "shared.", f.shared.ff)
                    out[y + "shared.sg"] = (1, W)
        out["final.norm"], out["head"] = (W,), (V, W)
        return out


class DitilixForCausalLM(LayeredForCausalLM):
    config_class = DitilixConfig

    @torch.no_grad()
    def init_random(self, seed: int = 0) -> "DitilixForCausalLM":
        """Random weights of sensible size (benchmarks, tests): unit-variance projections, norms of one."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for key, p in self.weights.items():
            name = key.rsplit("/", 1)[-1]
            if name == "embed":
                p.normal_(generator=g)
            elif name == "act":
                p.copy_(torch.tensor([0.6, -0.4, 0.3, 0.1]))
            elif p.dim() == 2:
                p.normal_(std=1.0 / math.sqrt(p.shape[1]), generator=g)
            else:
                p.fill_(1.0)
        return self


def ditilix_preset(name: str) -> DitilixConfig:
    """Configurations for benchmarks with the layer sizes of the Qwen3-1.7B backbone: ``ditilix-1.7b`` has dense layers only
    (feed-forwards of as many parameters as a SwiGLU of 6144), ``ditilix-moe`` a dense first layer and 64 experts behind it,
    8 of them and a shared one per token.  Every fourth layer reads the keys of the one before it."""
    def build(vocab, width, n, heads, kv_heads, dim, groups, dense, moe=None):
        layers = []
        for i in range(n):
            mix = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, softcap=30.0,
                       q_temp=dict(coef=0.1, every=2048))
            if i % 4 == 3:
                mix["kv_from"] = i - 1
            mlp = dict(kind="dense", ff=dense) if moe is None or i == 0 else dict(kind="moe", **moe)
            layers.append(dict(type="attention", mixer=mix, mlp=mlp))
        return DitilixConfig.from_dict(dict(architecture="Ditilix", vocab=vocab, width=width, residual_mult=0.5, logit_scale=0.5,
                                            norm=dict(eps=1e-6, groups=groups), layers=layers))

    if name == "ditilix-1.7b":
        return build(151936, 2048, 28, 16, 8, 128, 4, 9216)
    if name == "ditilix-moe":
        return build(151936, 2048, 28, 16, 8, 128, 4, 9216, dict(router=dict(experts=64, top=8), expert=dict(ff=768, limit=7.0),
                                                                 shared=dict(ff=768, limit=7.0)))
    if name == "ditilix-tiny":
        return build(300, 160, 4, 6, 2, 40, 5, 208, dict(router=dict(experts=5, top=2), expert=dict(ff=72, limit=1.1),
                                                         shared=dict(ff=48, limit=0.9)))
    raise KeyError(name)
