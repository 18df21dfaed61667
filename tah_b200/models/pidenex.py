"""Pidenex: a small decoder of windowed attention, latent-attention and attention-beside-recurrence layers, some of which run
several times in a row.

This module reads the family's ``config.json`` into the specs of :mod:`tah_b200.models.layered` and says which tensors a
checkpoint has.  The mechanisms:

* layer norms (no bias) in front of and behind every sublayer; a range of layers is a loop whose passes add a vector of their
  own and, from the second on, the embedding output to the residual stream;
* attention: grouped heads whose values are the keys, a window, and the means of the key blocks in front of it as further keys;
* latent attention: queries through a latent, keys and values from one cached latent per token, a shared rotated key part, a
  window;
* parallel: attention with norms over the whole projections, raw keys as values, a distance bias per head and a full-width
  output gate, beside a minGRU recurrence;
* feed-forward: dense with the xIELU activation.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from tah_b200.models.layered import (AttentionSpec, BranchesSpec, LatentAttentionSpec, LayeredConfig, LayeredForCausalLM, LayerSpec,
                                     LoopSpec, MinGRUSpec, RotarySpec, XIELUSpec, check_attention, check_rotary)


def _size(m: dict, name: str) -> Optional[int]:
    v = (m.get("mask") or {}).get(name)
    return None if v is None else int(v)


def _attention(i: int, m: dict, **kw) -> AttentionSpec:
    s = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                      window=_size(m, "size"), pool=_size(m, "pool"), keys_as_values=True, **kw)
    check_attention(i, s, [])
    return s


def _mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        return _attention(i, m)
    if kind == "latent_attention":
        s = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                rotary=RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"]), interleaved=True),
                                window=_size(m, "size"), sink=False, gate=False)
        check_rotary(i, s.rotary, s.rot_dim)
        if s.rotary.dims != s.rot_dim:
            raise ValueError(f"layer {i}: rotation of {s.rotary.dims} dims in a rotated part of {s.rot_dim}")
        if s.window is not None and s.window < 1:
            raise ValueError(f"layer {i}: a window of {s.window} tokens")
        return s
    if kind == "parallel":
        return BranchesSpec(_attention(i, m["left"], slopes=True, norm_all=True, wide_gate=True), MinGRUSpec(int(m["right"]["width"])),
                            float(m["left_scale"]), float(m["right_scale"]))
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def _feed_forward(i: int, m):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {m['kind']!r}")
    return XIELUSpec(int(m["ff"]))


def _attention_dict(m: AttentionSpec) -> dict:
    d = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale)
    mask = {k: v for k, v in (("size", m.window), ("pool", m.pool)) if v is not None}
    return dict(d, mask=mask) if mask else d


@dataclass
class PidenexConfig(LayeredConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "PidenexConfig":
        layers = [LayerSpec(_mixer(i, e["type"], e["mixer"]), _feed_forward(i, e.get("mlp"))) for i, e in enumerate(d["layers"])]
        loop = None
        if d.get("loop"):
            loop = LoopSpec(*(int(d["loop"][k]) for k in ("start", "stop", "times")))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"{loop.times} passes over the layers {loop.start} .. {loop.stop} of {len(layers)}")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=float(d["embedding"]["scale"]),
                   rms_norm_eps=float(d["norm"]["eps"]), layers=layers, centered=True, layer_scale=False, loop=loop, raw=dict(d))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, AttentionSpec):
                mix = _attention_dict(m)
            elif isinstance(m, LatentAttentionSpec):
                mix = dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale,
                           rot=dict(base=m.rotary.base, dims=m.rotary.dims))
                if m.window is not None:
                    mix["mask"] = dict(size=m.window)
            else:
                mix = dict(left=_attention_dict(m.left), right=dict(width=m.right.width), left_scale=m.left_scale,
                           right_scale=m.right_scale)
            layers.append(dict(type=m.kind, mixer=mix, mlp=None if l.ff is None else dict(kind="dense", ff=l.ff.ff)))
        out = dict(architecture="Pidenex", vocab=self.vocab_size, width=self.hidden_size, embedding=dict(scale=self.embedding_scale),
                   norm=dict(eps=self.rms_norm_eps), layers=layers)
        if self.loop is not None:
            out["loop"] = dict(start=self.loop.start, stop=self.loop.stop, times=self.loop.times)
        return out

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, V = self.hidden_size, self.vocab_size
        out: Dict[str, Tuple[int, ...]] = {"embed": (V, W)}
        if self.loop is not None:
            out["loop.step"] = (self.loop.times, W)

        def attention(x, m):
            out[x + "q"], out[x + "k"], out[x + "o"] = (m.heads * m.dim, W), (m.kv_heads * m.dim, W), (W, m.heads * m.vdim)
            if m.norm_all:
                out[x + "q.norm"], out[x + "k.norm"] = (m.heads * m.dim,), (m.kv_heads * m.dim,)
            if m.wide_gate:
                out[x + "g"] = (m.heads * m.vdim, W)

        for i, l in enumerate(self.layers):
            m, x, y = l.mixer, f"l{i}.mix.", f"l{i}.mlp."
            for q in (1,) if l.ff is None else (1, 2):
                out[f"l{i}.norm{q}"] = out[f"l{i}.norm{q}b"] = (W,)
            if isinstance(m, AttentionSpec):
                attention(x, m)
            elif isinstance(m, LatentAttentionSpec):
                out[x + "dq"], out[x + "dq.norm"] = (m.q_rank, W), (m.q_rank,)
                out[x + "uq"] = (m.heads * (m.dim + m.rot_dim), m.q_rank)
                out[x + "dkv"], out[x + "dkv.norm"] = (m.kv_rank + m.rot_dim, W), (m.kv_rank,)
                out[x + "uk"], out[x + "uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
                out[x + "o"] = (W, m.heads * m.vdim)
            else:
                attention(x + "left.", m.left)
                D, r = m.right.width, x + "right."
                out[r + "z"], out[r + "z.b"], out[r + "x"], out[r + "x.b"] = (D, W), (D,), (D, W), (D,)
                out[r + "g"], out[r + "o"] = (D, W), (W, D)
            if l.ff is not None:
                out[y + "up"], out[y + "down"], out[y + "act"] = (l.ff.ff, W), (W, l.ff.ff), (2,)
        out["final.norm"], out["head"] = (W,), (V, W)
        return out


class PidenexForCausalLM(LayeredForCausalLM):
    config_class = PidenexConfig

    @classmethod
    def _adapt(cls, cfg, tensors) -> None:
        if cfg.loop is None:                             # what a checkpoint may still hold for absent parts is unused
            tensors.pop("loop.step", None)
        for i, l in enumerate(cfg.layers):
            if l.ff is None:
                for n in ("norm2", "norm2b"):
                    tensors.pop(f"l{i}.{n}", None)

    @torch.no_grad()
    def init_random(self, seed: int = 0) -> "PidenexForCausalLM":
        """Random weights of sensible size (benchmarks, tests): unit-variance projections, norms of one, slow recurrences."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for key, p in self.weights.items():
            name = key.rsplit("/", 1)[-1]
            if name == "embed":
                p.normal_(std=1.0 / self.config.embedding_scale, generator=g)
            elif name == "step":
                p.normal_(std=0.3, generator=g)
            elif name == "act":
                p.copy_(torch.tensor([0.5, 0.2]))
            elif p.dim() == 2:
                p.normal_(std=1.0 / math.sqrt(p.shape[1]), generator=g)
            else:
                p.fill_(-3.0 if key.endswith("z/b") else 0.0 if name == "b" else 1.0)
        return self


def pidenex_preset(name: str) -> PidenexConfig:
    """Configurations for benchmarks with the layer sizes of the Qwen3-1.7B backbone.  ``pidenex-1.7b``: of every four layers two
    are attention, one latent attention and one parallel, 28 layer runs of which the middle 16 are two passes over eight layers;
    ``pidenex-flat``: the same 28 runs as layers of their own."""
    def build(vocab, width, kinds, ff, attn, latent, left, D, loop=None):
        mix = dict(attention=attn, latent_attention=latent, parallel=dict(left=left, right=dict(width=D), left_scale=0.7, right_scale=0.6))
        layers: List[dict] = [dict(type=k, mixer=mix[k], mlp=dict(kind="dense", ff=ff)) for k in kinds]
        return PidenexConfig.from_dict(dict(architecture="Pidenex", vocab=vocab, width=width, embedding=dict(scale=1.0), norm=dict(eps=1e-6),
                                            layers=layers, loop=loop))

    group = ["attention", "parallel", "attention", "latent_attention"]
    if name in ("pidenex-1.7b", "pidenex-flat"):
        heads = dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5)
        loop = dict(start=4, stop=12, times=2) if name == "pidenex-1.7b" else None
        return build(151936, 2048, group * (5 if loop else 7), 9216, dict(heads, mask=dict(size=1024, pool=16)),
                     dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512, scale=192 ** -0.5, rot=dict(dims=64, base=1e4),
                          mask=dict(size=1024)),
                     dict(heads, mask=dict(size=1024)), 2048, loop)
    if name == "pidenex-tiny":
        return build(300, 160, group, 208, dict(heads=6, kv_heads=2, dim=40, vdim=40, scale=0.2, mask=dict(size=21, pool=5)),
                     dict(heads=3, dim=24, rot_dim=12, vdim=40, q_rank=56, kv_rank=48, scale=0.16, rot=dict(dims=12, base=2e3), mask=dict(size=13)),
                     dict(heads=4, kv_heads=2, dim=24, vdim=24, scale=0.2, mask=dict(size=17)), 72, dict(start=1, stop=3, times=2))
    raise KeyError(name)
