"""Gunuvik: a small decoder that mixes windowed attention layers with matrix-memory recurrent (mLSTM) layers.

``config.json`` lists the layers one by one; every entry names its mixer (``attention`` or ``mlstm``), the mixer's sizes
and constants, and its feed-forward (or ``null``).  This module reads that configuration into typed specs and holds the
weights under their on-disk names; the computation is the engine's (:mod:`tah_b200.engine.hybrid`), whose mechanisms take
all of these values as parameters:

* layer: RMS norm before and after each sublayer and a learned per-channel layer scale on the sublayer's result;
* attention: grouped heads with separate q/k and v sizes, projection biases, per-head q/k norm, no rotation, a learned
  bias per (logarithmic) distance bucket and head, a sliding window with kept first tokens, a softmax sink per head, one
  output-gate number per head, and optionally the keys and values of another layer (``kv_from``);
* mlstm: matrix memory with exponential input and sigmoid forget gates (soft-capped), per-head output norm and a
  full-width output gate;
* feed-forward: SwiGLU.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Tuple

import torch

from tah_b200.models.layered import (AttentionSpec, LayeredConfig, LayeredForCausalLM, LayerSpec, MLSTMSpec, SwiGLUSpec,
                                     check_attention)


def _attention(**kw) -> AttentionSpec:
    """An attention spec with the mechanisms every attention layer of the design has."""
    return AttentionSpec(proj_bias=True, qk_norm=True, sink=True, head_gate=True, **kw)


@dataclass
class GunuvikConfig(LayeredConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "GunuvikConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            m = e["mixer"]
            if e["type"] == "attention":
                mask = m.get("mask") or {}
                mixer = _attention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                                   vdim=int(m["vdim"]), scale=float(m["scale"]), bias_max=int(m["bias_max"]),
                                   window=None if mask.get("size") is None else int(mask["size"]),
                                   keep_first=int(mask.get("keep_first") or 0),
                                   kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
                check_attention(i, mixer, layers)
            elif e["type"] == "mlstm":
                mixer = MLSTMSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerSpec(mixer, None if mlp is None else SwiGLUSpec(int(mlp["ff"]))))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=float(d["embedding"]["scale"]),
                   rms_norm_eps=float(d["norm"]["eps"]), layers=layers, raw=dict(d))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, AttentionSpec):
                mix = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, bias_max=m.bias_max)
                if m.window is not None or m.keep_first:
                    mix["mask"] = dict(size=m.window, keep_first=m.keep_first)
                if m.kv_from is not None:
                    mix["kv_from"] = m.kv_from
            else:
                mix = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, gate_cap=m.gate_cap)
            layers.append(dict(type=m.kind, mixer=mix, mlp=None if l.ff is None else dict(kind="dense", ff=l.ff.ff)))
        return dict(architecture="Gunuvik", vocab=self.vocab_size, width=self.hidden_size,
                    embedding=dict(scale=self.embedding_scale), norm=dict(eps=self.rms_norm_eps), layers=layers)

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, V = self.hidden_size, self.vocab_size
        out: Dict[str, Tuple[int, ...]] = {"embed": (V, W)}
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            x = p + "mix."
            out[p + "norm1"] = out[p + "norm1b"] = out[p + "ls1"] = (W,)
            if isinstance(m, AttentionSpec):
                own = [("q", m.heads * m.dim)]
                if m.kv_from is None:
                    own += [("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)]
                    out[x + "k.norm"] = (m.dim,)
                for n, rows in own:
                    out[x + n], out[x + n + ".b"] = (rows, W), (rows,)
                out[x + "q.norm"] = (m.dim,)
                out[x + "rel"], out[x + "sink"] = (m.rel_rows, m.heads), (m.heads,)
                out[x + "g"], out[x + "o"] = (m.heads, W), (W, m.heads * m.vdim)
            else:
                for n, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim),
                                ("g", m.heads * m.vdim), ("i", m.heads), ("f", m.heads)):
                    out[x + n] = (rows, W)
                out[x + "i.b"] = out[x + "f.b"] = (m.heads,)
                out[x + "norm"], out[x + "o"] = (m.heads * m.vdim,), (W, m.heads * m.vdim)
            if l.ff is not None:
                out[p + "norm2"] = out[p + "norm2b"] = out[p + "ls2"] = (W,)
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (l.ff.ff, W)
                out[p + "mlp.down"] = (W, l.ff.ff)
        out["final.norm"], out["head"] = (W,), (V, W)
        return out


class GunuvikForCausalLM(LayeredForCausalLM):
    config_class = GunuvikConfig

    @classmethod
    def _adapt(cls, cfg, tensors) -> None:
        for i, l in enumerate(cfg.layers):
            if isinstance(l.mixer, AttentionSpec):
                l.mixer.rel_rows = int(tensors[f"l{i}.mix.rel"].shape[0])

    @torch.no_grad()
    def init_random(self, seed: int = 0) -> "GunuvikForCausalLM":
        """Random weights of sensible size (benchmarks, tests): unit-variance projections, norms and scales near one."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for key, p in self.weights.items():
            name = key.rsplit("/", 1)[-1] if not key.endswith("/b") else "b"
            if p.dim() == 2 and name not in ("rel", "embed"):
                p.normal_(std=1.0 / math.sqrt(p.shape[1]), generator=g)
            elif name == "rel":
                p.normal_(std=0.5, generator=g)
            elif name == "embed":
                p.normal_(std=1.0 / max(1.0, self.config.embedding_scale), generator=g)
            elif name in ("norm", "norm1", "norm1b", "norm2", "norm2b"):
                p.fill_(1.0)
            elif name in ("ls1", "ls2"):
                p.fill_(0.5)
            elif key.endswith("f/b"):
                p.fill_(4.0)
        return self


def _rep(n: int, attn: AttentionSpec, mem: MLSTMSpec, width: int) -> List[LayerSpec]:
    """``n`` groups of four layers: an attention layer with keys of its own, a recurrent one, and two attention layers of
    which the second reads the keys of the first."""
    out: List[LayerSpec] = []
    ff = SwiGLUSpec(width)
    for _ in range(n):
        base = len(out)
        own = AttentionSpec(**{**attn.__dict__})
        out += [LayerSpec(own, ff), LayerSpec(MLSTMSpec(**mem.__dict__), None), LayerSpec(AttentionSpec(**{**attn.__dict__}), ff),
                LayerSpec(AttentionSpec(**{**attn.__dict__, "kv_from": base}), ff)]
    return out


def gunuvik_preset(name: str) -> GunuvikConfig:
    """Configurations for benchmarks: ``gunuvik-1.7b`` has the layer sizes of the Qwen3-1.7B backbone."""
    if name == "gunuvik-1.7b":
        attn = _attention(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, bias_max=512, window=1024, keep_first=4)
        return GunuvikConfig(151936, 2048, 1.0, 1e-6, _rep(7, attn, MLSTMSpec(heads=8, dim=128, vdim=256, gate_cap=15.0), 6144))
    if name == "gunuvik-0.6b":
        attn = _attention(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, bias_max=256, window=512, keep_first=4)
        return GunuvikConfig(151936, 1024, 1.0, 1e-6, _rep(7, attn, MLSTMSpec(heads=4, dim=128, vdim=256, gate_cap=15.0), 3072))
    if name == "gunuvik-tiny":
        attn = _attention(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.2, bias_max=50, window=21, keep_first=3, rel_rows=14)
        return GunuvikConfig(300, 160, 3.0, 1e-5, _rep(1, attn, MLSTMSpec(heads=3, dim=24, vdim=40, gate_cap=8.0), 208))
    raise KeyError(name)
