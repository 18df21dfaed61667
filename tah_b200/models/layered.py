"""What the decoders that list their layers one by one in ``config.json`` share: typed specs of the mechanisms a layer is
made of, the configuration the engine reads, and a model class that holds the weights under their on-disk names.

The computation is the engine's (:mod:`tah_b200.engine.hybrid`).  A family (:mod:`tah_b200.models.gunuvik`,
:mod:`tah_b200.models.ditilix`) reads its own ``config.json`` into these specs and says which tensors it has; every constant
of a mechanism is a field here, and a mechanism that a family does not have is absent (``None`` / ``False``).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn


# ------------------------------------------------------------------------------------
# mixers
# ------------------------------------------------------------------------------------
@dataclass
class AttentionSpec:
    """Causal attention over the paged cache: ``score = cap(temp(i) * (q . k) * scale) + bias[distance]``."""
    heads: int
    kv_heads: int
    dim: int                              # per-head size of queries and keys
    vdim: int                             # per-head size of values
    scale: float
    bias_max: Optional[int] = None        # far end of the learned distance bias; None: no bias
    window: Optional[int] = None          # None: every earlier key
    keep_first: int = 0                   # first tokens that stay visible behind the window
    kv_from: Optional[int] = None         # the layer whose keys and values this layer uses
    rel_rows: int = 32                    # rows of the distance table (a checkpoint's tensor decides)
    proj_bias: bool = False               # biases of the q / k / v projections
    qk_norm: bool = False                 # per-head RMS norm of q and k
    sink: bool = False                    # learned softmax sink per head
    head_gate: bool = False               # output gate number per head
    softcap: Optional[float] = None       # cap(s) = softcap * tanh(s / softcap)
    q_temp: Optional[Tuple[float, float]] = None      # (coef, every): temp(i) = 1 + coef * ln(floor((i + 1) / every) + 1)

    kind = "attention"


@dataclass
class MLSTMSpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"


def check_attention(i: int, m: AttentionSpec, layers: List["LayerSpec"]) -> None:
    """Refuse head counts that do not divide and a ``kv_from`` that names no earlier layer with keys of the same shape."""
    if m.heads < 1 or m.kv_heads < 1 or m.heads % m.kv_heads:
        raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} key/value heads")
    if m.softcap is not None and not m.softcap > 0:
        raise ValueError(f"layer {i}: score cap {m.softcap}")
    if m.q_temp is not None and not m.q_temp[1] > 0:
        raise ValueError(f"layer {i}: query temperature steps of {m.q_temp[1]} positions")
    if m.kv_from is not None:
        src = layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
        if not isinstance(src, AttentionSpec) or src.kv_from is not None or \
                (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
            raise ValueError(f"layer {i} cannot use the keys of layer {m.kv_from}")


# ------------------------------------------------------------------------------------
# feed-forwards
# ------------------------------------------------------------------------------------
@dataclass
class SwiGLUSpec:
    ff: int

    kind = "swiglu"


@dataclass
class PolyNormSpec:
    """``down(a N(z) + b N(z^2) + c N(z^3) + e)`` of ``z = up(h)``, ``N`` the division by the root mean square."""
    ff: int

    kind = "poly_norm"


@dataclass
class ExpertSpec:
    """A clamped gated unit: ``down(g sigmoid(1.702 g) (u + 1))``, ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""
    ff: int
    limit: float


@dataclass
class MixtureSpec:
    """``top`` of ``experts`` by sigmoid score; the score multiplies the expert's input.  ``shared``: an expert of every
    token, its output times a sigmoid gate."""
    experts: int
    top: int
    expert: ExpertSpec
    shared: Optional[ExpertSpec] = None

    kind = "moe"


@dataclass
class LayerSpec:
    mixer: object
    ff: object = None                     # feed-forward spec, None = the layer has none
    parallel: bool = False                # mixer and feed-forward side by side behind one norm


# ------------------------------------------------------------------------------------
# configuration
# ------------------------------------------------------------------------------------
@dataclass
class LayeredConfig:
    vocab_size: int
    hidden_size: int
    embedding_scale: float
    rms_norm_eps: float
    layers: List[LayerSpec]
    torch_dtype: str = "bfloat16"
    norm_groups: int = 1                  # parts of the hidden vector with a root mean square of their own
    sinusoidal: bool = False              # sinusoidal positions added to the embedding
    residual_mult: float = 1.0            # factor of the sublayers' sum in a parallel layer
    logit_scale: float = 1.0
    raw: Dict = field(default_factory=dict)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def dtype(self) -> torch.dtype:
        return getattr(torch, self.torch_dtype)

    @classmethod
    def from_dict(cls, d: dict) -> "LayeredConfig":
        raise NotImplementedError

    def to_dict(self) -> dict:
        raise NotImplementedError

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """On-disk tensor names and shapes of this configuration."""
        raise NotImplementedError

    @classmethod
    def from_pretrained(cls, path: str) -> "LayeredConfig":
        with open(os.path.join(path, "config.json"), encoding="utf-8") as fh:
            return cls.from_dict(json.load(fh))


class LayeredForCausalLM(nn.Module):
    """The weights of a model under their on-disk names; ``tensor(name)`` gives one of them."""
    config_class = LayeredConfig

    def __init__(self, cfg: LayeredConfig, dtype=None, device=None):
        super().__init__()
        self.config = cfg
        self.weights = nn.ParameterDict()
        for name, shape in cfg.tensor_shapes().items():
            self.weights[self._key(name)] = nn.Parameter(torch.zeros(*shape, dtype=dtype or cfg.dtype, device=device),
                                                         requires_grad=False)

    @staticmethod
    def _key(name: str) -> str:
        return name.replace(".", "/")

    def tensor(self, name: str) -> torch.Tensor:
        return self.weights[self._key(name)].detach()

    @property
    def device(self):
        return self.tensor("embed").device

    @property
    def dtype(self):
        return self.tensor("embed").dtype

    # ---- persistence -------------------------------------------------------------------
    @classmethod
    def _adapt(cls, cfg: LayeredConfig, tensors: Dict[str, torch.Tensor]) -> None:
        """Take into ``cfg`` what only the checkpoint's tensors say."""

    @classmethod
    def from_pretrained(cls, path: str, dtype=None, device=None) -> "LayeredForCausalLM":
        from tah_b200.utils.checkpoint import load_tensors
        cfg = cls.config_class.from_pretrained(path)
        tensors = load_tensors(path)
        cls._adapt(cfg, tensors)
        want = cfg.tensor_shapes()
        missing = [n for n in want if n not in tensors]
        extra = [n for n in tensors if n not in want]
        wrong = [n for n in want if n in tensors and tuple(tensors[n].shape) != want[n]]
        if missing or extra or wrong:
            raise ValueError(f"checkpoint does not fit its configuration: missing {missing[:4]}, unknown {extra[:4]}, "
                             f"of another shape {wrong[:4]}")
        model = cls(cfg, dtype=dtype, device=device)
        with torch.no_grad():
            for n, t in tensors.items():
                model.weights[cls._key(n)].copy_(t)
        return model

    def save_pretrained(self, path: str, max_shard_bytes: int = 5 * 1024 ** 3) -> None:
        from tah_b200.utils.checkpoint import save_tensors
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as fh:
            json.dump(self.config.to_dict(), fh, indent=2)
        save_tensors({n: self.tensor(n) for n in self.config.tensor_shapes()}, path, max_shard_bytes)
