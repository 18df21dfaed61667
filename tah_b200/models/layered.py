"""What the decoders that list their layers one by one in ``config.json`` share: typed specs of the mechanisms a layer is
made of, the configuration the engine reads, and a model class that holds the weights under their on-disk names.

The computation is the engine's (:mod:`tah_b200.engine.hybrid`).  A family (:mod:`tah_b200.models.gunuvik`,
:mod:`tah_b200.models.ditilix`, :mod:`tah_b200.models.niralix`, :mod:`tah_b200.models.pidenex`) reads its own ``config.json`` into
these specs and says which tensors it has; every constant of a mechanism is a field here, and a mechanism that a family does
not have is absent (``None`` / ``False``).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn


# ------------------------------------------------------------------------------------
# mixers
# ------------------------------------------------------------------------------------
@dataclass(frozen=True)
class YarnSpec:
    """Rotary frequencies stretched by ``factor`` for the slow pairs (fewer than ``slow`` turns within ``original`` positions),
    unchanged for the fast ones (more than ``fast`` turns), blended linearly between."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` entries of a head by position; pairs ``(2 i, 2 i + 1)`` when ``interleaved``, else
    ``(i, i + dims / 2)``."""
    dims: int
    base: float
    interleaved: bool = False
    yarn: Optional[YarnSpec] = None

    def frequencies(self) -> Tuple[List[float], float]:
        """``(frequency of every pair, factor of sine and cosine)`` in double precision."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        y = self.yarn
        if y is None:
            return f, 1.0

        def pair_at(turns):                   # (real-valued) index whose frequency makes `turns` turns within y.original
            return self.dims * math.log(y.original / (2 * math.pi * turns)) / (2 * math.log(self.base))

        lo, hi = max(math.floor(pair_at(y.fast)), 0), min(math.ceil(pair_at(y.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [a / y.factor * r + a * (1.0 - r) for a, r in zip(f, ramp)], 0.1 * math.log(y.factor) + 1.0


@dataclass
class AttentionSpec:
    """Causal attention over the paged cache: ``score = cap(temp(i) * (q . k) * scale) + bias[distance] - slope_h * distance``."""
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
    rotary: Optional[RotarySpec] = None
    out_bias: bool = False                # bias of the output projection
    v_mix: bool = False                   # values mixed with those of the first layer that has this flag
    keys_as_values: bool = False          # the values are the keys as projected (in front of any norm)
    pool: Optional[int] = None            # means of the blocks of that many keys wholly in front of the window are keys as well
    slopes: bool = False                  # distance bias: slope_h = 2 ** (-8 (h + 1) / heads) per token
    norm_all: bool = False                # RMS norm of q and of k over all heads at once
    wide_gate: bool = False               # the heads' outputs times sigmoid(W_g h), element by element

    kind = "attention"


@dataclass
class MLSTMSpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"


@dataclass
class LatentAttentionSpec:
    """Causal attention whose keys and values are linear in one cached latent of ``kv_rank`` and one rotated key part of
    ``rot_dim`` per token; queries come from a latent of ``q_rank``."""
    heads: int
    dim: int                              # unrotated part of queries and keys
    rot_dim: int                          # rotated part, keys share one
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rotary: RotarySpec
    window: Optional[int] = None          # None: every earlier token
    sink: bool = True                     # learned softmax sink per head
    gate: bool = True                     # output times sigmoid(W_g h), element by element

    kind = "latent_attention"


@dataclass
class GLASpec:
    """Gated linear attention: matrix memory with the decay ``sigmoid(z) ** (1 / tau)`` per key channel."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16                        # decay features (a checkpoint's tensor decides)

    kind = "gla"


@dataclass
class MinGRUSpec:
    """Elementwise gated recurrence whose gates read the current token only: ``S <- (1 - z) S + z * candidate``."""
    width: int

    kind = "min_gru"


@dataclass
class BranchesSpec:
    """Attention and an elementwise recurrence from one input, ``left_scale * left + right_scale * right``."""
    left: AttentionSpec
    right: MinGRUSpec
    left_scale: float
    right_scale: float

    kind = "parallel"


def check_rotary(i: int, r: Optional[RotarySpec], size: int) -> None:
    if r is not None and (r.dims < 2 or r.dims % 2 or r.dims > size or not r.base > 1.0):
        raise ValueError(f"layer {i}: rotation of {r.dims} of {size} dims with base {r.base}")


def check_attention(i: int, m: AttentionSpec, layers: List["LayerSpec"]) -> None:
    """Refuse head counts that do not divide and a ``kv_from`` that names no earlier layer with keys of the same shape."""
    if m.heads < 1 or m.kv_heads < 1 or m.heads % m.kv_heads:
        raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} key/value heads")
    if m.softcap is not None and not m.softcap > 0:
        raise ValueError(f"layer {i}: score cap {m.softcap}")
    if m.q_temp is not None and not m.q_temp[1] > 0:
        raise ValueError(f"layer {i}: query temperature steps of {m.q_temp[1]} positions")
    check_rotary(i, m.rotary, m.dim)
    if m.window is not None and m.window < 1:
        raise ValueError(f"layer {i}: a window of {m.window} tokens")
    if m.keys_as_values and m.dim != m.vdim:
        raise ValueError(f"layer {i}: keys of {m.dim} cannot be values of {m.vdim}")
    if m.pool is not None and (m.pool < 1 or m.window is None):
        raise ValueError(f"layer {i}: blocks of {m.pool} tokens in front of a window of {m.window}")
    if m.v_mix:
        first = next((l.mixer for l in layers if isinstance(l.mixer, AttentionSpec) and l.mixer.v_mix), m)
        if m.kv_from is not None or (first.kv_heads, first.vdim) != (m.kv_heads, m.vdim):
            raise ValueError(f"layer {i} cannot mix its values with those of the first layer that mixes")
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
class XIELUSpec:
    """``down(act(up(h)))``: ``softplus(p) z^2 + z / 2`` above zero, ``(1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2`` below, with
    two learned numbers."""
    ff: int

    kind = "xielu"


@dataclass
class ExpertSpec:
    """A clamped gated unit: ``down(g sigmoid(slope g) (u + offset))``, ``g = min(gate, limit)``, ``u = clamp(up, -limit,
    limit)``.  SwiGLU: slope 1, offset 0, no limit."""
    ff: int
    limit: float = math.inf
    slope: float = 1.702
    offset: float = 1.0


@dataclass
class MixtureSpec:
    """``top`` of ``experts`` by score: a sigmoid, or a softmax over all experts.  The score multiplies the expert's input or
    its output.  ``shared``: an expert of every token, its output times a sigmoid gate."""
    experts: int
    top: int
    expert: ExpertSpec
    shared: Optional[ExpertSpec] = None
    softmax: bool = False
    weight_output: bool = False

    kind = "moe"


@dataclass
class LayerSpec:
    mixer: object
    ff: object = None                     # feed-forward spec, None = the layer has none
    parallel: bool = False                # mixer and feed-forward side by side behind one norm


# ------------------------------------------------------------------------------------
# configuration
# ------------------------------------------------------------------------------------
@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same weights, each pass with caches and states of its
    own.  A pass begins by adding a learned vector of its own to the residual, and from the second on the embedding output."""
    start: int
    stop: int
    times: int


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
    norm_offset: float = 0.0              # stored norm weights of the residual stream are this much below their value
    streams: Optional[int] = None         # hyper-connections over that many residual streams; None: a plain residual sum
    tied_head: bool = False               # the embedding table is the output projection
    centered: bool = False                # layer norms (mean taken off) instead of RMS norms around the sublayers
    layer_scale: bool = True              # norms behind the sublayers are followed by a learned factor per channel
    loop: Optional[LoopSpec] = None
    raw: Dict = field(default_factory=dict)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order they run, as ``(layer, pass)``; the pass is given for the layer that begins one."""
        n, l = len(self.layers), self.loop
        if l is None:
            return [(i, None) for i in range(n)]
        return [(i, None) for i in range(l.start)] + \
            [(i, t if i == l.start else None) for t in range(l.times) for i in range(l.start, l.stop)] + \
            [(i, None) for i in range(l.stop, n)]

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
            self.weights[self._key(name)] = nn.Parameter(torch.zeros(shape, dtype=dtype or cfg.dtype, device=device),
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
