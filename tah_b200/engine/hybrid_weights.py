"""Kernel-ready weights of the layered decoders (:mod:`tah_b200.models.layered`): matrices that read the same input stacked
into one, sizes padded once with zeros that drop out of every result (matrix rows and columns to multiples of 64, head sizes
to multiples of 8), tables in the units of the kernels.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from tah_b200.models.layered import (AttentionSpec, LayeredForCausalLM, MixtureSpec, MLSTMSpec, PolyNormSpec, SwiGLUSpec)
from tah_b200.ops import cuda as K

LOG2E = 1.4426950408889634


def _pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def distance_table(rel: torch.Tensor, far: int) -> torch.Tensor:
    """``[heads, far + 1]`` fp32 bias by distance from a bucket table ``rel [rows, heads]``: distance ``n`` below
    ``half = rows // 2`` has a row of its own; larger ones share rows logarithmically up to ``far``, from where the last
    row serves.  The bucket's floor is evaluated in integers (``(far / half) ** k <= (n / half) ** (rows - half)``)."""
    rows = rel.shape[0]
    half = rows // 2
    if far <= half:
        raise ValueError(f"distance bias: the far end {far} lies inside the {half} exact distances")
    m, k, idx = rows - half, 0, []
    for n in range(far + 1):
        if n < half:
            idx.append(n)
            continue
        while k < m and far ** (k + 1) * half ** (m - k - 1) <= n ** m:
            k += 1
        idx.append(min(rows - 1, half + k))
    return rel.float()[torch.tensor(idx, device=rel.device)].t().contiguous()


@dataclass
class AttentionLayer:
    spec: AttentionSpec
    dk: int
    dv: int
    nkv: int                      # heads this layer writes (0: it reads another layer's cache)
    w_in: torch.Tensor            # rows: queries, own keys, own values, gate numbers, input rows of a parallel feed-forward
    w_o: torch.Tensor             # columns: heads, then those of a parallel feed-forward
    kv_col: int                   # first key column of the projection
    b_in: Optional[torch.Tensor] = None
    gate_col: Optional[int] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None   # [heads, far + 1], natural units for the plain kernel, log2 units for the others
    sink: Optional[torch.Tensor] = None

    @property
    def own_queries(self) -> bool:
        """Queries need a step of their own between projection and attention (bias or norm)."""
        return self.b_in is not None or self.q_norm is not None


@dataclass
class MemoryLayer:
    spec: MLSTMSpec
    dk: int
    dv: int
    w_in: torch.Tensor            # rows: q, k, v, output gate
    w_if: torch.Tensor            # input and forget gate rows
    b_if: torch.Tensor
    norm: torch.Tensor
    w_o: torch.Tensor


@dataclass
class PolyNormLayer:
    """Feed-forward beside the mixer: its input rows are part of ``w_in`` (at ``in_col`` of the projection), its activation
    part of the mixer's output (at ``out_col``), its down projection part of ``w_o``."""
    n: int
    cols: int                     # n padded to 64
    act: torch.Tensor
    in_col: int
    out_col: int


@dataclass
class SharedExpertLayer:
    """An expert of every token, laid out like :class:`PolyNormLayer` with interleaved gate / up rows."""
    cols: int
    limit: float
    in_col: int
    out_col: int


@dataclass
class MixtureLayer:
    spec: MixtureSpec
    cols: int
    w_router: torch.Tensor        # router rows, then the shared expert's gate row
    w_gu: torch.Tensor            # [experts, 2 * cols, Wp], interleaved gate / up rows
    w_down: torch.Tensor          # [experts, Wp, cols]
    shared: Optional[SharedExpertLayer] = None


@dataclass
class BlockWeights:
    mixer: object
    norm1: torch.Tensor
    parallel: bool = False        # mixer and feed-forward side by side (ff), one residual step for both
    ff: object = None
    out1: Optional[torch.Tensor] = None   # output norm weight x layer scale
    norm2: Optional[torch.Tensor] = None
    out2: Optional[torch.Tensor] = None
    w_gu: Optional[torch.Tensor] = None
    w_down: Optional[torch.Tensor] = None


class HybridWeights:
    """Kernel-ready layout of a layered model's weights in the activation type ``dtype``."""

    def __init__(self, model: LayeredForCausalLM, dtype: torch.dtype, plain: bool):
        cfg = model.config
        unit = 1.0 if plain else LOG2E
        dev = model.device
        self.W, self.Wp = cfg.hidden_size, _pad(cfg.hidden_size, 64)
        self.vocab = cfg.vocab_size
        self.vocab_shard = (0, self.vocab, _pad(self.vocab, 64))
        T = model.tensor

        def vec(t, n):                                       # fp32 vector padded to n
            o = torch.zeros(n, dtype=torch.float32, device=dev)
            o[:t.numel()] = t.float()
            return o

        def heads_rows(w, h, d, dp):                         # [h * d, W] -> [h * dp, Wp]
            o = torch.zeros(h, dp, self.Wp, dtype=dtype, device=dev)
            o[:, :d, :w.shape[1]] = w.view(h, d, -1)
            return o.view(h * dp, self.Wp)

        def heads_vec(b, h, d, dp):
            o = torch.zeros(h, dp, dtype=torch.float32, device=dev)
            o[:, :d] = b.float().view(h, d)
            return o.view(-1)

        def heads_cols(w, h, d, dp):                         # [W, h * d] -> [Wp, pad64(h * dp)]
            o = torch.zeros(self.Wp, _pad(h * dp, 64), dtype=dtype, device=dev)
            o[:w.shape[0], :h * dp].view(w.shape[0], h, dp)[:, :, :d] = w.view(w.shape[0], h, d)
            return o

        def mat(w, rows, cols):
            o = torch.zeros(rows, cols, dtype=dtype, device=dev)
            o[:w.shape[0], :w.shape[1]] = w
            return o

        def stack(parts):                                    # row blocks, padded to a multiple of 64 rows
            o = torch.zeros(_pad(sum(p.shape[0] for p in parts), 64), self.Wp, dtype=dtype, device=dev)
            at = 0
            for p in parts:
                o[at:at + p.shape[0], :p.shape[1]] = p
                at += p.shape[0]
            return o

        def cols_of(w, n):                                   # weight columns padded to n
            return mat(w, self.Wp, n)

        def gate_up(p, n):                                   # interleaved gate / up rows of a unit, padded to 2 n
            return K.interleave_gate_up(torch.cat([mat(T(p + "gate"), n, self.Wp), mat(T(p + "up"), n, self.Wp)]))

        self.embed = mat(T("embed"), self.vocab, self.Wp)
        self.head = mat(T("head"), self.vocab_shard[2], self.Wp)
        self.final_norm = vec(T("final.norm").float() * cfg.logit_scale, self.Wp)
        self.freq = K.sinusoid_frequencies(self.W, device=dev) if cfg.sinusoidal else None
        self.layers: List[BlockWeights] = []
        for i, l in enumerate(cfg.layers):
            p, m, f = f"l{i}.", l.mixer, l.ff
            x = p + "mix."
            dk, dv = _pad(m.dim, 8), _pad(m.vdim, 8)
            w_o = heads_cols(T(x + "o"), m.heads, m.vdim, dv)
            ff, ff_rows, ff_cols = None, [], []
            if isinstance(m, AttentionSpec):
                if max(dk, dv) > 256:
                    raise NotImplementedError("attention head sizes above 256")
                H, G, own = m.heads, m.kv_heads, m.kv_from is None
                rows = [heads_rows(T(x + "q"), H, m.dim, dk)]
                bias = [heads_vec(T(x + "q.b"), H, m.dim, dk)] if m.proj_bias else []
                if own:
                    rows += [heads_rows(T(x + "k"), G, m.dim, dk), heads_rows(T(x + "v"), G, m.vdim, dv)]
                    if m.proj_bias:
                        bias += [heads_vec(T(x + "k.b"), G, m.dim, dk), heads_vec(T(x + "v.b"), G, m.vdim, dv)]
                gate_col = None
                if m.head_gate:
                    gate_col = sum(r.shape[0] for r in rows)
                    rows.append(heads_rows(T(x + "g"), H, 1, 1))
                if l.parallel:
                    ff, ff_rows, ff_cols = self._parallel(p + "mlp.", f, _pad(sum(r.shape[0] for r in rows), 8), w_o.shape[1],
                                                          T, mat, cols_of, gate_up)
                    fill = -sum(r.shape[0] for r in rows) % 8
                    if fill:
                        rows.append(torch.zeros(fill, self.Wp, dtype=dtype, device=dev))
                w_in = stack(rows + ff_rows)
                mixer = AttentionLayer(m, dk, dv, G if own else 0, w_in, torch.cat([w_o] + ff_cols, 1) if ff_cols else w_o,
                                       kv_col=H * dk, b_in=vec(torch.cat(bias), w_in.shape[0]) if bias else None,
                                       gate_col=gate_col)
                if m.qk_norm:
                    mixer.q_norm, mixer.k_norm = vec(T(x + "q.norm"), dk), vec(T(x + "k.norm"), dk) if own else None
                if m.bias_max is not None:
                    mixer.bias = distance_table(T(x + "rel"), m.bias_max) * unit
                if m.sink:
                    mixer.sink = vec(T(x + "sink"), H) * unit
            else:
                if max(dk, dv) > 1024:
                    raise NotImplementedError("mLSTM head sizes above 1024")
                H = m.heads
                w_in = stack([heads_rows(T(x + "q"), H, m.dim, dk), heads_rows(T(x + "k"), H, m.dim, dk),
                              heads_rows(T(x + "v"), H, m.vdim, dv), heads_rows(T(x + "g"), H, m.vdim, dv)])
                w_if = mat(torch.cat([T(x + "i"), T(x + "f")]), 2 * H, self.Wp)
                mixer = MemoryLayer(m, dk, dv, w_in, w_if, torch.cat([T(x + "i.b"), T(x + "f.b")]).float(),
                                    heads_vec(T(x + "norm"), H, m.vdim, dv), w_o)
            b = BlockWeights(mixer, vec(T(p + "norm1"), self.Wp), l.parallel, ff)
            if l.parallel:
                if not isinstance(m, AttentionSpec):
                    raise NotImplementedError("a parallel layer around a recurrent mixer")
            else:
                if cfg.norm_groups != 1:
                    raise NotImplementedError("grouped norms in a layer with output norms")
                b.out1 = vec(T(p + "norm1b").float() * T(p + "ls1").float(), self.Wp)
                if f is not None:
                    if not isinstance(f, SwiGLUSpec):
                        raise NotImplementedError(f"feed-forward {f.kind} in a layer of two sublayers")
                    Ip = _pad(f.ff, 64)
                    gu = torch.cat([mat(T(p + "mlp.gate"), Ip, self.Wp), mat(T(p + "mlp.up"), Ip, self.Wp)])
                    b.w_gu = K.interleave_gate_up(gu) if dtype == torch.bfloat16 else gu
                    b.w_down = mat(T(p + "mlp.down"), self.Wp, Ip)
                    b.norm2 = vec(T(p + "norm2"), self.Wp)
                    b.out2 = vec(T(p + "norm2b").float() * T(p + "ls2").float(), self.Wp)
            self.layers.append(b)

    @staticmethod
    def _parallel(p, f, in_col, out_col, T, mat, cols_of, gate_up):
        """Layout of a feed-forward beside a mixer whose projection has ``in_col`` rows and whose output ``out_col``
        columns: ``(layer, rows for w_in, columns for w_o)``."""
        if f is None:
            return None, [], []
        if isinstance(f, PolyNormSpec):
            n = _pad(f.ff, 64)
            w = T(p + "up")
            return (PolyNormLayer(f.ff, n, T(p + "act").float().contiguous(), in_col, out_col),
                    [torch.nn.functional.pad(w, (0, 0, 0, n - f.ff))], [cols_of(T(p + "down"), n)])
        if not isinstance(f, MixtureSpec):
            raise NotImplementedError(f"feed-forward {f.kind} beside a mixer")
        n, E = _pad(f.expert.ff, 64), f.experts
        router, shared, rows, cols = T(p + "router"), None, [], []
        if f.shared is not None:
            ns = _pad(f.shared.ff, 64)
            router = torch.cat([router, T(p + "shared.sg")])
            shared = SharedExpertLayer(ns, f.shared.limit, in_col, out_col)
            rows, cols = [gate_up(p + "shared.", ns)], [cols_of(T(p + "shared.down"), ns)]
        first = gate_up(f"{p}e0.", n)
        w_gu = first.new_empty(E, *first.shape)
        w_down = first.new_empty(E, first.shape[1], n)
        for e in range(E):
            w_gu[e] = gate_up(f"{p}e{e}.", n)
            w_down[e] = cols_of(T(f"{p}e{e}.down"), n)
        return MixtureLayer(f, n, mat(router, router.shape[0], first.shape[1]), w_gu, w_down, shared), rows, cols
