"""Kernel-ready weights of the layered decoders (:mod:`tah_b200.models.layered`): matrices that read the same input stacked
into one, sizes padded once with zeros that drop out of every result (matrix rows and columns to multiples of 64, head sizes
to multiples of 8), tables in the units of the kernels.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from tah_b200.models.layered import (AttentionSpec, BranchesSpec, GLASpec, LatentAttentionSpec, LayeredForCausalLM, MinGRUSpec,
                                     MixtureSpec, MLSTMSpec, PolyNormSpec, RotarySpec, SwiGLUSpec, XIELUSpec)
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
    w_in: Optional[torch.Tensor]  # rows: queries, own keys, own values, gates, input rows of a parallel feed-forward; None: a branch
    w_o: Optional[torch.Tensor]   # columns: heads, then those of a parallel feed-forward; None: a branch
    kv_col: int                   # first key column of the projection
    b_in: Optional[torch.Tensor] = None
    gate_col: Optional[int] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None   # [heads, far + 1], natural units for the plain kernel, log2 units for the others
    sink: Optional[torch.Tensor] = None
    o_bias: Optional[torch.Tensor] = None
    v_keeps: bool = False                 # this layer's values are the ones later layers mix in
    v_lambda: Optional[torch.Tensor] = None   # [1] weight of those values in this layer's
    wide_col: Optional[int] = None            # first column of the gate of every output element
    slope: Optional[torch.Tensor] = None      # [heads], units as those of the bias
    norm_w: Optional[torch.Tensor] = None     # [heads * dk] weights of the norms over all heads, those of the keys folded in
    out_scale: float = 1.0

    @property
    def own_queries(self) -> bool:
        """Queries need a step of their own between projection and attention (bias, norm or rotation)."""
        return self.b_in is not None or self.q_norm is not None or self.norm_w is not None or self.spec.rotary is not None or self.spec.v_mix


@dataclass
class MinGRULayer:
    """Columns ``[z | x | g]`` of ``d`` each at ``in_col`` of the projection, output at ``out_col`` of the mixer's."""
    spec: MinGRUSpec
    d: int                        # width padded to 8
    zb: torch.Tensor
    xb: torch.Tensor
    in_col: int
    out_col: int
    out_scale: float


@dataclass
class BranchesLayer:
    """Two mixers from one projection whose outputs lie side by side, so that one product over both brings their sum back."""
    spec: BranchesSpec
    left: AttentionLayer
    right: MinGRULayer
    w_in: torch.Tensor
    w_o: torch.Tensor


@dataclass
class LatentLayer:
    """Latent attention.  Cached row: ``[c: Rp columns | rotated part: rw]``, both multiples of 64; head lists and expansions also carry the rotated
    part through their matrix products, by unit rows."""
    spec: LatentAttentionSpec
    dk: int                       # a head's query / key, dim + rot_dim padded to 8
    dv: int
    Qp: int                       # query latent, padded to 64
    Rp: int
    rw: int
    w_in: torch.Tensor            # rows: query latent, c, rotated part, output gate
    c_col: int
    r_col: int
    g_col: Optional[int]
    q_norm: torch.Tensor
    c_norm: torch.Tensor
    w_uq: torch.Tensor            # [heads * dk, Qp]
    w_abs: torch.Tensor           # [heads, row of the cache, dk padded to 64]: query -> query against cached rows
    w_uv: torch.Tensor            # [heads, dv padded to 64, Rp]: weighted c -> value
    w_exp: Optional[torch.Tensor]             # [heads * dk + heads * dv, row of the cache]: cached rows -> keys and values
    w_o: torch.Tensor
    sink: Optional[torch.Tensor]  # natural units for the plain kernel, log2 units for the others
    sink_log2: Optional[torch.Tensor]
    on_tensor_cores: bool         # single tokens run on the tensor-core kernel


@dataclass
class GLALayer:
    spec: GLASpec
    dk: int
    dv: int
    w_in: torch.Tensor            # rows: q, k, v, output gate
    w_a1: torch.Tensor            # decay features, rows padded to 4
    w_a2: torch.Tensor            # [heads * dk, features]
    b_a2: torch.Tensor
    norm: torch.Tensor            # [dv], shared by the heads
    w_o: torch.Tensor


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
class XIELULayer:
    """Numbers of the activation: ``up z^2 + z / 2`` above zero, ``low (exp(z) - 1 - z) + z / 2`` below."""
    up: float
    low: float


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
    w_up: Optional[torch.Tensor] = None
    w_down: Optional[torch.Tensor] = None
    hc1: Optional[torch.Tensor] = None    # hyper-connections behind the mixer: mix, out, in of the next reader
    hc2: Optional[torch.Tensor] = None    # the same behind the feed-forward


@dataclass
class LayerRun:
    """One run of a layer.  What the residual gets in front of it: ``add`` (a vector), ``embedding`` (the embedding output)."""
    layer: int
    add: Optional[torch.Tensor] = None
    embedding: bool = False


def mixer_parts(m) -> list:
    """A mixer, or the branches it has."""
    return [m.left, m.right] if isinstance(m, BranchesLayer) else [m]


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

        def attention(x, m):
            """``(layer without its matrices, row blocks of the projection, their biases)`` of the tensors ``x + ...``."""
            dk, dv, H, G, own = _pad(m.dim, 8), _pad(m.vdim, 8), m.heads, m.kv_heads, m.kv_from is None
            if max(dk, dv) > 256:
                raise NotImplementedError("attention head sizes above 256")
            if m.keys_as_values and (not own or m.proj_bias or m.qk_norm or m.rotary is not None or m.v_mix or m.softcap is not None):
                raise NotImplementedError("values that are the keys as projected beside shared keys, biases, head norms, rotation, mixed "
                                          "values or a score cap")
            if m.norm_all and (not m.keys_as_values or m.pool is not None) or m.pool is not None and (
                    not m.keys_as_values or m.keep_first or m.slopes or m.bias_max is not None):
                raise NotImplementedError("norms over all heads or pooled blocks in this combination")
            rows = [heads_rows(T(x + "q"), H, m.dim, dk)]
            bias = [heads_vec(T(x + "q.b"), H, m.dim, dk)] if m.proj_bias else []
            if own:
                rows.append(heads_rows(T(x + "k"), G, m.dim, dk))
                if not m.keys_as_values:
                    rows.append(heads_rows(T(x + "v"), G, m.vdim, dv))
                if m.proj_bias:
                    bias += [heads_vec(T(x + "k.b"), G, m.dim, dk), heads_vec(T(x + "v.b"), G, m.vdim, dv)]
            mixer = AttentionLayer(m, dk, dv, G if own else 0, None, None, kv_col=H * dk)
            if m.head_gate:
                mixer.gate_col = sum(r.shape[0] for r in rows)
                rows.append(heads_rows(T(x + "g"), H, 1, 1))
            if m.wide_gate:
                mixer.wide_col = sum(r.shape[0] for r in rows)
                rows.append(heads_rows(T(x + "g"), H, m.vdim, dv))
            if m.qk_norm:
                mixer.q_norm, mixer.k_norm = vec(T(x + "q.norm"), dk), vec(T(x + "k.norm"), dk) if own else None
            if m.norm_all:                                   # score = factor_j * (q * w_q * w_k) . k_j: both weights go to the queries
                wq, wk = heads_vec(T(x + "q.norm"), H, m.dim, dk), heads_vec(T(x + "k.norm"), G, m.dim, dk)
                mixer.norm_w = (wq.view(G, H // G, dk) * wk.view(G, 1, dk)).reshape(-1).contiguous()
            if m.bias_max is not None:
                mixer.bias = distance_table(T(x + "rel"), m.bias_max) * unit
            if m.slopes:
                mixer.slope = (torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=torch.float64) * unit).float().to(dev)
            if m.sink:
                mixer.sink = vec(T(x + "sink"), H) * unit
            if m.out_bias:
                mixer.o_bias = vec(T(x + "o.b"), self.Wp)
            if m.v_mix:
                mixer.v_keeps = not any(isinstance(b.mixer, AttentionLayer) and b.mixer.spec.v_mix for b in self.layers)
                if not mixer.v_keeps:
                    mixer.v_lambda = T(x + "vmix").float().reshape(1)
            return mixer, rows, bias

        self.embed = mat(T("embed"), self.vocab, self.Wp)
        self.head = mat(T("embed" if cfg.tied_head else "head"), self.vocab_shard[2], self.Wp)
        norm = lambda name: cfg.norm_offset + T(name).float()
        out_norm = lambda p, q: vec(T(f"{p}norm{q}b").float() * (T(f"{p}ls{q}").float() if cfg.layer_scale else 1.0), self.Wp)
        self.final_norm = vec(norm("final.norm") * cfg.logit_scale, self.Wp)
        self.rotary: Dict[RotarySpec, Tuple[torch.Tensor, float]] = {}       # frequencies (high, low parts), sine / cosine factor
        for r in {r for r in (getattr(l.mixer, "rotary", None) for l in cfg.layers) if r is not None}:
            f, m = r.frequencies()
            f = torch.tensor(f, dtype=torch.float64)
            self.rotary[r] = (torch.stack([f.float(), (f - f.float().double()).float()]).contiguous().to(dev), m)
        self.freq = K.sinusoid_frequencies(self.W, device=dev) if cfg.sinusoidal else None
        self.layers: List[BlockWeights] = []
        for i, l in enumerate(cfg.layers):
            p, m, f = f"l{i}.", l.mixer, l.ff
            x = p + "mix."
            ff, ff_rows, ff_cols = None, [], []
            if not isinstance(m, BranchesSpec):
                kd = m.dim + m.rot_dim if isinstance(m, LatentAttentionSpec) else m.dim
                dk, dv = _pad(kd, 8), _pad(m.vdim, 8)
                w_o = heads_cols(T(x + "o"), m.heads, m.vdim, dv)
            if isinstance(m, AttentionSpec):
                mixer, rows, bias = attention(x, m)
                if l.parallel:
                    ff, ff_rows, ff_cols = self._parallel(p + "mlp.", f, _pad(sum(r.shape[0] for r in rows), 8), w_o.shape[1],
                                                          T, mat, cols_of, gate_up)
                    fill = -sum(r.shape[0] for r in rows) % 8
                    if fill:
                        rows.append(torch.zeros(fill, self.Wp, dtype=dtype, device=dev))
                mixer.w_in, mixer.w_o = stack(rows + ff_rows), torch.cat([w_o] + ff_cols, 1) if ff_cols else w_o
                if bias:
                    mixer.b_in = vec(torch.cat(bias), mixer.w_in.shape[0])
            elif isinstance(m, BranchesSpec):
                left, rows, _ = attention(x + "left.", m.left)
                left.out_scale = m.left_scale
                D, D8 = m.right.width, _pad(m.right.width, 8)
                r, in_col, heads = x + "right.", _pad(sum(t.shape[0] for t in rows), 8), m.left.heads * left.dv
                if in_col != sum(t.shape[0] for t in rows):
                    rows.append(torch.zeros(in_col - sum(t.shape[0] for t in rows), self.Wp, dtype=dtype, device=dev))
                rows += [mat(T(r + n), D8, self.Wp) for n in ("z", "x", "g")]
                w_o = torch.zeros(self.Wp, _pad(heads + D8, 64), dtype=dtype, device=dev)
                w_o[:, :heads] = heads_cols(T(x + "left.o"), m.left.heads, m.left.vdim, left.dv)[:, :heads]
                w_o[:self.W, heads:heads + D] = T(r + "o")
                right = MinGRULayer(m.right, D8, vec(T(r + "z.b"), D8), vec(T(r + "x.b"), D8), in_col, heads, m.right_scale)
                mixer = BranchesLayer(m, left, right, stack(rows), w_o)
            elif isinstance(m, LatentAttentionSpec):
                mixer = self._latent(x, m, dk, dv, w_o, dtype, plain, T, mat, stack, heads_rows)
            elif isinstance(m, GLASpec):
                if max(dk, dv) > 1024:
                    raise NotImplementedError("gated linear attention head sizes above 1024")
                H, rank = m.heads, _pad(m.rank, 4)
                w_in = stack([heads_rows(T(x + "q"), H, m.dim, dk), heads_rows(T(x + "k"), H, m.dim, dk),
                              heads_rows(T(x + "v"), H, m.vdim, dv), heads_rows(T(x + "g"), H, m.vdim, dv)])
                w_a2 = torch.zeros(H, dk, rank, dtype=dtype, device=dev)
                w_a2[:, :m.dim, :m.rank] = T(x + "a2").view(H, m.dim, m.rank)
                mixer = GLALayer(m, dk, dv, w_in, mat(T(x + "a1"), rank, self.Wp), w_a2.view(H * dk, rank),
                                 heads_vec(T(x + "a2.b"), H, m.dim, dk), vec(T(x + "norm"), dv), w_o)
            else:
                if max(dk, dv) > 1024:
                    raise NotImplementedError("mLSTM head sizes above 1024")
                H = m.heads
                w_in = stack([heads_rows(T(x + "q"), H, m.dim, dk), heads_rows(T(x + "k"), H, m.dim, dk),
                              heads_rows(T(x + "v"), H, m.vdim, dv), heads_rows(T(x + "g"), H, m.vdim, dv)])
                w_if = mat(torch.cat([T(x + "i"), T(x + "f")]), 2 * H, self.Wp)
                mixer = MemoryLayer(m, dk, dv, w_in, w_if, torch.cat([T(x + "i.b"), T(x + "f.b")]).float(),
                                    heads_vec(T(x + "norm"), H, m.vdim, dv), w_o)
            b = BlockWeights(mixer, vec(norm(p + "norm1"), self.Wp), l.parallel, ff)
            if l.parallel:
                if not isinstance(m, AttentionSpec):
                    raise NotImplementedError("a parallel layer around a recurrent mixer")
            else:
                if cfg.streams is None:
                    if cfg.norm_groups != 1:
                        raise NotImplementedError("grouped norms in a layer with output norms")
                    b.out1 = out_norm(p, 1)
                if f is not None:
                    b.norm2 = vec(norm(p + "norm2"), self.Wp)
                    if cfg.streams is None:
                        b.out2 = out_norm(p, 2)
                if isinstance(f, SwiGLUSpec):
                    Ip = _pad(f.ff, 64)
                    gu = torch.cat([mat(T(p + "mlp.gate"), Ip, self.Wp), mat(T(p + "mlp.up"), Ip, self.Wp)])
                    b.w_gu = K.interleave_gate_up(gu) if dtype == torch.bfloat16 else gu
                    b.w_down = mat(T(p + "mlp.down"), self.Wp, Ip)
                elif isinstance(f, XIELUSpec) and cfg.streams is None:
                    Ip, act = _pad(f.ff, 64), T(p + "mlp.act").double()
                    soft = torch.logaddexp(act, torch.zeros_like(act)).tolist()
                    b.ff = XIELULayer(soft[0], 0.5 + soft[1])
                    b.w_up, b.w_down = mat(T(p + "mlp.up"), Ip, self.Wp), mat(T(p + "mlp.down"), self.Wp, Ip)
                elif isinstance(f, MixtureSpec) and f.shared is None and cfg.streams is not None:
                    b.ff = self._mixture(p + "mlp.", f, T(p + "mlp.router"), None, T, mat, cols_of, gate_up)
                elif f is not None:
                    raise NotImplementedError(f"feed-forward {f.kind} in a layer of two sublayers")
            self.layers.append(b)

        self.streams, self.hc_in0 = cfg.streams, None
        if cfg.streams is not None:
            self._streams(cfg, T)
        if cfg.loop is not None and (cfg.streams is not None or any(l.parallel or getattr(l.mixer, "kv_from", None) is not None or
                                                                    getattr(l.mixer, "v_mix", False) for l in cfg.layers)):
            raise NotImplementedError("a loop over layers with residual streams, parallel feed-forwards or another layer's keys or values")
        if cfg.centered and (cfg.streams is not None or cfg.norm_groups != 1 or any(l.parallel for l in cfg.layers)):
            raise NotImplementedError("layer norms with residual streams, grouped norms or parallel feed-forwards")
        self.runs = [LayerRun(i) if t is None else LayerRun(i, vec(T("loop.step")[t], self.Wp), t > 0) for i, t in cfg.layer_runs()]

    def parts(self) -> list:
        """The mixers of all layers, branches one by one."""
        return [p for b in self.layers for p in mixer_parts(b.mixer)]

    def _streams(self, cfg, T) -> None:
        """Hyper-connection weights of every seam: how the sublayer in front writes, how the next one (at the end: the plain
        sum) reads."""
        flat = lambda *names: torch.cat([T(n).float().reshape(-1) for n in names])
        subs = [(i, q) for i, l in enumerate(cfg.layers) for q in ((1,) if l.ff is None else (1, 2))]
        ins = [flat(f"l{i}.hc{q}.in") for i, q in subs] + [torch.ones(cfg.streams, device=self.embed.device)]
        self.hc_in0 = ins[0]
        for k, (i, q) in enumerate(subs):
            w = torch.cat([flat(f"l{i}.hc{q}.mix", f"l{i}.hc{q}.out"), ins[k + 1]]).contiguous()
            setattr(self.layers[i], f"hc{q}", w)

    def _latent(self, x, m, dk, dv, w_o, dtype, plain, T, mat, stack, heads_rows) -> LatentLayer:
        H, d, r, R = m.heads, m.dim, m.rot_dim, m.kv_rank
        dev = self.embed.device
        Qp, Rp, rw = _pad(m.q_rank, 64), _pad(R, 64), _pad(r, 64)
        lp, dkv, unit = Rp + rw, T(x + "dkv"), torch.arange(r, device=dev)
        w_in = stack([mat(T(x + "dq"), Qp, self.Wp), mat(dkv[:R], Rp, self.Wp), mat(dkv[R:], rw, self.Wp)] +
                     ([heads_rows(T(x + "g"), H, m.vdim, dv)] if m.gate else []))
        w_uq = torch.zeros(H, dk, Qp, dtype=dtype, device=dev)
        w_uq[:, :d + r, :m.q_rank] = T(x + "uq").view(H, d + r, m.q_rank)
        w_uq = mat(w_uq.view(H * dk, Qp), _pad(H * dk, 64), Qp)
        uk, uv = T(x + "uk").view(H, d, R), T(x + "uv").view(H, m.vdim, R)
        w_abs = torch.zeros(H, lp, _pad(dk, 64), dtype=dtype, device=dev)
        w_abs[:, :R, :d] = uk.transpose(1, 2)
        w_abs[:, Rp + unit, d + unit] = 1.0
        w_uv = torch.zeros(H, _pad(dv, 64), Rp, dtype=dtype, device=dev)
        w_uv[:, :m.vdim, :R] = uv
        w_exp = None
        if not plain and max(dk, dv) <= 256:
            w_exp = torch.zeros(_pad(H * (dk + dv), 64), lp, dtype=dtype, device=dev)
            k = w_exp[:H * dk].view(H, dk, lp)
            k[:, :d, :R] = uk
            k[:, d + unit, Rp + unit] = 1.0
            w_exp[H * dk:H * (dk + dv)].view(H, dv, lp)[:, :m.vdim, :R] = uv
        vec = lambda t, n: torch.nn.functional.pad(t.float(), (0, n - t.numel())).contiguous()
        sink = T(x + "sink").float().contiguous() if m.sink else None
        return LatentLayer(m, dk, dv, Qp, Rp, rw, w_in, Qp, Qp + Rp, Qp + Rp + rw if m.gate else None, vec(T(x + "dq.norm"), Qp),
                           vec(T(x + "dkv.norm"), Rp), w_uq, w_abs, w_uv, w_exp, w_o, sink, None if sink is None else sink * LOG2E,
                           not plain and K.latent_decode_fits(H, Rp, rw))

    @staticmethod
    def _mixture(p, f, router, shared, T, mat, cols_of, gate_up) -> MixtureLayer:
        n, E = _pad(f.expert.ff, 64), f.experts
        first = gate_up(f"{p}e0.", n)
        w_gu = first.new_empty(E, *first.shape)
        w_down = first.new_empty(E, first.shape[1], n)
        for e in range(E):
            w_gu[e] = gate_up(f"{p}e{e}.", n)
            w_down[e] = cols_of(T(f"{p}e{e}.down"), n)
        return MixtureLayer(f, n, mat(router, router.shape[0], first.shape[1]), w_gu, w_down, shared)

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
        router, shared, rows, cols = T(p + "router"), None, [], []
        if f.shared is not None:
            ns = _pad(f.shared.ff, 64)
            router = torch.cat([router, T(p + "shared.sg")])
            shared = SharedExpertLayer(ns, f.shared.limit, in_col, out_col)
            rows, cols = [gate_up(p + "shared.", ns)], [cols_of(T(p + "shared.down"), ns)]
        return HybridWeights._mixture(p, f, router, shared, T, mat, cols_of, gate_up), rows, cols
