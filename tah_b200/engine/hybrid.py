"""HybridEngine: decoders that list their layers one by one - windowed attention and latent attention over the paged cache,
recurrent layers with a state per row, mixers of several branches, dense feed-forwards and mixtures of experts, sublayers one
after the other or side by side, ranges of layers that run several times - on one or several fp32 residual streams.

One function, :meth:`HybridEngine._layers`, runs the layers for a packed set of tokens.  It serves

* :meth:`step` - any mixture of prompt portions and single decoded tokens of different rows in one batch: the step
  function of prefill, of request admission and of trace replay.  New keys and values go to the paged cache first and
  attention reads the cache only, so where a prompt was cut, which pages a row holds and what else is in the batch do not
  enter the arithmetic;
* the decode tick - one token of every row, captured in a CUDA graph (:class:`tah_b200.engine.base.DecodeEngine`).

Rows are cache rows: a row owns pages of the KV pool and one slot of the recurrent state.  ``admit`` / ``release`` hand
them out.  The weights are laid out for the kernels once, with padded sizes (:mod:`tah_b200.engine.hybrid_weights`).
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import List, Optional, Sequence

import torch

from tah_b200.engine.base import DecodeEngine
from tah_b200.engine.kv_cache import CacheGeometry, LayerKV, PagedKVCache, RecurrentState
from tah_b200.engine.hybrid_weights import (AttentionLayer, BlockWeights, BranchesLayer, GLALayer, HybridWeights, LatentLayer, LayerRun,
                                             MemoryLayer, MinGRULayer, MixtureLayer, PolyNormLayer, XIELULayer, distance_table, mixer_parts)
from tah_b200.models.layered import LayeredForCausalLM
from tah_b200.ops import cuda as K
from tah_b200.utils.observe import nvtx_range

NO_WINDOW = 2 ** 31 - 1
TILE = 128                        # tokens of an attention query tile and of a chunk of a recurrent layer
MEMORY_CHUNKS = 192               # chunks per launch of a recurrent layer (bounds the workspace)
LATENT_PAGES = 8192               # cache pages whose latents are expanded to keys and values at a time


class _Plan:
    """Which tokens a pass runs: packed token ids, positions, cache rows and KV slots.  The first ``n_dec`` tokens are
    single tokens of a row each; behind them lie the prompt portions, portion ``e`` at ``seq_start[e]``,
    ``seq_len[e]`` tokens long, cut into tiles of up to 128 tokens (attention query tiles and chunks of recurrent layers)."""
    tok = pos = row = slot = None
    n_dec = 0
    seq_start = seq_len = None
    tile_q0 = tile_qn = None
    groups = ()                   # recurrent launches: (tiles a..b, first tile and tile count of each of their portions)
    latent = None                 # window -> (latent expansions: (tiles a..b, cache pages of their portions), table of their pages)
    latent_pages = 0              # pages of the largest of them
    portion_of = None             # portion of every token
    pooled = None                 # (window, block) -> (pooled rows that the portions see, first page of 16 of every tile)
    pooled_rows = 0               # rows of the largest of them
    longest = 0                   # tokens of the longest portion


def decode_splits(m: AttentionLayer, n: int) -> int:
    """Key splits of the decode attention: enough CTAs to fill the SMs at small batches, at least four pages each."""
    if n == 0:
        return 1
    g = m.spec.heads // m.spec.kv_heads
    ctas = n * m.spec.kv_heads * ((g + 3) // 4)
    pages = 64 if m.spec.window is None else (m.spec.window + m.spec.keep_first) // 16 + 1
    if m.spec.pool is not None:
        pages += 64 // m.spec.pool
    return max(1, min(K.SM_COUNT * 4 // ctas, pages // 4, 16))


def latent_splits(m: LatentLayer, n: int) -> int:
    """Key splits of the absorbed latent attention: the number whose CTA waves (one CTA per SM) cost least, at 20 ns per key and
    3 us for start, end and merge of a CTA, for the window or a context of 2048 keys."""
    if n == 0 or not m.on_tensor_cores:
        return 1
    ctas = n * (1 if m.spec.heads <= 16 else (m.spec.heads + 31) // 32)
    keys = 2048 if m.spec.window is None else min(2048, m.spec.window)
    return min(range(1, 1 + max(1, min(16, keys // 96))), key=lambda s: -(-ctas * s // K.SM_COUNT) * (0.02 * keys / s + 3.0))


def gru_splits(m: MinGRULayer, portions: int, longest: int) -> int:
    """Segments of a portion in an elementwise recurrence (a CTA owns 64 channels of one): segments read the gates twice, so they
    pay when they fill SMs that would idle; 256 tokens and more each."""
    ctas = portions * ((m.d + 63) // 64)
    if ctas >= K.SM_COUNT:
        return 1
    return max(1, min(-(-K.SM_COUNT * 2 // max(1, ctas)), longest // 256, 32))


class _Buffers:
    """Activations of a pass over ``n`` tokens, the first ``n_dec`` of them single tokens; ``chunks``: chunks of a recurrent
    layer's launch; ``latent_pages``: cache pages of a latent expansion; ``pooled_rows``: rows of pooled blocks that portions
    see; ``portions`` / ``longest``: number of portions and tokens of the longest."""

    def __init__(self, w: HybridWeights, n: int, dtype, dev, n_dec: int, chunks: int = 0, latent_pages: int = 0, pooled_rows: int = 0,
                 portions: int = 0, longest: int = 0):
        e = lambda *s: torch.empty(*s, dtype=dtype, device=dev)
        whole, mix = [b.mixer for b in w.layers], w.parts()
        moe = [b.ff for b in w.layers if isinstance(b.ff, MixtureLayer)]
        self.x = torch.empty((n, w.Wp) if w.streams is None else (n, w.streams, w.Wp), dtype=torch.float32, device=dev)
        self.h, self.y = e(n, w.Wp), e(n, w.Wp)
        self.proj = e(n, max(m.w_in.shape[0] for m in whole))
        self.q = e(n, max([m.spec.heads * m.dk for m in mix if isinstance(m, AttentionLayer) and m.own_queries] +
                          [m.w_uq.shape[0] for m in mix if isinstance(m, LatentLayer)] or [0]))
        # columns between heads * dv and the padded width meet zero weight columns; they only have to be finite
        self.o = torch.zeros(n, max(m.w_o.shape[1] for m in whole), dtype=dtype, device=dev)
        self.gates = torch.empty(n * max([m.w_if.shape[0] for m in mix if isinstance(m, MemoryLayer)] or [0]),
                                 dtype=torch.float32, device=dev)
        f32 = lambda k: torch.empty(k, dtype=torch.float32, device=dev)
        self.attn_ws = f32(max([n_dec * m.spec.heads * decode_splits(m, n_dec) * (m.dv + 2) for m in mix
                                if isinstance(m, AttentionLayer)] or [0]))
        self.mem_ws = f32(max([K.mlstm_chunk_ws_floats(chunks, m.spec.heads, m.dk, m.dv) for m in mix if isinstance(m, MemoryLayer)] +
                              [K.gla_chunk_ws_floats(n, chunks, m.spec.heads, m.dk, m.dv) for m in mix if chunks and isinstance(m, GLALayer)]
                              or [0]))
        self.gru_ws = f32(max([portions * gru_splits(m, portions, longest) * 2 * m.d for m in mix if isinstance(m, MinGRULayer)] or [0]))
        self.pooled = e(pooled_rows * max([m.nkv * m.dk for m in mix if isinstance(m, AttentionLayer) and m.spec.pool is not None] or [0]))
        self.low = f32(n * max([m.w_a1.shape[0] for m in mix if isinstance(m, GLALayer)] or [0]))
        self.rope = {r: f32(n * r.dims).view(n, r.dims // 2, 2) for r in w.rotary}
        self.v_first = e(n, max([m.nkv * m.dv for m in mix if isinstance(m, AttentionLayer) and m.spec.v_mix] or [0]))
        # latent attention: query latents; head lists of the tokens in the absorbed form; expanded keys and values of the others
        lat = [m for m in mix if isinstance(m, LatentLayer)]
        listed = lambda m: n if m.w_exp is None else n_dec
        self.head_lists = {(k, h): K.HeadLists(k, h, dtype, dev) for k, h in {(listed(m), m.spec.heads) for m in lat} if k}
        rows = lambda m: self.head_lists[listed(m), m.spec.heads].rows if listed(m) else 0
        most = lambda size: e(max([size(m) for m in lat] or [0]))
        self.cq = most(lambda m: n * m.Qp)
        self.list_q, self.list_qa = most(lambda m: rows(m) * m.w_abs.shape[2]), most(lambda m: rows(m) * m.w_abs.shape[1])
        self.list_o, self.list_v = most(lambda m: rows(m) * m.Rp), most(lambda m: rows(m) * m.w_uv.shape[1])
        self.latents = most(lambda m: latent_pages * 16 * m.w_abs.shape[1] if m.w_exp is not None else 0)
        self.expanded = most(lambda m: latent_pages * 16 * m.w_exp.shape[0] if m.w_exp is not None else 0)
        self.latent_ws = f32(max([listed(m) * m.spec.heads * latent_splits(m, listed(m)) * (m.Rp + 2) for m in lat
                                  if latent_splits(m, listed(m)) > 1] or [0]))
        self.act = e(n, max([b.w_down.shape[1] for b in w.layers if b.w_down is not None] or [0]))
        # experts: logits of router and shared gate, token lists, their rows, activations and outputs
        self.router = f32(n * max([f.w_router.shape[0] for f in moe] or [0]))
        self.lists = {k: K.ExpertLists(n, *k, dtype, dev) for k in {(f.spec.experts, f.spec.top) for f in moe}}
        rows = lambda f: self.lists[f.spec.experts, f.spec.top].rows
        most = max([rows(f) for f in moe] or [0])
        self.list_x, self.list_y = e(most * w.Wp), e(most * w.Wp)
        self.list_act = e(max([rows(f) * f.cols for f in moe] or [0]))


@dataclass
class StepEntry:
    """One row's part of a step: its next tokens and the places among them whose logits are wanted."""
    row: int
    tokens: Sequence[int]
    want: Sequence[int] = ()


class HybridEngine(DecodeEngine):
    def __init__(self, model: LayeredForCausalLM, max_rows: int = 64, max_seq_len: int = 2048, page_size: int = 16,
                 use_cuda_graph: bool = True, prefill_tokens: int = 16384):
        """``prefill_tokens``: the most prompt tokens one step runs (longer prompts are cut into portions)."""
        self.model, self.cfg = model, model.config
        self.device = model.device
        if self.device.type != "cuda":
            raise RuntimeError("HybridEngine needs the model on a CUDA device")
        self.dtype = model.dtype
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"HybridEngine runs in bfloat16 or float32, not {self.dtype}")
        self.max_iter, self.topk, self.tp = 1, 1, None
        # the plain kernels (any page size, fp32; bring-up and comparison in bf16) instead of the tensor-core / pipelined ones
        self.plain = (self.dtype != torch.bfloat16 or page_size != 16
                      or os.environ.get("TAH_B200_NAIVE_PREFILL", "0") == "1")
        self.w = HybridWeights(model, self.dtype, self.plain)
        self.prefill_tokens = prefill_tokens
        self.state: Optional[RecurrentState] = None
        self._free_rows: List[int] = []
        self.layer_hook = None                     # optional callable(layer index, residual stream) after every layer
        self._init_scheduler(max_rows, max_seq_len, page_size, use_cuda_graph)

    # ------------------------------------------------------------------------------------------
    # cache, state, rows
    # ------------------------------------------------------------------------------------------
    def _new_cache(self, rows: int, max_tokens: int, pool_tokens: Optional[int] = None) -> None:
        kv, st = [], []
        for r in self.w.runs:                                # every run of a layer has a cache and a state of its own
            cache, state = None, None
            for m in mixer_parts(self.w.layers[r.layer].mixer):
                if isinstance(m, AttentionLayer):
                    s = m.spec
                    cache = LayerKV(shared_with=s.kv_from) if m.nkv == 0 else \
                        LayerKV(m.nkv, m.dk, 0 if s.keys_as_values else m.dv, factor=s.norm_all, block=s.pool)
                elif isinstance(m, LatentLayer):             # one vector per token, key and value of all heads
                    cache = LayerKV(1, m.Rp + m.rw, 0)
                elif isinstance(m, GLALayer):
                    state = [(m.spec.heads, m.dk, m.dv)]
                elif isinstance(m, MinGRULayer):
                    state = [(m.d,)]
                else:
                    state = [(m.spec.heads, m.dk, m.dv), (m.spec.heads, m.dk), (m.spec.heads,)]
            kv.append(cache)
            st.append(state)
        self.kv = self.state = None
        self._states.clear()                       # captured ticks point into the old pools
        torch.cuda.empty_cache()
        self.kv = PagedKVCache(CacheGeometry.per_layer(kv, self.page_size), rows, max_tokens, 1, device=self.device,
                               dtype=self.dtype, pool_tokens=pool_tokens)
        self.state = RecurrentState(st, rows, self.device)
        self._free_rows = list(range(rows - 1, -1, -1))

    def open(self, rows: int, pool_tokens: int, max_tokens_per_row: Optional[int] = None) -> None:
        """Make the cache for ``rows`` live requests that together hold at most ``pool_tokens`` tokens (each request's
        count rounded up to whole pages), for use with :meth:`admit` / :meth:`step` / :meth:`release`."""
        self._new_cache(rows, max_tokens_per_row or pool_tokens, pool_tokens)

    def admit(self) -> int:
        """A free row for a new request."""
        if not self._free_rows:
            raise RuntimeError("no free row: every row holds a request")
        return self._free_rows.pop()

    def release(self, row: int) -> None:
        """The request of ``row`` is finished: its pages and its state slot may be used again."""
        self.kv.free_rows(torch.tensor([row], device=self.device))
        self._free_rows.append(row)

    # ------------------------------------------------------------------------------------------
    # the layers
    # ------------------------------------------------------------------------------------------
    def _attention(self, li: int, m: AttentionLayer, proj: torch.Tensor, b: _Buffers, plan: _Plan) -> torch.Tensor:
        """Attention of one layer run from its projection ``proj``; returns ``b.o`` with the heads in its first columns."""
        s = m.spec
        n = b.h.shape[0]
        pool = self.kv.layer_pool(0, li)
        if s.keys_as_values:
            return self._attend(m, *self._tied_keys(li, m, proj, b, plan, pool), pool, proj, b, plan)
        post = dict(dk=m.dk, dv=m.dv, dim=s.dim, page_size=self.page_size, eps=self.cfg.rms_norm_eps)
        if m.own_queries:
            q = b.q.view(-1)[:n * s.heads * m.dk].view(n, s.heads * m.dk)
            if s.rotary is not None:
                post.update(rope=b.rope[s.rotary], rot=s.rotary.dims, interleaved=s.rotary.interleaved)
            if s.v_mix:
                v = b.v_first.view(-1)[:n * m.nkv * m.dv].view(n, m.nkv * m.dv)
                post.update(dict(v_keep=v) if m.v_keeps else dict(v_first=v, lam=m.v_lambda))
            K.qkv_post(proj, m.b_in, m.q_norm, m.k_norm, q, pool, plan.slot, s.heads, m.nkv, **post)
        else:                                      # queries as projected; only new keys and values have to move
            q = proj[:, :s.heads * m.dk]
            if m.nkv:
                K.qkv_post(proj[:, m.kv_col:], None, None, None, None, pool, plan.slot, 0, m.nkv, **post)
        return self._attend(m, q, {}, pool, proj, b, plan)

    def _tied_keys(self, li: int, m: AttentionLayer, proj, b: _Buffers, plan: _Plan, pool):
        """Keys that are the values as well on their way to the cache, with the factors of their norm or the block means that they
        complete; returns the queries and what attention has to know."""
        s, n, pt = m.spec, b.h.shape[0], self.kv.page_table[0]
        extra = dict(tied=True, factor=self.kv.factors[0][li], pooled=self.kv.pooled[0][li])
        k = proj[:, m.kv_col:m.kv_col + m.nkv * m.dk]
        if s.pool is not None:
            extra.update(block=s.pool, pool_rows=self.kv.geo.layers[li].pool_rows(self.page_size))
        if m.norm_w is None:
            K.tied_keys(k, pool, plan.slot, plan.pos, plan.row, pt, m.nkv, m.dk, self.page_size, extra["pooled"],
                        extra.get("block", 0), extra.get("pool_rows", 0))
            return proj[:, :s.heads * m.dk], extra
        q = b.q.view(-1)[:n * s.heads * m.dk].view(n, s.heads * m.dk)
        K.norm_all(proj[:, :s.heads * m.dk], k, m.norm_w, q, pool, extra["factor"], plan.slot, nq=s.heads, nkv=m.nkv, dk=m.dk, dim=s.dim,
                   page_size=self.page_size, eps=self.cfg.rms_norm_eps)
        return q, extra

    def _attend(self, m: AttentionLayer, q, extra: dict, pool, proj, b: _Buffers, plan: _Plan) -> torch.Tensor:
        """Attention of queries ``q`` over the keys of ``pool``; ``extra``: see :meth:`_tied_keys`."""
        s, n = m.spec, b.h.shape[0]
        o = b.o if m.w_o is None else b.o[:, :m.w_o.shape[1]]
        kw = dict(extra, slope=m.slope, out_scale=m.out_scale,
                  nq=s.heads, nkv=s.kv_heads, dk=m.dk, dv=m.dv, page_size=self.page_size, scale=s.scale,
                  window=NO_WINDOW if s.window is None else s.window, keep_first=s.keep_first, bias=m.bias, sink=m.sink,
                  softcap=s.softcap, q_temp=s.q_temp)
        if m.gate_col is not None:
            kw["gate"] = proj[:, m.gate_col:m.gate_col + s.heads]
        if m.wide_col is not None:
            kw["wide_gate"] = proj[:, m.wide_col:m.wide_col + s.heads * m.dv]
        pt, nd = self.kv.page_table[0], plan.n_dec
        if self.plain:
            K.window_attn_plain(q, o, pool, pt, plan.pos, plan.row, **kw)
            return o
        if nd:
            K.window_attn_decode(q[:nd], o[:nd], pool, pt, plan.pos, plan.row, n_split=decode_splits(m, nd), ws=b.attn_ws, **kw)
        if nd < n:
            if s.pool is not None:                 # the block means that the portions see, as a matrix
                src, base = plan.pooled[s.window, s.pool]
                rows = src.numel()
                kw["pooled"] = None if rows == 0 else K.pool_gather(kw["pooled"], src, m.nkv, m.dk, kw["pool_rows"],
                                                                    b.pooled[:rows * m.nkv * m.dk].view(rows, m.nkv * m.dk))
                kw["pool_base"] = base
            K.window_attn_tiles(q, o, pool, pt, plan.pos, plan.row, plan.tile_q0, plan.tile_qn, self.kv.n_pages[0], **kw)
        return o

    def _branches(self, li: int, m: BranchesLayer, proj: torch.Tensor, b: _Buffers, plan: _Plan) -> torch.Tensor:
        """Attention and the elementwise recurrence, both scaled, side by side in ``b.o``."""
        self._attention(li, m.left, proj, b, plan)
        r, n, nd = m.right, b.h.shape[0], plan.n_dec
        x, o, state = proj[:, r.in_col:], b.o[:, r.out_col:r.out_col + r.d], self.state.layers[li]
        if nd:
            K.min_gru_step(x[:nd], r.zb, r.xb, o[:nd], state, plan.pos, plan.row, r.out_scale, slot=plan.slot)
        if nd < n:
            K.min_gru_scan(x, r.zb, r.xb, o, state, plan.pos, plan.row, r.out_scale, seq_start=plan.seq_start, seq_len=plan.seq_len,
                           n_split=gru_splits(r, plan.seq_start.numel(), plan.longest), ws=b.gru_ws)
        return b.o[:, :m.w_o.shape[1]]

    def _memory(self, li: int, m: MemoryLayer, proj: torch.Tensor, b: _Buffers, plan: _Plan) -> torch.Tensor:
        s = m.spec
        n, nd = b.h.shape[0], plan.n_dec
        gates = K.few_linear(b.h, m.w_if, m.b_if, out=b.gates[:n * m.w_if.shape[0]].view(n, -1))
        o = b.o[:, :m.w_o.shape[1]]
        kw = dict(heads=s.heads, dk=m.dk, dv=m.dv, dim=s.dim, vdim=s.vdim, cap=s.gate_cap, eps=self.cfg.rms_norm_eps)
        state = self.state.layers[li]
        if nd:
            K.mlstm_recurrent(proj[:nd], gates[:nd], m.norm, o[:nd], state, plan.pos, plan.row, slot=plan.slot, **kw)
        if nd < n and (self.plain or m.dk > 128 or m.dv > 256):
            K.mlstm_recurrent(proj, gates, m.norm, o, state, plan.pos, plan.row, seq_start=plan.seq_start,
                              seq_len=plan.seq_len, **kw)
        elif nd < n:
            for ta, tb, chunk0, chunks in plan.groups:
                K.mlstm_chunks(proj, gates, m.norm, o, state, plan.pos, plan.row, chunk_start=plan.tile_q0[ta:tb],
                               chunk_len=plan.tile_qn[ta:tb], seq_chunk0=chunk0, seq_chunks=chunks, ws=b.mem_ws, **kw)
        return o

    def _gla(self, li: int, m: GLALayer, proj: torch.Tensor, b: _Buffers, plan: _Plan) -> torch.Tensor:
        s = m.spec
        n, nd = b.h.shape[0], plan.n_dec
        low = K.few_linear(b.h, m.w_a1, None, out=b.low[:n * m.w_a1.shape[0]].view(n, -1))
        o = b.o[:, :m.w_o.shape[1]]
        kw = dict(heads=s.heads, dk=m.dk, dv=m.dv, dim=s.dim, vdim=s.vdim, tau=s.tau, eps=self.cfg.rms_norm_eps)
        w = (m.w_a2, m.b_a2, m.norm)
        state = self.state.layers[li]
        if nd:
            K.gla_recurrent(proj[:nd], low[:nd], *w, o[:nd], state, plan.pos, plan.row, slot=plan.slot, **kw)
        if nd < n and (self.plain or m.dk > 128 or m.dv > 256):
            K.gla_recurrent(proj, low, *w, o, state, plan.pos, plan.row, seq_start=plan.seq_start, seq_len=plan.seq_len, **kw)
        elif nd < n:
            for ta, tb, chunk0, chunks in plan.groups:
                K.gla_chunks(proj, low, *w, o, state, plan.pos, plan.row, chunk_start=plan.tile_q0[ta:tb],
                             chunk_len=plan.tile_qn[ta:tb], seq_chunk0=chunk0, seq_chunks=chunks, ws=b.mem_ws, **kw)
        return o

    def _latent(self, li: int, m: LatentLayer, proj: torch.Tensor, b: _Buffers, plan: _Plan) -> torch.Tensor:
        """Latent attention: single tokens (without expansion weights, all tokens) against the cached latents themselves,
        portions against keys and values expanded from the cached latents of their rows."""
        s, n = m.spec, b.h.shape[0]
        H, pool, rope = s.heads, self.kv.layer_pool(0, li), b.rope[s.rotary]
        view = lambda t, r, c: t[:r * c].view(r, c)
        cq = view(b.cq, n, m.Qp)
        K.latent_post(proj, m.q_norm, m.c_norm, rope, cq, pool, plan.slot, q_rank=s.q_rank, q_col=0, kv_rank=s.kv_rank, Rp=m.Rp,
                      c_col=m.c_col, rot=s.rot_dim, rw=m.rw, r_col=m.r_col, eps=self.cfg.rms_norm_eps)
        q = K.linear(cq, m.w_uq, out=view(b.q.view(-1), n, m.w_uq.shape[0]))
        nl = n if m.w_exp is None else plan.n_dec
        L = b.head_lists[nl, H] if nl else None
        list_q = view(b.list_q, L.rows, m.w_abs.shape[2]) if nl else None
        K.latent_query(q, rope, L, list_q, heads=H, dk=m.dk, dim=s.dim, rot=s.rot_dim)
        o, gate = b.o[:, :m.w_o.shape[1]], None if m.g_col is None else proj[:, m.g_col:m.g_col + H * m.dv]
        window = NO_WINDOW if s.window is None else s.window
        if nl:
            qa = K.moe_linear(list_q, m.w_abs, L, view(b.list_qa, L.rows, m.w_abs.shape[1]))
            oc = view(b.list_o, L.rows, m.Rp)
            kw = dict(Rp=m.Rp, rw=m.rw, page_size=self.page_size, scale=s.scale, window=window)
            if m.on_tensor_cores:
                K.latent_attn_decode(qa, oc, pool, self.kv.page_table[0], plan.pos, plan.row, L, sink=m.sink_log2,
                                     n_split=latent_splits(m, nl), ws=b.latent_ws, **kw)
            else:
                K.latent_attn_plain(qa, oc, pool, self.kv.page_table[0], plan.pos, plan.row, L, sink=m.sink, **kw)
            K.latent_gate(K.moe_linear(oc, m.w_uv, L, view(b.list_v, L.rows, m.w_uv.shape[1])), L,
                          None if gate is None else gate[:nl], o[:nl], m.dv)
        if nl < n:
            launches, table = plan.latent[s.window]
            for ta, tb, src in launches:
                c = K.latent_gather(pool, src, self.page_size, m.Rp + m.rw, view(b.latents, src.numel() * 16, m.w_exp.shape[1]))
                kv = K.linear(c, m.w_exp, out=view(b.expanded, c.shape[0], m.w_exp.shape[0]))
                K.window_attn_tiles(q, o, kv, table, plan.pos, plan.portion_of, plan.tile_q0[ta:tb], plan.tile_qn[ta:tb],
                                    src.numel(), kv_ld=kv.stride(0), nq=H, nkv=H, dk=m.dk, dv=m.dv, page_size=self.page_size,
                                    scale=s.scale, window=window, keep_first=0, sink=m.sink_log2, wide_gate=gate)
        return o

    def _mixture(self, f: MixtureLayer, proj: torch.Tensor, b: _Buffers):
        """Routed experts of the tokens in ``b.h``: ``(outputs by list row, list rows of every token, their weights or None
        when the inputs were weighted)``; the shared expert's activation goes to its columns of ``b.o``."""
        s, n = f.spec, b.h.shape[0]
        L = b.lists[s.experts, s.top]
        z = K.few_linear(b.h, f.w_router, None, out=b.router[:n * f.w_router.shape[0]].view(n, -1))
        K.moe_route(z, L, softmax=s.softmax)
        view = lambda t, cols: t[:L.rows * cols].view(L.rows, cols)
        x = K.moe_gather(b.h, L, view(b.list_x, b.h.shape[1]))
        ex = s.expert
        act = K.moe_glu_linear(x, f.w_gu, ex.limit, L, view(b.list_act, f.cols), slope=ex.slope, offset=ex.offset,
                               weighted=not s.weight_output)
        y = K.moe_linear(act, f.w_down, L, view(b.list_y, b.h.shape[1]))
        if f.shared is not None:
            c = f.shared
            K.clamped_glu(proj[:, c.in_col:c.in_col + 2 * c.cols], c.limit, b.o[:, c.out_col:c.out_col + c.cols],
                          gate=z[:, s.experts], slope=s.shared.slope, offset=s.shared.offset)
        return y, L.slot, L.weight if s.weight_output else None

    def _parallel_layer(self, li: int, L: BlockWeights, proj: torch.Tensor, w_next: torch.Tensor, b: _Buffers, plan: _Plan) -> None:
        """Mixer and feed-forward beside each other: both read the projection of ``b.h``, one product over the columns of
        both brings them back, and one residual step adds their sum."""
        f, y_ex, slot = L.ff, None, None
        if isinstance(f, PolyNormLayer):
            K.poly_norm(proj[:, f.in_col:f.in_col + f.cols], f.act, f.n, self.cfg.rms_norm_eps,
                        b.o[:, f.out_col:f.out_col + f.cols])
        elif isinstance(f, MixtureLayer):
            y_ex, slot, weight = self._mixture(f, proj, b)
            if weight is not None:
                raise NotImplementedError("weighted expert outputs beside a mixer")
        K.linear(self._attention(li, L.mixer, proj, b, plan), L.mixer.w_o, out=b.y)
        K.residual_add_norm(b.y, b.x, self.cfg.residual_mult, w_next, self.w.W, self.cfg.norm_groups, self.cfg.rms_norm_eps,
                            b.h, y_ex, slot)

    def _layers(self, b: _Buffers, plan: _Plan) -> torch.Tensor:
        """Run every layer on the packed tokens of ``plan`` (``b.x`` / ``b.h`` hold their embeddings and first normed
        input); returns the final-norm output."""
        w = self.w
        run = {AttentionLayer: self._attention, BranchesLayer: self._branches, LatentLayer: self._latent, GLALayer: self._gla,
               MemoryLayer: self._memory}
        for r, (freq, m) in w.rotary.items():
            K.rotary_table(plan.pos, freq, m, b.rope[r])
        for ri, r in enumerate(w.runs):
            L, follow = w.layers[r.layer], w.runs[ri + 1] if ri + 1 < len(w.runs) else None
            after = w.final_norm if follow is None else w.layers[follow.layer].norm1
            b.before = None if self.layer_hook is None or follow is None or follow.add is None else torch.empty_like(b.x)
            proj = K.linear(b.h, L.mixer.w_in, out=b.proj[:, :L.mixer.w_in.shape[0]])
            if L.parallel:
                self._parallel_layer(ri, L, proj, after, b, plan)
            else:
                K.linear(run[type(L.mixer)](ri, L.mixer, proj, b, plan), L.mixer.w_o, out=b.y)
                if w.streams is not None:
                    K.streams_norm(b.y, b.x, L.hc1, after if L.norm2 is None else L.norm2, w.W, self.cfg.norm_groups, self.cfg.rms_norm_eps,
                                   b.h, y_bias=getattr(L.mixer, "o_bias", None))
                elif L.norm2 is not None:
                    self._seam(b.y, L.out1, L.norm2, None, b, plan)
                else:
                    self._seam(b.y, L.out1, after, follow, b, plan)
                if L.norm2 is not None:
                    self._feed_forward(L, after, follow, b, plan)
            if self.layer_hook is not None:
                x = b.x if b.before is None else b.before
                self.layer_hook(ri, (x if w.streams is None else x.sum(1))[:, :w.W])
        return b.h

    def _seam(self, y: torch.Tensor, w_out: torch.Tensor, w_next: torch.Tensor, follow: Optional[LayerRun], b: _Buffers, plan: _Plan) -> None:
        """Between two sublayers with norms before and behind: output norm, residual sum, what the residual gets in front of the
        run ``follow``, next norm."""
        w, more = self.w, {}
        if follow is not None and follow.add is not None:
            more = dict(add=follow.add, before=b.before,
                        embedding=(w.embed, plan.tok, self.cfg.embedding_scale) if follow.embedding else None)
        K.residual_norm(y, b.x, w_out, w_next, w.W, self.cfg.rms_norm_eps, b.h, centered=self.cfg.centered, **more)

    def _feed_forward(self, L: BlockWeights, w_next: torch.Tensor, follow: Optional[LayerRun], b: _Buffers, plan: _Plan) -> None:
        """The second sublayer: its output joins the residual, and ``b.h`` becomes the next layer's input."""
        w, eps = self.w, self.cfg.rms_norm_eps
        y, ex = b.y, {}
        if isinstance(L.ff, MixtureLayer):
            y, (ex["y_ex"], ex["slot"], ex["y_weight"]) = None, self._mixture(L.ff, None, b)
        elif isinstance(L.ff, XIELULayer):
            K.linear(K.xielu_linear(b.h, L.w_up, L.ff.up, L.ff.low, out=b.act[:, :L.w_down.shape[1]]), L.w_down, out=y)
        else:
            act = K.swiglu_linear(b.h, L.w_gu, out=b.act[:, :L.w_down.shape[1]])
            K.linear(act, L.w_down, out=y)
        if w.streams is None:
            self._seam(y, L.out2, w_next, follow, b, plan)
        else:
            K.streams_norm(y, b.x, L.hc2, w_next, w.W, self.cfg.norm_groups, eps, b.h, **ex)

    def _embed(self, b: _Buffers, plan: _Plan) -> None:
        """``b.x``: the residual stream of the tokens of ``plan``; ``b.h``: the first layer's normed input."""
        w, first = self.w, self.w.runs[0]
        K.embed_norm(w.embed, plan.tok, self.cfg.embedding_scale, w.layers[first.layer].norm1, w.W, self.cfg.rms_norm_eps, b.x, b.h,
                     groups=self.cfg.norm_groups, pos=plan.pos, freq=w.freq, streams=w.streams or 1, w_in=w.hc_in0, add=first.add,
                     centered=self.cfg.centered)

    def _portion_plan(self, plan: _Plan, rows: List[int], counts: List[int], tiles: List[int], n: int) -> None:
        """What the layers that do not read the paged cache directly need to know about a step's portions: the cache pages whose
        latents are expanded, the pooled blocks that are seen.  Call when the step's tokens have their pages."""
        lat = {m.spec.window for m in self.w.parts() if isinstance(m, LatentLayer) and m.w_exp is not None}
        pools = {(m.spec.window, m.spec.pool) for m in self.w.parts() if isinstance(m, AttentionLayer) and m.spec.pool is not None}
        if self.plain or not (lat or pools):
            return
        dev, table = self.device, self.kv.page_table[0]
        rows_t = torch.tensor(rows, device=dev)
        lens = self.kv.len[0][rows_t].tolist()
        if any(l < c for l, c in zip(lens, counts)):         # nothing was appended: the pool or a row's table is full
            K.check_status(dev)
            raise RuntimeError("KV pool too small for the step")
        e = torch.repeat_interleave(torch.arange(len(rows), device=dev), torch.tensor(counts, device=dev), output_size=sum(counts))
        plan.portion_of = torch.nn.functional.pad(e.to(torch.int32), (n - e.numel(), 0))
        plan.latent = {w: self._latent_plan(plan, w, rows_t, lens, counts, tiles) for w in lat}
        plan.pooled = {}
        for window, block in pools:
            S = LayerKV(block=block).pool_rows(self.page_size)
            seen = [max(0, l - window) // block for l in lens]               # by the portion's last token
            pages = torch.tensor([(k + 15) // 16 for k in seen], device=dev)
            total = sum((k + 15) // 16 for k in seen)
            first = torch.cumsum(pages, 0) - pages
            which = torch.repeat_interleave(torch.arange(len(rows), device=dev), pages * 16, output_size=total * 16)
            k = torch.arange(total * 16, device=dev) - first[which] * 16
            live = k < torch.tensor(seen, device=dev)[which]
            page = table[rows_t[which], torch.where(live, k // S, 0)]
            src = torch.where(live, page * S + k % S, -1).to(torch.int32)
            base = torch.repeat_interleave(first, torch.tensor(tiles, device=dev), output_size=sum(tiles)).to(torch.int32)
            plan.pooled[window, block] = (src, base)
            plan.pooled_rows = max(plan.pooled_rows, total * 16)

    def _latent_plan(self, plan: _Plan, window: Optional[int], rows_t: torch.Tensor, lens: List[int], counts: List[int], tiles: List[int]):
        """Which cache pages the portions' latent layers of a window expand, in launches of at most ``LATENT_PAGES`` pages (a single
        longer row is a launch of its own), and where logical pages lie in them."""
        dev, table, ps = self.device, self.kv.page_table[0], self.page_size
        # first page that a portion's first token sees, in whole key blocks of the attention kernel
        skip = [0 if window is None else max(0, l - c - window + 1) // 64 * 64 // ps for l, c in zip(lens, counts)]
        pages = [(l + ps - 1) // ps - k for l, k in zip(lens, skip)]
        launches, base, at = [], [], 0                       # tiles a..b, pages a..b
        for k, t in zip(pages, tiles):
            first = launches[-1][1] if launches else 0
            if not launches or launches[-1][3] - launches[-1][2] + k > LATENT_PAGES:
                launches.append([first, first, at, at])
            base.append(at - launches[-1][2])
            launches[-1][1] += t
            at += k
            launches[-1][3] = at
        pages_t, skip_t = torch.tensor(pages, device=dev), torch.tensor(skip, device=dev)
        which = torch.repeat_interleave(torch.arange(len(pages), device=dev), pages_t, output_size=at)
        col = torch.arange(at, device=dev) - (torch.cumsum(pages_t, 0) - pages_t - skip_t)[which]
        src = table[rows_t[which], col].contiguous()
        plan.latent_pages = max([plan.latent_pages] + [d - c for _, _, c, d in launches])
        logical = torch.arange(max(k + f for k, f in zip(pages, skip)), device=dev)
        where = (torch.tensor(base, device=dev) - skip_t).view(-1, 1) + logical
        return [(a, b, src[c:d]) for a, b, c, d in launches], where.clamp(min=0).to(torch.int32)

    # ------------------------------------------------------------------------------------------
    # one step of portions and single tokens
    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def _run(self, rows: Sequence[int], counts: Sequence[int], tok: torch.Tensor, want: Sequence[int]) -> torch.Tensor:
        """Append ``counts[e]`` tokens to row ``rows[e]`` for every entry and run them as one batch.  ``tok``: int32 token
        ids of all entries back to back (device); ``want``: indices into ``tok`` whose logits are returned, in order."""
        dev, n = self.device, int(tok.numel())
        if len(set(rows)) != len(rows) or min(counts) < 1:
            raise ValueError("a step needs distinct rows with at least one token each")
        start, first = [], 0
        for c in counts:
            start.append(first)
            first += c
        order = [e for e, c in enumerate(counts) if c == 1] + [e for e, c in enumerate(counts) if c > 1]
        n_dec = sum(1 for c in counts if c == 1)
        if order != list(range(len(counts))):                    # single tokens first: move the packed tokens along
            perm, place, new_start, at = [], [0] * n, [0] * len(counts), 0
            for e in order:
                new_start[e] = at
                for t in range(counts[e]):
                    place[start[e] + t] = at + t
                    perm.append(start[e] + t)
                at += counts[e]
            tok = tok[torch.tensor(perm, device=dev)]
            want = [place[i] for i in want]
            start = new_start
        rows, counts, start = [rows[e] for e in order], [counts[e] for e in order], [start[e] for e in order]
        q0, qn, first_tile, tiles, groups = [], [], [], [], []
        for s0, c in zip(start[n_dec:], counts[n_dec:]):
            k = (c + TILE - 1) // TILE
            if not groups or groups[-1][3] + k > MEMORY_CHUNKS:
                groups.append([len(first_tile), len(first_tile), len(q0), 0])       # portions a..b, first tile, tiles
            groups[-1][1] += 1
            first_tile.append(groups[-1][3])
            tiles.append(k)
            groups[-1][3] += k
            q0 += [s0 + a for a in range(0, c, TILE)]
            qn += [min(TILE, c - a) for a in range(0, c, TILE)]
        parts = [rows, counts, start, q0, qn, first_tile, tiles, list(want)]
        meta = torch.tensor(sum(parts, []), dtype=torch.int32).pin_memory().to(dev, non_blocking=True)
        d_rows, d_counts, d_start, d_q0, d_qn, d_first, d_tiles, d_want = meta.split([len(p) for p in parts])
        plan = _Plan()
        plan.tok = tok
        plan.pos, plan.row, plan.slot = (torch.empty(n, dtype=torch.int32, device=dev) for _ in range(3))
        plan.n_dec = n_dec
        plan.seq_start, plan.seq_len = d_start[n_dec:], d_counts[n_dec:]
        plan.tile_q0, plan.tile_qn = d_q0, d_qn
        plan.groups = [(t, t + k, d_first[a:z], d_tiles[a:z]) for a, z, t, k in groups]
        K.kv_append(d_rows, d_counts, d_start, self.kv, 0, plan.pos, plan.row, plan.slot)
        plan.longest = max(counts)
        if n_dec < n:
            self._portion_plan(plan, rows[n_dec:], counts[n_dec:], tiles, n)
        b = _Buffers(self.w, n, self.dtype, dev, n_dec, 0 if self.plain else max([g[3] for g in groups] or [0]), plan.latent_pages,
                     plan.pooled_rows, len(counts) - n_dec, plan.longest)
        self._embed(b, plan)
        h = self._layers(b, plan)
        if not want:
            return torch.empty(0, self.w.vocab, dtype=self.dtype, device=dev)
        return K.linear(h[d_want.long()], self.w.head)[:, :self.w.vocab]

    def step(self, entries: Sequence[StepEntry]) -> torch.Tensor:
        """Run the entries as one batch, from the cache and state that earlier steps left; returns the logits
        ``[wanted, vocab]`` in the order of the entries and of their ``want``."""
        toks, want, at = [], [], 0
        entries = [e for e in entries if len(e.tokens)]
        if not entries:
            return torch.empty(0, self.w.vocab, dtype=self.dtype, device=self.device)
        for e in entries:
            if any(not 0 <= w < len(e.tokens) for w in e.want):
                raise ValueError("a wanted place lies outside the entry's tokens")
            toks += list(e.tokens)
            want += [at + w for w in e.want]
            at += len(e.tokens)
        if any(not 0 <= t < self.w.vocab for t in toks):
            raise ValueError("token id outside the vocabulary")
        tok = torch.tensor(toks, dtype=torch.int32).to(self.device)
        with nvtx_range("engine/step"):
            return self._run([e.row for e in entries], [len(e.tokens) for e in entries], tok, want)

    # ------------------------------------------------------------------------------------------
    # prefill / decode tick for generate() and serve()
    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def prefill(self, input_ids: torch.Tensor, attention_mask: Optional[torch.Tensor], max_new_tokens: int,
                row_ids: Optional[torch.Tensor] = None):
        """Run a batch of prompts (left- or right-padded) in steps of at most ``prefill_tokens`` tokens.  Without
        ``row_ids`` the cache is (re)built for exactly this batch; with it the prompts go into those empty rows."""
        dev = self.device
        B, T = input_ids.shape
        valid = attention_mask[:, -T:].bool() if attention_mask is not None else torch.ones(B, T, dtype=torch.bool, device=dev)
        lens = valid.sum(1)
        host_lens = lens.tolist()
        max_total = max(host_lens) + max_new_tokens + 1
        fits = self.kv is not None and self.kv.max_pages[0] * self.page_size >= max_total
        if row_ids is not None:
            if not fits:
                raise RuntimeError("admission needs an existing KV cache whose rows can hold prompt + new tokens")
        else:
            if not fits or self.kv.rows != B or self.kv.n_pages[0] < B * self.kv.max_pages[0]:
                self._new_cache(B, max_total)
            self.kv.reset()
        rows = list(range(B)) if row_ids is None else [int(r) for r in row_ids.tolist()]
        packed = input_ids[valid].to(torch.int32).contiguous()
        last: List[Optional[torch.Tensor]] = [None] * B
        portion_rows, portion_counts, ends, used, at = [], [], [], 0, 0

        def flush():
            nonlocal at
            if not portion_rows:
                return
            want, first = [], 0
            for r, c, e in zip(portion_rows, portion_counts, ends):
                first += c
                if e:
                    want.append(first - 1)
            lg = self._run([rows[r] for r in portion_rows], list(portion_counts), packed[at:at + first], want)
            for j, r in enumerate(r for r, e in zip(portion_rows, ends) if e):
                last[r] = lg[j]
            at += first
            portion_rows.clear(), portion_counts.clear(), ends.clear()

        for r, n in enumerate(host_lens):
            done = 0
            while done < n:
                c = min(n - done, self.prefill_tokens - used)
                portion_rows.append(r)
                portion_counts.append(c)
                done += c
                ends.append(done == n)
                used += c
                if used == self.prefill_tokens or len(portion_rows) == K.APPEND_MAX_ENTRIES:
                    flush()
                    used = 0
        flush()
        out = torch.empty(B, self.w.vocab_shard[2], dtype=self.dtype, device=dev)[:, :self.w.vocab]
        out.copy_(torch.stack(last))
        return out, lens, None

    def _alloc_tick_buffers(self, B: int, max_new: int):
        s = self._alloc_scheduler_state(B, max_new)
        dev = self.device
        s.buf = _Buffers(self.w, B, self.dtype, dev, B)
        s.plan = _Plan()
        s.plan.tok, s.plan.pos, s.plan.slot = s.tok, s.pos, s.slot
        s.plan.row = torch.arange(B, dtype=torch.int32, device=dev)
        s.plan.n_dec = B
        z = lambda dt: torch.zeros(B, self.w.vocab_shard[2], dtype=dt, device=dev)
        s.logits, s.cum = z(self.dtype), z(self.dtype)
        s.cum16 = s.cum if self.dtype == torch.bfloat16 else z(torch.bfloat16)
        return s

    def _tick(self, s, sampling):
        """Enqueue one decode tick on the current stream (graph-capturable)."""
        w = self.w
        s.binding.tick_begin(None, None, None)
        self._embed(s.buf, s.plan)
        K.linear(self._layers(s.buf, s.plan), w.head, out=s.logits)
        V = w.vocab
        K.logits_post(s.logits[:, :V], s.cum[:, :V], None, s.best, s.best_val)
        if sampling is not None and self.dtype != torch.bfloat16:
            s.cum16.copy_(s.cum)                      # the samplers take bf16 logits
        s.binding.tick_end(s.need_soft, self._pick_next(s, s.cum16[:, :V], sampling))

    # ------------------------------------------------------------------------------------------
    # serving: prompt portions ride along with the decoding rows
    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def serve(self, prompts: Sequence[torch.Tensor], *, max_new_tokens: int = 128, rows: Optional[int] = None,
              eos_token_id: Optional[int] = None, do_sample: bool = False, temperature: float = 1.0, top_p: float = 1.0,
              top_k: int = 0, min_p: float = 0.0, seed: Optional[int] = None, check_every: int = 16, portion: int = 2048):
        """Continuous batching over a queue of requests (1-D token id tensors of any lengths).

        While a prompt is being read its portions (at most ``portion`` prompt tokens a step) share mixed steps with the
        decoding rows, one token each, so admission never stalls them; when no prompt is pending the rows advance by
        captured decode ticks, ``check_every`` at a time.  A finished row hands back its tokens, its pages and its state
        slot.  Returns the generated token lists in request order and a statistics dict."""
        dev = self.device
        n_req = len(prompts)
        B = min(rows or self.max_rows, n_req, self.max_rows)
        lens = [int(p.numel()) for p in prompts]
        if min(lens) < 1:
            raise ValueError("serve: an empty prompt")
        need = max(lens) + max_new_tokens + 1
        sampling = None
        if do_sample:
            sampling = dict(temperature=float(temperature), top_p=float(top_p), min_p=float(min_p), top_k=int(top_k))
            seed = int(torch.randint(0, 2 ** 62, (1,)).item()) if seed is None else int(seed)
        if self.kv is None or self.kv.rows != B or self.kv.max_pages[0] * self.page_size < need or \
                self.kv.n_pages[0] < B * self.kv.max_pages[0]:
            self._new_cache(B, need)
        self.kv.reset()
        self._calls += 1
        s = self._tick_state(B, max_new_tokens, sampling, eos_token_id)
        if sampling is not None:
            s.seed_dev.fill_(seed & (2 ** 62 - 1))
        s.finished.fill_(1)                                  # idle rows are frozen for the tick kernels
        if self.use_cuda_graph and s.graph is None:
            self._tick(s, sampling)                          # lazy one-time kernel setup outside capture; no row is live
        run = self._tick_runner(s, sampling)
        owner, read, queue = [-1] * B, [0] * B, 0            # request of a row, prompt tokens read
        ids = [p.to(device=dev, dtype=torch.int32).flatten() for p in prompts]
        results: List[Optional[List[int]]] = [None] * n_req
        stats = {"ticks": 0, "mixed_steps": 0, "admitted": 0, "rows": B, "peak_pages": [0], "pages_released": 0}
        while True:
            done = ((s.finished != 0) | (s.n_out >= max_new_tokens)).tolist()
            decoding = [r for r in range(B) if owner[r] >= 0 and read[r] == lens[owner[r]]]
            fin = [r for r in decoding if done[r]]
            if fin:
                n_out = s.n_out.tolist()
                for r, row_toks in zip(fin, s.out_tokens[fin].tolist()):
                    results[owner[r]] = row_toks[:n_out[r]]
                    owner[r] = -1
                fin_t = torch.tensor(fin, device=dev)
                s.finished[fin_t] = 1
                stats["pages_released"] += self.kv.free_rows(fin_t)
                decoding = [r for r in decoding if not done[r]]
            for r in range(B):
                if owner[r] < 0 and queue < n_req:
                    owner[r], read[r] = queue, 0
                    queue += 1
                    stats["admitted"] += 1
            reading = [r for r in range(B) if owner[r] >= 0 and read[r] < lens[owner[r]]]
            if not reading and not decoding:
                break
            if not reading:
                for _ in range(check_every):
                    run()
                stats["ticks"] += check_every
            else:
                step_rows, counts, toks, finish = list(decoding), [1] * len(decoding), [], []
                if decoding:
                    toks.append(s.tok[torch.tensor(decoding, device=dev)])
                left, at, want = portion, len(decoding), list(range(len(decoding)))
                for r in reading:
                    c = min(left, lens[owner[r]] - read[r])
                    if c == 0 or len(step_rows) == K.APPEND_MAX_ENTRIES:
                        break
                    step_rows.append(r)
                    counts.append(c)
                    toks.append(ids[owner[r]][read[r]:read[r] + c])
                    read[r] += c
                    at += c
                    left -= c
                    if read[r] == lens[owner[r]]:
                        finish.append(r)
                        want.append(at - 1)
                logits = self._run(step_rows, counts, torch.cat(toks), want)
                stats["mixed_steps"] += 1
                if want:
                    where = torch.tensor(decoding + finish, device=dev)
                    last = torch.cat([s.pos[where[:len(decoding)]],
                                      torch.tensor([lens[owner[r]] - 1 for r in finish], dtype=torch.int32, device=dev)])
                    nxt = self._choose(logits, last, sampling, seed or 0, None)
                    if finish:                               # they emit their first token below, as a decoding row does
                        f = where[len(decoding):]
                        s.n_out[f], s.finished[f], s.depth[f], s.cur_iters[f], s.iter_sum[f] = 0, 0, 0, 0, 0
                        s.out_tokens[f] = 0
                        s.pos[f] = last[len(decoding):]
                    s.best[where] = nxt
                    s.need_soft.zero_()
                    s.binding.tick_end(s.need_soft, s.best)
            stats["peak_pages"][0] = max(stats["peak_pages"][0], self.kv.pages_in_use(0))
        torch.cuda.synchronize()
        K.check_status(dev)
        stats["tokens"] = sum(len(r) for r in results)
        return results, stats
