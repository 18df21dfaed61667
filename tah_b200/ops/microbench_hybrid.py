"""Micro-benchmark cases of the layered decoders' kernels (windowed, tied and latent attention, mLSTM, gated linear attention,
minGRU, fp32-residual norms, PolyNorm, xIELU, routed experts); run through :mod:`tah_b200.ops.microbench`, whose timing rules and flags apply.

FLOPs and bytes are those of the algorithm: visible (query, key) pairs for attention, for the chunkwise mLSTM one
128-token causal block plus the state read-out and update per chunk with every product counted once.
"""
from __future__ import annotations

import torch

from tah_b200.ops import cuda as K


def _bf(*s):
    return torch.randn(*s, device="cuda").to(torch.bfloat16)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _paged(rows, ctx, nkv, dk, dv):
    per = (ctx + 15) // 16
    pool = _bf(rows * per, nkv * 16 * (dk + dv))
    pt = torch.randperm(rows * per, device="cuda").to(torch.int32).view(rows, per)
    return pool, pt


def _window_kw(a):
    far = min(a.ctx, 512)
    kw = dict(nq=a.nq, nkv=a.nkv, dk=a.hd, dv=a.hd, page_size=16, scale=a.hd ** -0.5, window=a.window or 2 ** 31 - 1,
              keep_first=a.keep if a.window else 0)
    if a.softcap:
        return dict(kw, softcap=a.softcap, q_temp=(0.1, 2048))
    return dict(kw, bias=torch.randn(a.nq, far + 1, device="cuda"), sink=torch.randn(a.nq, device="cuda"))


def _visible(i, a):
    return min(i + 1, a.window + min(a.keep, max(0, i + 1 - a.window))) if a.window else i + 1


def bench_window_prefill(a):
    B, T = a.rows, a.ctx
    n = B * T
    pool, pt = _paged(B, T, a.nkv, a.hd, a.hd)
    q, out, gate = _bf(n, a.nq * a.hd), torch.empty(n, a.nq * a.hd, dtype=torch.bfloat16, device="cuda"), None if a.softcap else _bf(n, a.nq)
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    q0 = [b * T + t for b in range(B) for t in range(0, T, 128)]
    qn = [min(128, T - t) for b in range(B) for t in range(0, T, 128)]
    q0, qn, kw = _i32(q0), _i32(qn), _window_kw(a)
    fn = lambda i: K.window_attn_tiles(q, out, pool, pt, pos, row, q0, qn, pool.shape[0], gate=gate, **kw)
    pairs = B * sum(_visible(i, a) for i in range(T))
    res = {"op": "window_prefill", "seqs": B, "T": T, "window": a.window, "keep": a.keep}
    return res, fn, 4.0 * pairs * a.nq * a.hd, n * (2 * a.nq + 2 * a.nkv) * a.hd * 2


def bench_window_decode(a):
    from tah_b200.engine.hybrid import decode_splits
    B, T = a.rows, a.ctx
    pool, pt = _paged(B, T, a.nkv, a.hd, a.hd)
    q, out, gate = _bf(B, a.nq * a.hd), torch.empty(B, a.nq * a.hd, dtype=torch.bfloat16, device="cuda"), None if a.softcap else _bf(B, a.nq)
    pos, row, kw = _i32([T - 1] * B), _i32(list(range(B))), _window_kw(a)
    ws = torch.empty(B * a.nq * a.nsplit * (a.hd + 2), device="cuda")
    fn = lambda i: K.window_attn_decode(q, out, pool, pt, pos, row, gate=gate, n_split=a.nsplit, ws=ws, **kw)
    keys = B * _visible(T - 1, a)
    res = {"op": "window_decode", "rows": B, "ctx": T, "window": a.window, "n_split": a.nsplit}
    return res, fn, 4.0 * keys * a.nq * a.hd, keys * a.nkv * 2 * a.hd * 2


def _tied_kw(a, pages):
    """Tied layers: ``--block`` P pooled blocks in front of the window, or with 0 key factors and slopes."""
    from tah_b200.engine.kv_cache import LayerKV
    kw = dict(nq=a.nq, nkv=a.nkv, dk=a.hd, dv=a.hd, page_size=16, scale=a.hd ** -0.5, window=a.window or 2 ** 31 - 1, keep_first=0, tied=True)
    if not a.block:
        return dict(kw, factor=torch.rand(pages, 16, device="cuda"), slope=torch.tensor([2.0 ** (-8 * (h + 1) / a.nq) for h in range(a.nq)], device="cuda"))
    S = LayerKV(block=a.block).pool_rows(16)
    return dict(kw, pooled=_bf(pages, a.nkv * S * a.hd), block=a.block, pool_rows=S)


def _blocks(i, a):
    return max(0, i - a.window + 1) // a.block if a.block else 0


def bench_tied_prefill(a):
    """The like of ``window_prefill``: values that are the keys.  FLOPs: visible keys and block means."""
    B, T, a.keep = a.rows, a.ctx, 0
    n = B * T
    pool, pt = _paged(B, T, a.nkv, a.hd, 0)
    q, out = _bf(n, a.nq * a.hd), torch.empty(n, a.nq * a.hd, dtype=torch.bfloat16, device="cuda")
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    q0 = [b * T + t for b in range(B) for t in range(0, T, 128)]
    qn = [min(128, T - t) for b in range(B) for t in range(0, T, 128)]
    kw, per = _tied_kw(a, pool.shape[0]), (_blocks(T - 1, a) + 15) // 16
    if a.block:
        kw["pooled"] = _bf(B * per * 16, a.nkv * a.hd) if per else None
        kw["pool_base"] = _i32([b * per for b in range(B) for _ in range(0, T, 128)])
    else:
        kw["wide_gate"] = _bf(n, a.nq * a.hd)
    q0, qn = _i32(q0), _i32(qn)
    fn = lambda i: K.window_attn_tiles(q, out, pool, pt, pos, row, q0, qn, pool.shape[0], **kw)
    pairs = B * sum(_visible(i, a) + _blocks(i, a) for i in range(T))
    res = {"op": "tied_prefill", "seqs": B, "T": T, "window": a.window, "block": a.block}
    return res, fn, 4.0 * pairs * a.nq * a.hd, n * (2 * a.nq + a.nkv + (0 if a.block else a.nq)) * a.hd * 2


def bench_tied_decode(a):
    B, T, a.keep = a.rows, a.ctx, 0
    pool, pt = _paged(B, T, a.nkv, a.hd, 0)
    q, out, kw = _bf(B, a.nq * a.hd), torch.empty(B, a.nq * a.hd, dtype=torch.bfloat16, device="cuda"), _tied_kw(a, pool.shape[0])
    if not a.block:
        kw["wide_gate"] = _bf(B, a.nq * a.hd)
    pos, row = _i32([T - 1] * B), _i32(list(range(B)))
    ws = torch.empty(B * a.nq * a.nsplit * (a.hd + 2), device="cuda")
    fn = lambda i: K.window_attn_decode(q, out, pool, pt, pos, row, n_split=a.nsplit, ws=ws, **kw)
    keys = B * (_visible(T - 1, a) + _blocks(T - 1, a))
    res = {"op": "tied_decode", "rows": B, "ctx": T, "window": a.window, "block": a.block, "n_split": a.nsplit}
    return res, fn, 4.0 * keys * a.nq * a.hd, keys * (a.nkv * a.hd * 2 + (0 if a.block else 4)) + B * a.nq * a.hd * (4 if a.block else 6)


def bench_tied_keys(a):
    """``--m`` tokens of rows of ``--ctx``."""
    from tah_b200.engine.kv_cache import LayerKV
    M, T = a.m, min(a.ctx, a.m)
    pages, S = M // 16, LayerKV(block=a.block or 16).pool_rows(16)
    k, pool, means = _bf(M, a.nkv * a.hd + 2048), _bf(pages, a.nkv * 16 * a.hd), _bf(pages, a.nkv * S * a.hd)
    slot = torch.arange(M, device="cuda", dtype=torch.int32)
    pt, pos, row = torch.arange(pages, device="cuda", dtype=torch.int32).view(M // T, -1), slot % T, slot // T
    fn = lambda i: K.tied_keys(k, pool, slot, pos, row, pt, a.nkv, a.hd, 16, means, a.block or 16, S)
    return {"op": "tied_keys", "M": M, "block": a.block or 16}, fn, 0.0, M * a.nkv * a.hd * 4 * (1 + 1 / (a.block or 16))


def bench_norm_all(a):
    M, F = a.m, (a.nq + a.nkv) * a.hd
    x, q = _bf(M, F + 64), torch.empty(M, a.nq * a.hd, dtype=torch.bfloat16, device="cuda")
    pages = (M + 15) // 16
    pool, fac, slot = _bf(pages, a.nkv * 16 * a.hd), torch.empty(pages, 16, device="cuda"), torch.arange(M, device="cuda", dtype=torch.int32)
    w = torch.ones(a.nq * a.hd, device="cuda")
    fn = lambda i: K.norm_all(x[:, :a.nq * a.hd], x[:, a.nq * a.hd:F], w, q, pool, fac, slot, nq=a.nq, nkv=a.nkv, dk=a.hd, dim=a.hd, page_size=16, eps=1e-6)
    return {"op": "norm_all", "M": M}, fn, 0.0, 2 * M * F * 2


def _gru_case(a, n, rows):
    D = a.f
    x, out = _bf(n, 3 * D), torch.empty(n, D, dtype=torch.bfloat16, device="cuda")
    return (x, torch.full((D,), -2.0, device="cuda"), torch.zeros(D, device="cuda"), out, (torch.zeros(rows, D, device="cuda"),))


def bench_min_gru_scan(a):
    """``--f`` channels; ``--nsplit`` 0: the engine's choice."""
    from types import SimpleNamespace
    from tah_b200.engine.hybrid import gru_splits
    B, T, D = a.rows, a.ctx, a.f
    ops = _gru_case(a, B * T, B)
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    split = a.nsplit or gru_splits(SimpleNamespace(d=D), B, T)
    ws = torch.empty(B * split * 2 * D, device="cuda")
    start, lens = _i32([b * T for b in range(B)]), _i32([T] * B)
    fn = lambda i: K.min_gru_scan(*ops, pos, row, 0.7, seq_start=start, seq_len=lens, n_split=split, ws=ws)
    return {"op": "min_gru_scan", "seqs": B, "T": T, "D": D, "n_split": split}, fn, 0.0, B * T * D * 8 + B * D * 8


def bench_min_gru_step(a):
    B, D = a.rows, a.f
    ops, pos, row = _gru_case(a, B, B), _i32([5] * B), _i32(list(range(B)))
    fn = lambda i: K.min_gru_step(*ops, pos, row, 0.7)
    return {"op": "min_gru_step", "rows": B, "D": D}, fn, 0.0, B * D * 16


def bench_xielu_product(a):
    """The like of a plain product of the same size (``gemm``) and of the SwiGLU product."""
    x, w, out = _bf(a.m, a.k), _bf(a.f, a.k), torch.empty(a.m, a.f, dtype=torch.bfloat16, device="cuda")
    fn = lambda i: K.xielu_linear(x, w, 0.9, 1.2, out=out)
    return {"op": "xielu_product", "M": a.m, "K": a.k, "F": a.f}, fn, 2.0 * a.m * a.k * a.f, (a.m * (a.k + a.f) + a.k * a.f) * 2


def _mlstm_case(a, n, rows):
    H, dk, dv = a.nkv, a.hd, a.dv
    F = H * (2 * dk + 2 * dv)
    x, z, out = _bf(n, F), torch.randn(n, 2 * H, device="cuda"), torch.empty(n, H * dv, dtype=torch.bfloat16, device="cuda")
    z[:, H:] += 4.0
    state = tuple(torch.zeros(rows, *s, device="cuda") for s in ((H, dk, dv), (H, dk), (H,)))
    return x, z, torch.ones(H * dv, device="cuda"), out, state, dict(heads=H, dk=dk, dv=dv, dim=dk, vdim=dv, cap=15.0, eps=1e-6)


def bench_mlstm_chunks(a):
    B, T = a.rows, a.ctx
    n, H, dk, dv = B * T, a.nkv, a.hd, a.dv
    x, z, nw, out, state, kw = _mlstm_case(a, n, B)
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    starts = [b * T + t for b in range(B) for t in range(0, T, 128)]
    lens = [min(128, T - t) for b in range(B) for t in range(0, T, 128)]
    per = (T + 127) // 128
    ws = torch.empty(K.mlstm_chunk_ws_floats(len(starts), H, dk, dv), device="cuda")
    c = dict(chunk_start=_i32(starts), chunk_len=_i32(lens), seq_chunk0=_i32([b * per for b in range(B)]), seq_chunks=_i32([per] * B))
    fn = lambda i: K.mlstm_chunks(x, z, nw, out, state, pos, row, ws=ws, **c, **kw)
    flops = H * sum(l * (l + 1) * (dk + dv) + 4.0 * l * dk * dv for l in lens)
    byts = n * H * ((2 * dk + 3 * dv) * 2 + 8) + B * H * dk * dv * 8
    return {"op": "mlstm_chunks", "seqs": B, "T": T, "heads": H, "dk": dk, "dv": dv}, fn, flops, byts


def bench_mlstm_step(a):
    B, H, dk, dv = a.rows, a.nkv, a.hd, a.dv
    x, z, nw, out, state, kw = _mlstm_case(a, B, B)
    pos, row = _i32([5] * B), _i32(list(range(B)))
    fn = lambda i: K.mlstm_recurrent(x, z, nw, out, state, pos, row, **kw)
    return {"op": "mlstm_step", "rows": B, "heads": H, "dk": dk, "dv": dv}, fn, 6.0 * B * H * dk * dv, B * H * (dk * dv * 8 + (2 * dk + 3 * dv) * 2)


def _gla_case(a, n, rows):
    H, dk, dv, rank = a.nkv, a.hd, a.dv, 16
    x, low, out = _bf(n, H * (2 * dk + 2 * dv)), torch.randn(n, rank, device="cuda"), torch.empty(n, H * dv, dtype=torch.bfloat16, device="cuda")
    w2, b2 = _bf(H * dk, rank) / 4, torch.full((H * dk,), 2.0, device="cuda")
    state = (torch.zeros(rows, H, dk, dv, device="cuda"),)
    return (x, low, w2, b2, torch.ones(dv, device="cuda"), out, state), dict(heads=H, dk=dk, dv=dv, dim=dk, vdim=dv, tau=a.tau, eps=1e-6)


def bench_gla_chunks(a):
    """The like of ``mlstm_chunks``; ``--tau`` 16 has no steep channels, small values do."""
    B, T = a.rows, a.ctx
    n, H, dk, dv = B * T, a.nkv, a.hd, a.dv
    ops, kw = _gla_case(a, n, B)
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    starts = [b * T + t for b in range(B) for t in range(0, T, 128)]
    lens = [min(128, T - t) for b in range(B) for t in range(0, T, 128)]
    per = (T + 127) // 128
    ws = torch.empty(K.gla_chunk_ws_floats(n, len(starts), H, dk, dv), device="cuda")
    c = dict(chunk_start=_i32(starts), chunk_len=_i32(lens), seq_chunk0=_i32([b * per for b in range(B)]), seq_chunks=_i32([per] * B))
    fn = lambda i: K.gla_chunks(*ops, pos, row, ws=ws, **c, **kw)
    flops = H * sum(l * (l + 1) * (dk + dv) + 4.0 * l * dk * dv for l in lens)
    byts = n * (H * (2 * dk + 3 * dv) * 2 + 64) + B * H * dk * dv * 8
    return {"op": "gla_chunks", "seqs": B, "T": T, "heads": H, "dk": dk, "dv": dv, "tau": a.tau}, fn, flops, byts


def bench_gla_step(a):
    B, H, dk, dv = a.rows, a.nkv, a.hd, a.dv
    ops, kw = _gla_case(a, B, B)
    pos, row = _i32([5] * B), _i32(list(range(B)))
    fn = lambda i: K.gla_recurrent(*ops, pos, row, **kw)
    return {"op": "gla_step", "rows": B, "heads": H, "dk": dk, "dv": dv}, fn, 6.0 * B * H * dk * dv, B * H * (dk * dv * 8 + (2 * dk + 3 * dv) * 2)


def bench_latent_decode(a):
    """``--nq`` heads over cached rows of ``--rank`` + ``--rot``; ``--nsplit`` 0: the engine's choice."""
    B, T, H, R, rw = a.rows, a.ctx, a.nq, a.rank, a.rot
    lq = (R + rw + 63) // 64 * 64
    pool, pt = _paged(B, T, 1, R + rw, 0)
    L = K.HeadLists(B, H, torch.bfloat16, "cuda")
    q, out, sink = _bf(L.rows, lq), torch.empty(L.rows, R, dtype=torch.bfloat16, device="cuda"), torch.randn(H, device="cuda")
    split = a.nsplit
    if split == 0:
        from types import SimpleNamespace
        from tah_b200.engine.hybrid import latent_splits
        split = latent_splits(SimpleNamespace(on_tensor_cores=True, spec=SimpleNamespace(heads=H, window=a.latent_window or None)), B)
    pos, row, ws = _i32([T - 1] * B), _i32(list(range(B))), torch.empty(B * H * split * (R + 2), device="cuda")
    fn = lambda i: K.latent_attn_decode(q, out, pool, pt, pos, row, L, Rp=R, rw=rw, page_size=16, scale=0.07, sink=sink, n_split=split, ws=ws,
                                        window=a.latent_window or 2 ** 31 - 1)
    T = min(T, a.latent_window or T)
    return {"op": "latent_decode", "rows": B, "ctx": a.ctx, "window": a.latent_window, "heads": H, "rank": R, "rot": rw, "n_split": split}, fn, \
        2.0 * B * T * H * (2 * R + rw), B * T * (R + rw) * 2 + B * H * (2 * R + rw) * 2


def bench_latent_prefill(a):
    """Attention of portions over expanded keys and values: ``--nq`` heads, keys of ``--hd`` + ``--rot``, values of ``--hd``."""
    B, T, H, dk, dv = a.rows, a.ctx, a.nq, a.hd + a.rot, a.hd
    n, pages = B * T, B * ((T + 15) // 16)
    kv = _bf(pages * 16, H * (dk + dv))
    pt = torch.arange(pages, device="cuda", dtype=torch.int32).view(B, -1)
    q, out, gate = _bf(n, H * dk), torch.empty(n, H * dv, dtype=torch.bfloat16, device="cuda"), _bf(n, H * dv)
    pos = torch.arange(T, device="cuda", dtype=torch.int32).repeat(B)
    row = torch.arange(B, device="cuda", dtype=torch.int32).repeat_interleave(T)
    q0 = _i32([b * T + t for b in range(B) for t in range(0, T, 128)])
    qn = _i32([min(128, T - t) for b in range(B) for t in range(0, T, 128)])
    sink = torch.randn(H, device="cuda")
    fn = lambda i: K.window_attn_tiles(q, out, kv, pt, pos, row, q0, qn, pages, kv_ld=kv.shape[1], nq=H, nkv=H, dk=dk, dv=dv, page_size=16,
                                       scale=dk ** -0.5, window=a.latent_window or 2 ** 31 - 1, keep_first=0, sink=sink, wide_gate=gate)
    seen = B * sum(min(i + 1, a.latent_window or T) for i in range(T))
    return {"op": "latent_prefill", "seqs": B, "T": T, "window": a.latent_window, "heads": H, "dk": dk, "dv": dv}, fn, 2.0 * seen * H * (dk + dv), \
        n * H * (2 * dk + 3 * dv) * 2


def bench_latent_post(a):
    M, Q, R, rw = a.m, a.k, a.rank, a.rot
    proj, cq = _bf(M, Q + R + rw + 64), torch.empty(M, Q, dtype=torch.bfloat16, device="cuda")
    pool, slot = _bf((M + 15) // 16, 16 * (R + rw)), torch.arange(M, device="cuda", dtype=torch.int32)
    w, rope = torch.ones(max(Q, R), device="cuda"), torch.randn(M, rw // 2, 2, device="cuda")
    fn = lambda i: K.latent_post(proj, w, w, rope, cq, pool, slot, q_rank=Q, q_col=0, kv_rank=R, Rp=R, c_col=Q, rot=rw, rw=rw, r_col=Q + R, eps=1e-6)
    return {"op": "latent_post", "M": M, "q_rank": Q, "rank": R}, fn, 0.0, M * ((Q + R + rw) * 4 + rw * 4)


def bench_latent_query(a):
    """In place for portions (``--lists`` 0) or into head lists."""
    M, H, d, r = a.m, a.nq, a.hd, a.rot
    dk, lists = d + r, K.HeadLists(a.m, a.nq, torch.bfloat16, "cuda") if a.lists else None
    q, rope = _bf(M, H * dk), torch.randn(M, r // 2, 2, device="cuda")
    out = _bf(lists.rows, (dk + 63) // 64 * 64) if a.lists else None
    fn = lambda i: K.latent_query(q, rope, lists, out, heads=H, dk=dk, dim=d, rot=r)
    return {"op": "latent_query", "M": M, "lists": bool(a.lists)}, fn, 0.0, M * H * (dk if a.lists else r) * 4 + M * r * 4


def bench_latent_gather(a):
    pages, row = a.m // 16, a.rank + a.rot
    pool, src = _bf(pages, 16 * row), torch.randperm(pages, device="cuda").to(torch.int32)
    out = _bf(pages * 16, (row + 63) // 64 * 64)
    return {"op": "latent_gather", "tokens": a.m}, lambda i: K.latent_gather(pool, src, 16, row, out), 0.0, a.m * (row + out.shape[1]) * 2


def bench_latent_gate(a):
    M, H, dv = a.m, a.nq, a.hd
    L = K.HeadLists(M, H, torch.bfloat16, "cuda")
    v, g, out = _bf(L.rows, dv), _bf(M, H * dv), torch.empty(M, H * dv, dtype=torch.bfloat16, device="cuda")
    return {"op": "latent_gate", "M": M}, lambda i: K.latent_gate(v, L, g, out, dv), 0.0, M * H * dv * 6


def bench_head_product(a):
    """Grouped product over head lists: ``--f`` outputs of ``--k`` inputs for each of ``--nq`` heads."""
    L = K.HeadLists(a.m, a.nq, torch.bfloat16, "cuda")
    x, w, out = _bf(L.rows, a.k), _bf(a.nq, a.f, a.k), torch.empty(L.rows, a.f, dtype=torch.bfloat16, device="cuda")
    return {"op": "head_product", "M": a.m, "heads": a.nq, "K": a.k, "F": a.f}, lambda i: K.moe_linear(x, w, L, out), \
        2.0 * a.m * a.nq * a.k * a.f, (w.numel() + a.m * a.nq * (a.k + a.f)) * 2


def bench_streams_norm(a):
    """``--streams`` residual streams; ``--topk`` weighted expert rows per token instead of one row when ``--experts`` is given."""
    M, W, S, top = a.m, a.k, a.streams, a.topk if a.experts else 0
    y, x, h = _bf(M, W), torch.randn(M, S, W, device="cuda"), torch.empty(M, W, dtype=torch.bfloat16, device="cuda")
    hc = torch.cat([0.5 * torch.eye(S).flatten(), torch.full((2 * S,), 0.5)]).cuda()
    w = torch.full((W,), 0.5, device="cuda")
    ex = dict(y_ex=_bf(M * top, W), slot=torch.randperm(M * top, device="cuda").to(torch.int32).view(M, top),
              y_weight=torch.rand(M, top, device="cuda")) if top else {}
    fn = lambda i: K.streams_norm(None if top else y, x, hc, w, W, 1, 1e-6, h, **ex)
    return {"op": "streams_norm", "M": M, "W": W, "streams": S, "experts": top}, fn, 0.0, M * W * (2 * max(1, top) + 8 * S + 2)


def bench_rotary_table(a):
    M, half = a.m, a.rot // 2
    pos, freq, out = torch.arange(M, device="cuda", dtype=torch.int32), torch.rand(2, half, device="cuda"), torch.empty(M, half, 2, device="cuda")
    return {"op": "rotary_table", "M": M, "half": half}, lambda i: K.rotary_table(pos, freq, 1.1, out), 0.0, M * (half * 8 + 4)


def bench_residual_norm(a):
    M, W = a.m, a.k
    y, x, h = _bf(M, W), torch.randn(M, W, device="cuda"), torch.empty(M, W, dtype=torch.bfloat16, device="cuda")
    w = torch.full((W,), 0.5, device="cuda")
    enter = dict(add=w, embedding=(_bf(1000, W), torch.randint(0, 1000, (M,), device="cuda").to(torch.int32), 0.5)) if a.enter else {}
    fn = lambda i: K.residual_norm(y, x, w, w, W, 1e-6, h, centered=a.centered, **enter)
    return {"op": "residual_norm", "M": M, "W": W, "centered": a.centered, "enter": a.enter}, fn, 0.0, M * W * (2 + 8 + 2)


def bench_qkv_post(a):
    M = a.m
    F = (a.nq + 2 * a.nkv) * a.hd
    qkv, q = _bf(M, F + 64), torch.empty(M, a.nq * a.hd, dtype=torch.bfloat16, device="cuda")
    pool = _bf((M + 15) // 16, a.nkv * 16 * 2 * a.hd)
    slot = torch.arange(M, device="cuda", dtype=torch.int32)
    b, w = torch.randn(F + 64, device="cuda"), torch.ones(a.hd, device="cuda")
    kw, extra = {}, 0
    if a.rotate:                              # rotation of --rot dims and mixed values instead of the norms
        kw = dict(rope=torch.randn(M, a.rot // 2, 2, device="cuda"), rot=a.rot, v_first=_bf(M, a.nkv * a.hd), lam=torch.full((1,), 0.3, device="cuda"))
        w, extra = None, M * (a.rot * 4 + a.nkv * a.hd * 2)
    fn = lambda i: K.qkv_post(qkv, b, w, w, q, pool, slot, a.nq, a.nkv, a.hd, a.hd, a.hd, 16, 1e-6, **kw)
    return {"op": "qkv_post", "M": M, "rotate": bool(a.rotate)}, fn, 0.0, 2 * M * F * 2 + extra


def bench_qk_norm_rope(a):
    """The like kernel of the Qwen3 engine."""
    M = a.m
    F = (a.nq + 2 * a.nkv) * a.hd
    qkv, q = _bf(M, F), torch.empty(M, a.nq * a.hd, dtype=torch.bfloat16, device="cuda")
    pool = torch.zeros((M + 15) // 16, 2, a.nkv, 16, a.hd, dtype=torch.bfloat16, device="cuda")
    slot = torch.arange(M, device="cuda", dtype=torch.int32)
    w = torch.ones(a.hd, device="cuda", dtype=torch.bfloat16)
    fn = lambda i: K.qk_norm_rope_kv(qkv, w, w, slot, a.nq, a.nkv, a.hd, 1e-6, 1e6, q_out=q, caches=[pool], slot=slot)
    return {"op": "qk_norm_rope", "M": M}, fn, 0.0, 2 * M * F * 2


def bench_few_linear(a):
    M, W, F = a.m, a.k, a.f
    x, w, b, out = _bf(M, W), _bf(F, W), torch.randn(F, device="cuda"), torch.empty(M, F, device="cuda")
    fn = lambda i: K.few_linear(x, w, b, out=out)
    return {"op": "few_linear", "M": M, "K": W, "F": F}, fn, 2.0 * M * W * F, (M * W + F * W) * 2 + M * F * 4


def bench_residual_add_norm(a):
    """``--topk`` expert rows per token when ``--experts`` is given."""
    M, W, top = a.m, a.k, a.topk if a.experts else 0
    y, x, h = _bf(M, W), torch.randn(M, W, device="cuda"), torch.empty(M, W, dtype=torch.bfloat16, device="cuda")
    w = torch.full((W,), 0.5, device="cuda")
    ex = _bf(M * top, W) if top else None
    slot = torch.randperm(M * top, device="cuda").to(torch.int32).view(M, top) if top else None
    fn = lambda i: K.residual_add_norm(y, x, 0.5, w, W, 4, 1e-6, h, ex, slot)
    return {"op": "residual_add_norm", "M": M, "W": W, "experts": top}, fn, 0.0, M * W * (2 + 8 + 2 + 2 * top)


def bench_poly_norm(a):
    M, F = a.m, a.f
    z, out, act = _bf(M, F), torch.empty(M, F, dtype=torch.bfloat16, device="cuda"), torch.tensor([0.6, -0.4, 0.3, 0.1], device="cuda")
    fn = lambda i: K.poly_norm(z, act, F, 1e-6, out)
    return {"op": "poly_norm", "M": M, "F": F}, fn, 0.0, M * F * 4


def bench_swiglu(a):
    """The like kernel of the training path: an activation over rows in a launch of its own."""
    M, F = a.m, a.f
    z, out = _bf(M, 2 * F), torch.empty(M, F, dtype=torch.bfloat16, device="cuda")
    return {"op": "swiglu", "M": M, "F": F}, lambda i: K.swiglu(z, out=out), 0.0, M * F * 6


def bench_clamped_glu(a):
    M, F = a.m, a.f
    z, out, gate = _bf(M, 2 * F), torch.empty(M, F, dtype=torch.bfloat16, device="cuda"), torch.randn(M, 8, device="cuda")
    fn = lambda i: K.clamped_glu(z, 7.0, out, gate=gate[:, 3])
    return {"op": "clamped_glu", "M": M, "F": F}, fn, 0.0, M * F * 6


def _lists(a):
    L = K.ExpertLists(a.m, a.experts, a.topk, torch.bfloat16, "cuda", bn=a.bn or None)
    z = torch.randn(a.m, a.experts + 1, device="cuda")
    K.moe_route(z, L)
    return L, z


def bench_moe_route(a):
    L, z = _lists(a)
    return {"op": "moe_route", "M": a.m, "experts": a.experts, "top": a.topk, "softmax": bool(a.plain_glu)}, \
        lambda i: K.moe_route(z, L, softmax=bool(a.plain_glu)), 0.0, \
        a.m * (4 * a.experts + 12 * a.topk)


def bench_moe_gather(a):
    L, _ = _lists(a)
    h, x = _bf(a.m, a.k), torch.empty(L.rows, a.k, dtype=torch.bfloat16, device="cuda")
    return {"op": "moe_gather", "M": a.m, "top": a.topk}, lambda i: K.moe_gather(h, L, x), 0.0, a.m * a.k * 2 * (1 + a.topk)


def _moe(a, glu):
    """FLOPs of the (token, expert) pairs; bytes: weights of the experts in use, list rows in and out."""
    L, _ = _lists(a)
    K.moe_gather(_bf(a.m, 64), L, torch.empty(L.rows, 64, dtype=torch.bfloat16, device="cuda"))
    Kd, F = (a.k, 2 * a.f) if glu else (a.f, a.k)
    x, w = _bf(L.rows, Kd), _bf(a.experts, F, Kd)
    out = torch.empty(L.rows, a.f if glu else a.k, dtype=torch.bfloat16, device="cuda")
    form = dict(slope=1.0, offset=0.0, weighted=False) if a.plain_glu else {}
    fn = (lambda i: K.moe_glu_linear(x, w, float("inf") if a.plain_glu else 7.0, L, out, **form)) if glu else (lambda i: K.moe_linear(x, w, L, out))
    pairs, used = a.m * a.topk, int(L.expert.unique().numel())
    return {"op": "moe_glu" if glu else "moe_down", "M": a.m, "experts": a.experts, "top": a.topk, "bn": L.bn,
            "rows": int(L.n_blocks) * L.bn}, fn, 2.0 * pairs * F * Kd, used * F * Kd * 2 + pairs * (Kd + out.shape[1]) * 2


def bench_moe_glu(a):
    return _moe(a, True)


def bench_moe_down(a):
    return _moe(a, False)


CASES = {"tied_prefill": bench_tied_prefill, "tied_decode": bench_tied_decode, "tied_keys": bench_tied_keys, "norm_all": bench_norm_all,
         "min_gru_scan": bench_min_gru_scan, "min_gru_step": bench_min_gru_step, "xielu_product": bench_xielu_product,
         "window_prefill": bench_window_prefill, "window_decode": bench_window_decode, "mlstm_chunks": bench_mlstm_chunks,
         "mlstm_step": bench_mlstm_step, "residual_norm": bench_residual_norm, "qkv_post": bench_qkv_post,
         "qk_norm_rope": bench_qk_norm_rope, "few_linear": bench_few_linear, "residual_add_norm": bench_residual_add_norm,
         "poly_norm": bench_poly_norm, "clamped_glu": bench_clamped_glu, "swiglu": bench_swiglu, "moe_route": bench_moe_route,
         "gla_chunks": bench_gla_chunks, "gla_step": bench_gla_step, "latent_decode": bench_latent_decode,
         "latent_prefill": bench_latent_prefill, "latent_post": bench_latent_post, "latent_query": bench_latent_query,
         "latent_gather": bench_latent_gather, "latent_gate": bench_latent_gate, "head_product": bench_head_product,
         "streams_norm": bench_streams_norm, "rotary_table": bench_rotary_table, "moe_gather": bench_moe_gather, "moe_glu": bench_moe_glu, "moe_down": bench_moe_down}
