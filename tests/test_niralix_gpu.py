"""Niralix on the GPU: every mechanism against a plain statement of it, and the engine's steps, ticks and scheduler."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from tests import niralix_helpers as H
from tests.oracle import niralix_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16


def engine(d, dtype, rows=4, pool=2048, **kw):
    from tah_b200.models import load_model, make_engine
    e = make_engine(load_model(d, dtype, "cuda"), max_rows=rows, **kw)
    e.open(rows, pool)
    return e


def run_portions(e, toks, portions):
    """Feed one request in portions; logits of every token."""
    from tah_b200.engine import StepEntry
    row, at, out = e.admit(), 0, []
    for c in portions:
        out.append(e.step([StepEntry(row, toks[at:at + c], range(c))]).float().cpu())
        at += c
    assert at == len(toks)
    e.release(row)
    return torch.cat(out)


def check_ok():
    from tah_b200.ops import cuda as K
    torch.cuda.synchronize()
    K.check_status()


def _i32(x):
    return torch.tensor(list(x), dtype=torch.int32, device="cuda")


def _pad(n, m):
    return (n + m - 1) // m * m


def _err(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def _rope(rot, pos):
    """The engine's table of (cos, sin) for a rotation given as in config.json."""
    from tah_b200.models.niralix import _rotary
    from tah_b200.ops import cuda as K
    f, m = _rotary(rot, False).frequencies()
    f = torch.tensor(f, dtype=torch.float64)
    freq = torch.stack([f.float(), (f - f.float().double()).float()]).contiguous().cuda()
    return K.rotary_table(pos, freq, m, torch.empty(len(pos), rot["dims"] // 2, 2, device="cuda"))


# ------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [dict(dims=64, base=1e4), dict(dims=2, base=3.0), dict(dims=24, base=1e6, scaling=dict(factor=8.0, original=1024, fast=20, slow=2)),
                                 dict(dims=128, base=5e5, scaling=dict(factor=40.0, original=4096, fast=16, slow=2))])
def test_rotary_table(rot):
    pos = [0, 1, 2, 63, 1000, 4095, 40000, 131071]
    tab = _rope(rot, _i32(pos)).cpu().double()
    f, m = O.rotary_frequencies(rot)
    for r, p in enumerate(pos):
        for i in range(rot["dims"] // 2):
            assert abs(float(tab[r, i, 0]) - m * math.cos(p * f[i])) < 1e-6 and abs(float(tab[r, i, 1]) - m * math.sin(p * f[i])) < 1e-6
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", [(4, 2, 40, 24, 20), (3, 1, 18, 33, 6), (2, 2, 128, 64, 128), (5, 5, 200, 136, 66), (1, 1, 7, 9, 2)])
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("normed", [False, True])
def test_rotation_and_mixed_values_behind_the_projection(dtype, case, interleaved, normed):
    from tah_b200.ops import cuda as K
    nq, G, dim, vdim, rd = case
    dk, dv, page, M = _pad(dim, 8), _pad(vdim, 8), 16, 21
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v, first = (rnd(M, h, d).to(dtype) for h, d in ((nq, dim), (G, dim), (G, vdim), (G, vdim)))
    bq, bk, bv, wq, wk = rnd(nq, dim), rnd(G, dim), rnd(G, vdim), 1 + 0.2 * rnd(dim), 1 + 0.2 * rnd(dim)
    padh = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1]))
    flat = lambda *ts: torch.cat([t.flatten(-2) for t in ts], -1)
    qkv = torch.full((M, (nq + G) * dk + G * dv + 16), 2.0)
    row = flat(padh(q, dk), padh(k, dk), padh(v, dv))
    qkv[:, :row.shape[1]] = row
    bias = flat(padh(bq, dk), padh(bk, dk), padh(bv, dv)).cuda()
    rot = dict(dims=rd, base=700.0, scaling=dict(H.YARN))
    pos = torch.randint(0, 5000, (M,), generator=g).to(torch.int32)
    rope = _rope(rot, pos.cuda())
    slot = torch.randperm(64, generator=g)[:M].to(torch.int32)
    slot[3] = -1
    pool = torch.zeros(4, G * page * (dk + dv), dtype=dtype, device="cuda")
    out, keep = torch.zeros(M, nq * dk, dtype=dtype, device="cuda"), torch.zeros(M, G * dv, dtype=dtype, device="cuda")
    norms = (padh(wq, dk).cuda(), padh(wk, dk).cuda()) if normed else (None, None)
    args = (qkv.to("cuda", dtype), bias, *norms, out, pool, slot.cuda(), nq, G, dk, dv, dim, page, 1e-3)
    kw = dict(rope=rope, rot=rd, interleaved=interleaved)
    tol = 2e-5 if dtype == F32 else 1e-2
    n = lambda t, w: O.rms_norm(t, w.double(), 1e-3) if normed else t
    turn = lambda t: O.rotate(t, pos.tolist(), rot, interleaved)
    want_q, want_k = turn(n(q.double() + bq.double(), wq)), turn(n(k.double() + bk.double(), wk))
    own = v.double() + bv.double()

    def compare(want_v):
        assert _err(out.view(M, nq, dk)[..., :dim], want_q) < tol
        pc = pool.cpu().double()
        for t in range(M):
            s = int(slot[t])
            if s < 0:
                continue
            kt = pc[s // page][:G * page * dk].view(G, page, dk)[:, s % page]
            vt = pc[s // page][G * page * dk:].view(G, page, dv)[:, s % page]
            assert float((kt[:, :dim] - want_k[t]).abs().max()) < tol * float(want_k.abs().max())
            assert float((vt[:, :vdim] - want_v[t]).abs().max()) < tol * float(want_v.abs().max())
            assert float(kt[:, dim:].abs().sum()) == 0 and float(vt[:, vdim:].abs().sum()) == 0

    K.qkv_post(*args, v_keep=keep, **kw)
    compare(own)
    assert _err(keep.view(M, G, dv)[..., :vdim], own) < tol
    K.qkv_post(*args, v_first=padh(first, dv).reshape(M, -1).contiguous().cuda(), lam=torch.full((1,), 0.3, device="cuda"), **kw)
    compare(0.7 * own + 0.3 * first.double())
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 8])
def test_residual_streams(dtype, S):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(S)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == F32 else 1e-2
    for width, ld, M in ((512, 512, 5), (77, 128, 9), (2048, 2048, 3), (132, 192, 40), (5000, 5056, 2)):
        z = lambda t: torch.nn.functional.pad(t, (0, ld - width))
        E, w, w2, w_in = rnd(50, width).to(dtype), rnd(width), rnd(width), rnd(S)
        ids = torch.randint(0, 50, (M,), generator=g).to(torch.int32)
        x, h = torch.full((M, S, ld), 9.0, device="cuda"), torch.empty(M, ld, dtype=dtype, device="cuda")
        K.embed_norm(z(E).cuda(), ids.cuda(), 1.0, z(w).cuda(), width, 1e-4, x, h, streams=S, w_in=w_in.cuda())
        xs = [E.double()[ids.long()]] * S
        assert _err(h[:, :width], O.rms_norm(O.streams_in(xs, w_in.double()), w.double(), 1e-4)) < tol
        for ex in (False, True):
            mix, out, nxt, bias = rnd(S, S), rnd(S), rnd(S), rnd(width)
            y, ye = rnd(M, width).to(dtype), rnd(11, width).to(dtype)
            slot, wt = torch.randint(0, 11, (M, 3), generator=g).to(torch.int32), torch.rand(M, 3, generator=g)
            hc = torch.cat([mix.flatten(), out, nxt]).cuda()
            if ex:
                K.streams_norm(None, x, hc, z(w2).cuda(), width, 1, 1e-4, h, y_ex=z(ye).cuda(), slot=slot.cuda(), y_weight=wt.cuda())
                full = (ye.double()[slot.long()] * wt.double().unsqueeze(-1)).sum(1)
            else:
                K.streams_norm(z(y).cuda(), x, hc, z(w2).cuda(), width, 1, 1e-4, h, y_bias=z(bias).cuda())
                full = y.double() + bias.double()
            xs = O.streams_out(xs, full, mix.double(), out.double())
            assert _err(x[..., :width], torch.stack(xs, 1)) < 1e-5
            assert _err(h[:, :width], O.rms_norm(O.streams_in(xs, nxt.double()), w2.double(), 1e-4)) < tol
        assert float(h[:, width:].float().abs().sum()) == 0 and float(x[..., width:].abs().sum()) == 0
    check_ok()


# T per portion, heads, dim, vdim, rank, tau, decay bias
GLA = [([1], 3, 24, 56, 12, 6.0, 2.0), ([150], 2, 128, 256, 16, 16.0, 2.0), ([128, 5, 260, 2], 3, 40, 24, 8, 3.0, 4.0), ([129], 1, 13, 19, 5, 1.0, 0.0),
       ([300, 17], 4, 72, 136, 20, 0.5, -2.0), ([257], 2, 64, 64, 16, 2.0, 8.0), ([140], 2, 128, 200, 32, 0.25, 1.0)]


@pytest.mark.parametrize("form", ["recurrent32", "recurrent", "chunks", "steps"])
@pytest.mark.parametrize("case", GLA)
@pytest.mark.parametrize("fresh", [True, False])
def test_gated_linear_attention(form, case, fresh):
    """Portions side by side from an empty and from a given state: outputs and the state they leave."""
    from tah_b200.ops import cuda as K
    lens, nh, dim, vdim, rank, tau, bias = case
    dtype = F32 if form == "recurrent32" else BF16
    dk, dv, rp, n = _pad(dim, 8), _pad(vdim, 8), _pad(rank, 4), sum(lens)
    g = torch.Generator().manual_seed(n)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v, gate = (rnd(n, nh, d).to(dtype).double() for d in (dim, dim, vdim, vdim))
    low, w2, b2, nw = rnd(n, rank).float().double(), (rnd(nh * dim, rank) / math.sqrt(rank)).to(dtype).double(), (bias + rnd(nh * dim)).float().double(), \
        (1 + 0.2 * rnd(vdim)).float().double()
    S0 = [torch.zeros(nh, dim, vdim, dtype=torch.float64) if fresh else rnd(nh, dim, vdim).float().double() for _ in lens]
    alpha = O.gla_decay((low @ w2.T + b2).view(n, nh, dim), tau)
    want, states, at = [], [], 0
    for c, s in zip(lens, S0):
        o, s = O.gla_core(q[at:at + c] * dim ** -0.5, k[at:at + c], v[at:at + c], alpha[at:at + c], s)
        want.append(o)
        states.append(s)
        at += c
    want = O.rms_norm(torch.cat(want), nw, 1e-4) * gate * torch.sigmoid(gate)
    pad = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1]))
    m = torch.full((n, 2 * nh * (dk + dv) + 64), 3.0, dtype=dtype, device="cuda")
    flat = torch.cat([pad(t, d).flatten(1) for t, d in ((q, dk), (k, dk), (v, dv), (gate, dv))], 1).to(dtype)
    m[:, :flat.shape[1]] = flat.cuda()
    w2p = pad(torch.nn.functional.pad(w2.view(nh, dim, rank), (0, 0, 0, dk - dim)), rp).reshape(nh * dk, rp).to("cuda", dtype)
    b2p = pad(b2.view(nh, dim), dk).reshape(-1).float().cuda()
    rows = torch.randperm(len(lens) + 2, generator=g)[:len(lens)]
    S = torch.full((len(lens) + 2, nh, dk, dv), float("nan") if fresh else 0.0, device="cuda")
    if not fresh:
        for r, s in zip(rows, S0):
            S[r, :, :dim, :vdim] = s.float().cuda()
    off = 0 if fresh else 1000
    pos, row = _i32([off + t for c in lens for t in range(c)]), _i32([int(r) for r, c in zip(rows, lens) for _ in range(c)])
    out = torch.zeros(n, nh * dv + 64, dtype=dtype, device="cuda")
    lowp = pad(low, rp).float().contiguous().cuda()
    kw = dict(heads=nh, dk=dk, dv=dv, dim=dim, vdim=vdim, tau=tau, eps=1e-4)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    nwp = pad(nw, dv).float().cuda()
    args = lambda sl=slice(None): (m[sl], lowp[sl], w2p, b2p, nwp, out[sl, :nh * dv], (S,), pos[sl], row[sl])
    if form == "chunks":
        tiles = [(s + a, min(128, c - a)) for s, c in zip(starts, lens) for a in range(0, c, 128)]
        per = [(c + 127) // 128 for c in lens]
        ws = torch.empty(K.gla_chunk_ws_floats(n, len(tiles), nh, dk, dv), device="cuda")
        K.gla_chunks(*args(), chunk_start=_i32(t for t, _ in tiles), chunk_len=_i32(c for _, c in tiles),
                     seq_chunk0=_i32(sum(per[:i]) for i in range(len(per))), seq_chunks=_i32(per), ws=ws, **kw)
    elif form == "steps":
        live, idle = _i32([5]), _i32([-1])
        for t in range(max(lens)):
            for s, c in zip(starts, lens):
                if t < c:
                    K.gla_recurrent(*args(slice(s + t, s + t + 1)), slot=live, **kw)
        before = S.clone()
        K.gla_recurrent(*args(slice(0, 1)), slot=idle, **kw)                 # an idle row keeps its state
        assert torch.equal(before.nan_to_num(), S.nan_to_num())
        out[0] = 0
    else:
        K.gla_recurrent(*args(), seq_start=_i32(starts), seq_len=_i32(lens), **kw)
    got = out[:, :nh * dv].double().cpu().view(n, nh, dv)
    first = 1 if form == "steps" else 0
    scale = want.abs().amax((1, 2)).clamp(min=0.2 * float(want.abs().max()))
    tol = 3e-5 if dtype == F32 else 1.2e-2
    assert float(((got[..., :vdim] - want).abs().amax((1, 2)) / scale)[first:].max() if n > first else 0.0) < tol
    assert float(out[:, nh * dv:].float().abs().sum()) == 0
    for r, s in zip(rows, states):
        assert _err(S[r, :, :dim, :vdim], s) < (1e-5 if form != "chunks" else 1e-4)
    check_ok()


LATENT = [  # T, heads, dim, rot, vdim, kv_rank
    (150, 3, 24, 12, 40, 72), (300, 16, 64, 64, 64, 512), (260, 36, 32, 16, 24, 192), (140, 1, 8, 2, 8, 8), (200, 20, 40, 64, 72, 64), (270, 5, 48, 72, 16, 320),
]


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode"])
@pytest.mark.parametrize("case", LATENT)
@pytest.mark.parametrize("peaked", [False, True])
def test_absorbed_latent_attention(kernel, case, peaked):
    """Queries against the cached rows themselves, for tokens at page and tile borders; with a sink that takes a share."""
    from tah_b200.ops import cuda as K
    T, nh, _, r, _, R = case
    dtype = F32 if kernel == "plain32" else BF16
    Rp, rw = _pad(R, 64), _pad(r, 64)
    g = torch.Generator().manual_seed(R)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, kk, sink = rnd(T, nh, R + r), rnd(T, 1, R + r), 2 * rnd(nh)
    if peaked:
        u = torch.nn.functional.normalize(rnd(R + r), dim=0) * math.sqrt(R + r)
        q, kk = 0.2 * q + 1.5 * u, 0.3 * kk
        for j in (0, 15, 16, 63, 64, 127, 128, T - 1):
            kk[j] = 3.0 * u + 0.5 * rnd(R + r)
    q, kk = q.to(dtype).double(), kk.to(dtype).double()
    scale = 1.0 / math.sqrt(R + r)
    want = O.attention_core(q, kk, kk[..., :R], scale, sink.double())
    n_pages = (T + 15) // 16
    perm = torch.randperm(n_pages + 3, generator=g)[:n_pages]
    pool = torch.zeros(n_pages + 3, 16, Rp + rw)
    for t in range(T):
        pool[perm[t // 16], t % 16, :R], pool[perm[t // 16], t % 16, Rp:Rp + r] = kk[t, 0, :R].float(), kk[t, 0, R:].float()
    pool = pool.view(n_pages + 3, -1).to("cuda", dtype)
    rows = list(range(T)) if kernel == "plain32" else sorted({p for p in (0, 1, 15, 16, 17, 63, 64, 99, 126, 127, 128, 129, T - 2, T - 1)})
    L = K.HeadLists(len(rows), nh, dtype, "cuda")
    lq = _pad(Rp + rw, 64)
    ql = torch.zeros(nh, L.npad, lq)
    ql[:, :len(rows), :R], ql[:, :len(rows), Rp:Rp + r] = q[rows, :, :R].transpose(0, 1).float(), q[rows, :, R:].transpose(0, 1).float()
    ql = ql.view(-1, lq).to("cuda", dtype)
    pt = perm.to("cuda", torch.int32).view(1, -1).contiguous()
    tol = 3e-5 if dtype == F32 else 2e-2
    kw = dict(Rp=Rp, rw=rw, page_size=16, scale=scale)
    at, zero, natural = _i32(rows), _i32([0] * len(rows)), sink.cuda()
    log2 = natural * 1.4426950408889634
    for split in (1, 2, 5) if kernel == "decode" else (1,):
        out = torch.full((L.rows, Rp), 7.0, dtype=dtype, device="cuda")
        a = (ql, out, pool, pt, at, zero, L)
        if kernel == "decode":
            assert K.latent_decode_fits(nh, Rp, rw)
            ws = torch.empty(len(rows) * nh * split * (Rp + 2), device="cuda")
            K.latent_attn_decode(*a, sink=log2, n_split=split, ws=ws, **kw)
        else:
            K.latent_attn_plain(*a, sink=natural, **kw)
        got = out.double().cpu().view(nh, L.npad, Rp)[:, :len(rows)].transpose(0, 1)
        err = (got[..., :R] - want[rows]).abs().amax((1, 2)) / want[rows].abs().amax((1, 2)).clamp(min=0.3 * float(want.abs().max()))
        assert float(err.max()) < tol, (split, err)
        assert float(got[..., R:].abs().max() if Rp > R else 0.0) == 0.0
    check_ok()


@pytest.mark.parametrize("heads", [16, 24])
def test_growing_scores_in_latent_decoding(heads):
    """Keys whose scores rise from tile to tile, in some heads only: the running maximum of a long row changes again and again."""
    from tah_b200.ops import cuda as K
    T, R, r = 700, 128, 64
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)
    u = torch.nn.functional.normalize(rnd(R + r), dim=0)
    kk = (0.5 * rnd(T, 1, R + r) + torch.linspace(-10, 10, T).view(T, 1, 1) * u).to(BF16).double()
    q = (rnd(1, heads, R + r) + torch.linspace(-8, 8, heads).view(1, heads, 1) * u).to(BF16).double()
    s = torch.einsum("ahd,tbd->ht", q, kk)
    want = torch.softmax(s, -1) @ kk[:, 0, :R]
    n_pages = (T + 15) // 16
    pool = torch.zeros(n_pages * 16, R + r)
    pool[:T] = kk[:, 0].float()
    L = K.HeadLists(1, heads, BF16, "cuda")
    ql = torch.zeros(heads, L.npad, R + r)
    ql[:, 0] = q[0].float()
    pos, row, pt = _i32([T - 1]), _i32([0]), _i32(range(n_pages)).view(1, -1)
    pool, ql = pool.view(n_pages, -1).to("cuda", BF16), ql.view(-1, R + r).to("cuda", BF16)
    for split in (1, 3):
        out, ws = torch.zeros(L.rows, R, dtype=BF16, device="cuda"), torch.empty(heads * split * (R + 2), device="cuda")
        K.latent_attn_decode(ql, out, pool, pt, pos, row, L, Rp=R, rw=r, page_size=16, scale=1.0, n_split=split, ws=ws)
        assert _err(out.view(heads, L.npad, R)[:, 0], want) < 2e-2
    check_ok()


@pytest.mark.parametrize("case", LATENT)
def test_latent_portions_over_expanded_keys(case):
    """Keys and values as rows of a matrix, gate pre-activations of every output element."""
    from tah_b200.engine.hybrid import NO_WINDOW
    from tah_b200.ops import cuda as K
    T, nh, dim, r, vdim, _ = case
    d, dk, dv = dim + r, _pad(dim + r, 8), _pad(vdim, 8)
    g = torch.Generator().manual_seed(T)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v, gate, sink = rnd(T, nh, d), rnd(T, nh, d), rnd(T, nh, vdim), rnd(T, nh, vdim), 2 * rnd(nh)
    for j in (0, 16, 63, 64, 127, 128):
        k[j] = 2.0 * q[min(T - 1, j + 9)]
    q, k, v, gate = (t.to(BF16).double() for t in (q, k, v, gate))
    scale = d ** -0.5
    want = O.attention_core(q, k, v, scale, sink.double()) * torch.sigmoid(gate)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).flatten(1)
    rows = (T + 15) // 16 * 16
    kv = torch.zeros(rows + 32, _pad(nh * (dk + dv), 64), dtype=BF16, device="cuda")     # two pages of another request in front
    kv[:32] = 5.0
    kv[32:32 + T, :nh * (dk + dv)] = torch.cat([pad(k, dk), pad(v, dv)], 1).to("cuda", BF16)
    table = torch.stack([torch.zeros(rows // 16), torch.arange(2, 2 + rows // 16)]).to("cuda", torch.int32).contiguous()
    qm = torch.zeros(T, _pad(nh * dk, 64), dtype=BF16, device="cuda")
    qm[:, :nh * dk] = pad(q, dk).to("cuda", BF16)
    gm = torch.zeros(T, nh * dv + 64, dtype=BF16, device="cuda")
    gm[:, 64:] = pad(gate, dv).to("cuda", BF16)
    log2 = sink.cuda() * 1.4426950408889634
    for a, b in ((0, T), (37, T), (T - 2, T), (100, 129)):
        n, t0 = b - a, list(range(0, b - a, 128))
        out = torch.zeros(n, nh * dv, dtype=BF16, device="cuda")
        meta = [_i32(range(a, b)), _i32([1] * n), _i32(t0), _i32(min(128, n - x) for x in t0)]
        K.window_attn_tiles(qm[a:b], out, kv, table, *meta, 2 + rows // 16, kv_ld=kv.shape[1], nq=nh, nkv=nh, dk=dk, dv=dv, page_size=16,
                            scale=scale, window=NO_WINDOW, keep_first=0, sink=log2, wide_gate=gm[a:b, 64:])
        got = out.double().cpu().view(n, nh, dv)[..., :vdim]
        err = (got - want[a:b]).abs().amax((1, 2)) / want[a:b].abs().amax((1, 2)).clamp(min=0.3 * float(want.abs().max()))
        assert float(err.max()) < 2e-2
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Q,R,r", [(56, 72, 12), (768, 512, 64), (21, 19, 10), (8, 8, 2)])
def test_latent_rows_and_queries(dtype, Q, R, r):
    """Norms and rotation on the way to the cache, queries into head lists and in place, pages gathered, gated outputs."""
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(Q)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-5 if dtype == F32 else 1e-2
    M, nh, dim = 23, 3, 20
    Qp, Rp, rw, dk = _pad(Q, 64), _pad(R, 64), _pad(r, 64), _pad(dim + r, 8)
    dq, c, kr, wq, wc = rnd(M, Q).to(dtype), rnd(M, R).to(dtype), rnd(M, r).to(dtype), 1 + 0.2 * rnd(Q), 1 + 0.2 * rnd(R)
    rot, pos = dict(dims=r, base=300.0), torch.randint(0, 3000, (M,), generator=g).to(torch.int32)
    rope = _rope(rot, pos.cuda())
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    proj = torch.cat([pad(dq, Qp), pad(c, Rp), pad(kr, rw), torch.full((M, 64), 3.0, dtype=dtype)], 1).cuda()
    cq = torch.empty(M, Qp, dtype=dtype, device="cuda")
    pool = torch.full((4, 16 * (Rp + rw)), 2.0, dtype=dtype, device="cuda")
    slot = torch.randperm(64, generator=g)[:M].to(torch.int32)
    slot[5] = -1
    wqp, wcp, slot_d = pad(wq, Qp).cuda(), pad(wc, Rp).cuda(), slot.cuda()
    K.latent_post(proj, wqp, wcp, rope, cq, pool, slot_d, q_rank=Q, q_col=0, kv_rank=R, Rp=Rp, c_col=Qp, rot=r, rw=rw, r_col=Qp + Rp, eps=1e-3)
    assert _err(cq[:, :Q], O.rms_norm(dq.double(), wq.double(), 1e-3)) < tol and float(cq[:, Q:].float().abs().sum()) == 0
    want_c, want_r = O.rms_norm(c.double(), wc.double(), 1e-3), O.rotate(kr.double().view(M, 1, r), pos.tolist(), rot, True)[:, 0]
    rows = pool.view(64, Rp + rw).cpu().double()
    ok = [t for t in range(M) if slot[t] >= 0]
    at = rows[slot[ok].long()]
    assert _err(at[:, :R], want_c[ok]) < tol and _err(at[:, Rp:Rp + r], want_r[ok]) < tol
    assert float(at[:, R:Rp].abs().sum()) == 0 and float(at[:, Rp + r:].abs().sum()) == 0
    untouched = [s for s in range(64) if s not in slot.tolist()]
    assert bool((rows[untouched] == 2.0).all())
    src = _i32([3, 0, 0, 2])
    got = K.latent_gather(pool, src, 16, Rp + rw, torch.full((64, Rp + rw + 64), 8.0, dtype=dtype, device="cuda"))
    want = torch.zeros(64, got.shape[1], dtype=torch.float64)
    want[:, :Rp + rw] = rows.view(4, 16, -1)[[3, 0, 0, 2]].reshape(64, -1)
    assert torch.equal(got.cpu().double(), want)
    q = rnd(M, nh, dim + r).to(dtype)
    want = q.double().clone()
    want[..., dim:] = O.rotate(q.double()[..., dim:], pos.tolist(), rot, True)
    qm = torch.full((M, nh * dk + 64), 4.0, dtype=dtype)
    qm[:, :nh * dk] = pad(q, dk).flatten(1)
    for n_list in (0, 9, M):
        m = qm.cuda()
        L = K.HeadLists(n_list, nh, dtype, "cuda") if n_list else None
        lst = torch.full((L.rows, _pad(dk, 64)), 6.0, dtype=dtype, device="cuda") if n_list else None
        K.latent_query(m, rope, L, lst, heads=nh, dk=dk, dim=dim, rot=r)
        if n_list < M:
            assert _err(m[n_list:, :nh * dk].view(M - n_list, nh, dk)[..., :dim + r], want[n_list:]) < tol
        assert torch.equal(m[:n_list].cpu(), qm[:n_list])
        if n_list:
            l = lst.view(nh, L.npad, -1)[:, :n_list].transpose(0, 1)
            assert _err(l[..., :dim + r], want[:n_list]) < tol and float(l[..., dim + r:].float().abs().sum()) == 0
            assert int(L.n_blocks) * L.bn == L.rows and torch.equal(L.blk_expert.cpu().long(), torch.arange(L.rows // L.bn) * L.bn // L.npad)
    L, dv = K.HeadLists(M, nh, dtype, "cuda"), 24
    v, gate, out = rnd(L.rows, 64).to(dtype), rnd(M, nh * dv).to(dtype), torch.zeros(M, nh * dv, dtype=dtype, device="cuda")
    K.latent_gate(v.cuda(), L, gate.cuda(), out, dv)
    want = v.double().view(nh, L.npad, 64)[:, :M, :dv].transpose(0, 1).reshape(M, -1) * torch.sigmoid(gate.double())
    assert _err(out, want) < tol
    check_ok()


@pytest.mark.parametrize("M,E,top", [(1, 5, 5), (7, 37, 3), (300, 9, 1), (4200, 64, 8), (33, 1000, 4)])
def test_softmax_router(M, E, top):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(M + E)
    L = K.ExpertLists(M, E, top, BF16, "cuda", bn=16)
    z = 2 * torch.randn(M, E + 1, generator=g)
    K.moe_route(z.cuda(), L, softmax=True)
    s = torch.softmax(z[:, :E].double(), -1)
    got = L.expert.cpu().long()
    assert torch.equal(got.sort(-1).values, z[:, :E].topk(top, -1).indices.sort(-1).values)
    assert torch.allclose(L.weight.cpu().double(), s.gather(1, got), rtol=1e-5)
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M", [3, 700])
def test_swiglu_experts(dtype, M):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(M)
    rnd = lambda *s: torch.randn(*s, generator=g)
    E, top, W, F = 6, 2, 128, 192
    L = K.ExpertLists(M, E, top, dtype, "cuda")
    h, w = (3 * rnd(M, W)).to(dtype), (rnd(E, 2 * F, W) / math.sqrt(W)).to(dtype)
    K.moe_route(rnd(M, E).cuda(), L, softmax=True)
    e = lambda c: torch.full((L.rows, c), float("nan"), dtype=dtype, device="cuda")
    x = K.moe_gather(h.cuda(), L, e(W))
    act = K.moe_glu_linear(x, w.cuda(), math.inf, L, e(F), slope=1.0, offset=0.0, weighted=False)
    slot, which = L.slot.cpu().long(), L.expert.cpu().long()
    gu = torch.einsum("tjfk,tk->tjf", w.double()[which], h.double())
    want = gu[..., 0::2] * torch.sigmoid(gu[..., 0::2]) * gu[..., 1::2]
    assert _err(act.cpu()[slot], want) < (2e-5 if dtype == F32 else 1e-2)
    check_ok()


# ------------------------------------------------------------------------------------
# the model through the engine's step function
# ------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(H.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompt_portions_and_single_tokens(tmp_path, name, dtype):
    cfg, sd, d = H.make(tmp_path, name)
    T = 210 if name in ("tiles", "steep") else 150
    toks = H.tokens(cfg, T)
    layers = []
    want = O.forward(cfg, sd, toks, layers_out=layers)
    e = engine(d, dtype)
    seen = []
    e.layer_hook = lambda i, x: seen.append(x.clone())
    whole = run_portions(e, toks, [T])
    e.layer_hook = None
    for i, (x, y) in enumerate(zip(seen, layers)):
        err = float((x.cpu().double() - y).abs().max() / y.abs().max())
        assert err < (3e-5 if dtype == F32 else 6e-2), (i, err)
    assert H.close(whole, want, dtype)
    for portions in ([1] * T, [2] * (T // 2), [3, 1, 64, 1, 2, T - 71], [17] * (T // 17) + [T % 17], [T - 40] + [1] * 40, [16, 16, 48, T - 80],
                     [128, T - 128]):
        got = run_portions(e, toks, [p for p in portions if p])
        assert H.close(got, want, dtype), portions[:4]
    assert e.kv.pages_in_use(0) == 0
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("place", [0, 1, 15, 16, 63, 64, 127, 130])
@pytest.mark.parametrize("layers", [(0, 1), (1,)])
def test_a_far_key_is_found(tmp_path, dtype, place, layers):
    """One key that every later query finds, by attention or by latent attention only: in a prompt, in portions and in
    decoding, wherever the key lies."""
    cfg = H.CONFIGS["far"]()
    special, T = 7, 300
    sd = H.stand_out(cfg, O.random_model(cfg, 3), special, layers=layers)
    d = os.path.join(str(tmp_path), "ckpt")
    H.write_checkpoint(d, cfg, sd)
    plain = [t if t != special else special + 1 for t in H.tokens(cfg, T, 3)]
    toks = list(plain)
    toks[place] = special
    want = O.forward(cfg, sd, toks)
    # it is this key that the last tokens answer to
    assert float(H.row_errors(O.forward(cfg, sd, plain)[-40:], want[-40:]).min()) > 0.2
    e = engine(d, dtype)
    for portions in ([T], [100, 100, 60] + [1] * 40, [place + 2, 2, T - place - 4]):
        assert H.close(run_portions(e, toks, portions), want, dtype), portions[:3]
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_and_reused_pages_and_slots(tmp_path, dtype, monkeypatch):
    """Requests of unequal lengths in shared steps, in a pool that only holds a few of them, rows handed on, latents of a few
    pages expanded at a time; every request's logits equal those of the request alone."""
    from tah_b200.engine import StepEntry, hybrid
    monkeypatch.setattr(hybrid, "LATENT_PAGES", 6)
    cfg, sd, d = H.make(tmp_path, "mixed", seed=1)
    g = torch.Generator().manual_seed(11)
    reqs = [H.tokens(cfg, n, seed=20 + i) for i, n in enumerate([90, 1, 37, 64, 130, 2, 17, 75, 50])]
    want = [O.forward(cfg, sd, t) for t in reqs]
    e = engine(d, dtype, rows=3, pool=288)
    live, at, queue, got = {}, {}, list(range(len(reqs))), [[] for _ in reqs]
    rows_used = set()
    pages = lambda r: (len(reqs[r]) + 15) // 16 * 16
    while queue or live:
        while queue and len(live) < 3 and sum(map(pages, live)) + pages(queue[0]) <= 288:
            r = queue.pop(0)
            live[r], at[r] = e.admit(), 0
            rows_used.add(live[r])
        entries, who = [], []
        for r in list(live):
            if len(live) > 1 and torch.rand((), generator=g) < 0.25:
                continue                                           # left out of this step
            n = min(int(torch.tensor([1, 1, 2, 5, 16, 31, 60])[torch.randint(0, 7, (), generator=g)]), len(reqs[r]) - at[r])
            entries.append(StepEntry(live[r], reqs[r][at[r]:at[r] + n], range(n)))
            who.append((r, n))
        if not entries:
            continue
        lg = e.step(entries).float().cpu()
        first = 0
        for r, n in who:
            got[r].append(lg[first:first + n])
            first += n
            at[r] += n
            if at[r] == len(reqs[r]):
                e.release(live.pop(r))
    for r, w in enumerate(want):
        assert H.close(torch.cat(got[r]), w, dtype), r
    assert e.kv.pages_in_use(0) == 0 and len(rows_used) == 3
    check_ok()


def test_logits_do_not_depend_on_pages_and_company(tmp_path):
    from tah_b200.engine import StepEntry
    cfg, sd, d = H.make(tmp_path, "tiles", seed=2)
    a, b = H.tokens(cfg, 150, 1), H.tokens(cfg, 61, 2)
    e = engine(d, BF16)
    row = e.admit()
    alone = e.step([StepEntry(row, a[:100], [99])]).clone(), e.step([StepEntry(row, a[100:], range(50))]).clone()
    other, again = e.admit(), e.admit()
    e.step([StepEntry(other, b[:30], ())])
    first = e.step([StepEntry(again, a[:100], [99]), StepEntry(other, b[30:], ())])
    assert float(H.row_errors(first.float(), alone[0].float().cpu()).max()) < 2e-2
    second = e.step([StepEntry(again, a[100:], range(50))])
    assert float(H.row_errors(second.float(), alone[1].float().cpu()).max()) < 2e-2
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_large_steps(tmp_path, dtype, monkeypatch):
    """More than a thousand tokens in a step (wide token tiles of the dense and the grouped products), unequal requests,
    recurrent chunks and latent expansions in several launches."""
    from tah_b200.engine import StepEntry, hybrid
    cfg, sd, d = H.make(tmp_path, "tiles", seed=9)
    reqs = [H.tokens(cfg, n, 60 + n) for n in (1150, 200, 260, 131)]
    want = [O.forward(cfg, sd, t) for t in reqs]
    for chunks, pages in ((hybrid.MEMORY_CHUNKS, hybrid.LATENT_PAGES), (3, 30)):
        monkeypatch.setattr(hybrid, "MEMORY_CHUNKS", chunks)
        monkeypatch.setattr(hybrid, "LATENT_PAGES", pages)
        e = engine(d, dtype, rows=4, pool=2048)
        rows = [e.admit() for _ in reqs]
        a = e.step([StepEntry(r, t[:len(t) - 70], range(len(t) - 70)) for r, t in zip(rows, reqs)]).float().cpu()
        b = e.step([StepEntry(r, t[len(t) - 70:], range(70)) for r, t in zip(rows, reqs)]).float().cpu()
        at = 0
        for i, w in enumerate(want):
            n = len(reqs[i]) - 70
            assert H.close(torch.cat([a[at:at + n], b[70 * i:70 * i + 70]]), w, dtype), i
            at += n
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_pool_exhaustion_is_an_error_and_leaves_the_cache_usable(tmp_path, dtype):
    from tah_b200.engine import StepEntry
    from tah_b200.ops import cuda as K
    cfg, sd, d = H.make(tmp_path, "mixed")
    toks = H.tokens(cfg, 200)
    e = engine(d, dtype, rows=2, pool=96)
    row = e.admit()
    e.step([StepEntry(row, toks[:50], ())])
    with pytest.raises(K.KernelTimeout):
        e.step([StepEntry(row, toks[50:200], ())])
        K.check_status()
    e.release(row)
    assert e.kv.pages_in_use(0) == 0
    assert H.close(run_portions(e, toks[:90], [60, 30]), O.forward(cfg, sd, toks[:90]), dtype)


def test_plain_kernels_in_bf16(tmp_path):
    """Other page sizes take the plain kernels, with the same routed experts."""
    cfg, sd, d = H.make(tmp_path, "mixed")
    toks = H.tokens(cfg, 100)
    e = engine(d, BF16, page_size=8)
    assert e.plain and H.close(run_portions(e, toks, [60, 1, 1, 38]), O.forward(cfg, sd, toks), BF16)
    check_ok()


def test_sizes_beyond_the_tensor_core_kernels(tmp_path):
    """Latents and heads that fit neither the decode kernel nor the portion kernel, recurrent heads beyond the chunk kernels."""
    cfg = H.config([(H.latent(heads=2, dim=250, rot_dim=16, vdim=24, kv_rank=1300, scale=0.06), H.dense()), (H.gla(heads=1, dim=136, vdim=24), None),
                    (H.latent(heads=2, dim=40, rot_dim=8, vdim=264, kv_rank=64), None)])
    cfg, sd, d = H.make(tmp_path, cfg)
    toks = H.tokens(cfg, 140)
    e = engine(d, BF16)
    assert [getattr(b.mixer, "w_exp", 0) is None for b in e.w.layers] == [True, False, True] and not e.w.layers[0].mixer.on_tensor_cores
    assert H.close(run_portions(e, toks, [90, 1, 1, 48]), O.forward(cfg, sd, toks), BF16)
    check_ok()


# ------------------------------------------------------------------------------------
# generation through generate() and serve()
# ------------------------------------------------------------------------------------
def _tokens_follow(cfg, sd, prompt, out, slack):
    """Every generated token is the arg-max of the plain model on the text so far, up to ``slack`` of its logit range."""
    lg = O.forward(cfg, sd, list(prompt) + list(out))[len(prompt) - 1:-1]
    gap = lg.amax(-1) - lg.gather(1, torch.tensor(out).view(-1, 1)).flatten()
    return float((gap / lg.std(-1)).max()) <= slack


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation(tmp_path, dtype, graph):
    from tah_b200.models import load_model, make_engine
    cfg, sd, d = H.make(tmp_path, "mixed", seed=3)
    e = make_engine(load_model(d, dtype, "cuda"), max_rows=4, use_cuda_graph=graph, prefill_tokens=48)
    lens = [40, 7, 23]
    ids, mask = torch.zeros(3, 40, dtype=torch.long), torch.zeros(3, 40, dtype=torch.long)
    prompts = [H.tokens(cfg, n, 30 + i) for i, n in enumerate(lens)]
    for i, p in enumerate(prompts):
        ids[i, 40 - len(p):], mask[i, 40 - len(p):] = torch.tensor(p), 1
    for _ in range(2):                                  # the second call replays the captured tick
        res = e.generate(ids, mask, max_new_tokens=60)
        for p, out in zip(prompts, res.tokens):
            assert len(out) == 60 and _tokens_follow(cfg, sd, p, out, 1e-4 if dtype == F32 else 0.15)


def test_long_decoding(tmp_path):
    from tah_b200.models import load_model, make_engine
    cfg, sd, d = H.make(tmp_path, "tiles", seed=4)
    for dtype, slack in ((F32, 1e-4), (BF16, 0.15)):
        e = make_engine(load_model(d, dtype, "cuda"), max_rows=1)
        p = H.tokens(cfg, 5, 9)
        out = e.generate(torch.tensor([p]), None, max_new_tokens=340).tokens[0]
        assert len(out) == 340 and _tokens_follow(cfg, sd, p, out, slack)


def test_serve_mixes_prompts_with_decoding(tmp_path):
    """More requests than rows, prompts longer than a portion: each request's greedy tokens are those of the plain model."""
    from tah_b200.models import load_model, make_engine
    cfg, sd, d = H.make(tmp_path, "mixed", seed=5)
    prompts = [H.tokens(cfg, n, 40 + i) for i, n in enumerate([30, 3, 71, 12, 1, 44, 25])]
    for dtype, slack in ((BF16, 0.15), (F32, 1e-4)):
        e = make_engine(load_model(d, dtype, "cuda"), max_rows=3)
        for _ in range(2):
            res, stats = e.serve([torch.tensor(p) for p in prompts], max_new_tokens=20, portion=16, check_every=4)
            assert stats["admitted"] == 7 and stats["mixed_steps"] > 7 and stats["tokens"] == 140
            assert all(_tokens_follow(cfg, sd, p, out, slack) for p, out in zip(prompts, res))
            assert e.kv.pages_in_use(0) == 0
    eos = res[2][5]                                     # an EOS ends a request early, and its place goes to the next one
    res2, _ = e.serve([torch.tensor(p) for p in prompts], max_new_tokens=20, portion=16, check_every=4, eos_token_id=eos)
    for a, b in zip(res, res2):
        assert b == (a[:a.index(eos)] if eos in a else a)


def test_sampling(tmp_path):
    from tah_b200.engine import get_engine
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, "odd", seed=6)
    e = get_engine(load_model(d, BF16, "cuda"), max_rows=4)
    ids = torch.tensor([H.tokens(cfg, 12, 1), H.tokens(cfg, 12, 2)])
    for kw in (dict(top_k=5), dict(top_k=0, top_p=0.9)):
        a, b, c = (e.generate(ids, None, max_new_tokens=12, do_sample=True, temperature=8.0, seed=s, **kw).tokens for s in (7, 7, 8))
        assert a == b and a != c and all(0 <= t < cfg["vocab"] for r in a for t in r)
    g = e.generate(ids, None, max_new_tokens=12).tokens
    assert e.generate(ids, None, max_new_tokens=12, do_sample=True, top_k=1, seed=3).tokens == g


def test_trace_replay_program(tmp_path):
    cfg, sd, d = H.make(tmp_path, "odd", seed=7)
    a, b = H.tokens(cfg, 40, 1), H.tokens(cfg, 9, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:25], want=[24])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[8, 0]), dict(id="a", tokens=a[25:26], want=[0])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=b[:2], want=[1]), dict(id="a", tokens=a[26:], want=[13])], end=["a", "c"])]
    out = os.path.join(str(tmp_path), "out")
    la, lb = O.forward(cfg, sd, a), O.forward(cfg, sd, b)
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out, "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(3)]
        for step, want in ((0, la[24:25]), (1, torch.stack([lb[8], lb[0], la[25]])), (2, torch.stack([lb[1], la[39]]))):
            raw = torch.frombuffer(bytearray(open(os.path.join(out, f"{step}.f32"), "rb").read()), dtype=torch.float32)
            assert H.close(raw.view(-1, cfg["vocab"]), want, getattr(torch, dtype))
            os.unlink(os.path.join(out, f"{step}.f32"))


def test_playground_command_line(tmp_path):
    cfg, sd, d = H.make(tmp_path, "mixed", seed=8)
    prompts = [H.tokens(cfg, 9, 1), H.tokens(cfg, 4, 2)]
    cmd = [sys.executable, os.path.join(ROOT, "script", "playground", "inference_example.py"), "--model", d, "--dtype", "float32",
           "--temperature", "0", "--max_new_tokens", "8"]
    for p in prompts:
        cmd += ["--prompt_ids", ",".join(map(str, p))]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    rows = [[int(t) for t in l.split(",")] for l in r.stdout.split()]
    assert len(rows) == 2 and all(_tokens_follow(cfg, sd, p, o, 1e-4) for p, o in zip(prompts, rows))
