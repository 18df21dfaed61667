"""Pidenex on the GPU: every mechanism against a plain statement of it, and the engine's steps, ticks and scheduler."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from tests import pidenex_helpers as H
from tests.oracle import pidenex_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16
LOG2E = 1.4426950408889634


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


def _padt(t, n):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1]))


def _err(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def _row_err(got, want):
    """Error of every token relative to its own size (at least a third of the largest)."""
    return (got - want).abs().amax((1, 2)) / want.abs().amax((1, 2)).clamp(min=0.3 * float(want.abs().max()))


# ------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("centered", [True, False])
def test_norm_seams(dtype, centered):
    """Layer (and RMS) norms in front of and behind a sublayer, with and without what begins a pass."""
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g)
    norm = O.layer_norm if centered else O.rms_norm
    tol = 1e-5 if dtype == F32 else 1e-2
    for width, ld, M in ((512, 512, 5), (77, 128, 9), (2048, 2048, 3), (130, 192, 40), (5003, 5056, 2), (1, 64, 3) if not centered else (2, 64, 3)):
        z = lambda t: _padt(t, ld)
        E, w, wo, wn, add = (rnd(50, width) + 3.0).to(dtype), rnd(width), rnd(width), rnd(width), rnd(width)
        ids = torch.randint(0, 50, (M,), generator=g).to(torch.int32)
        x, h = torch.full((M, ld), 9.0, device="cuda"), torch.empty(M, ld, dtype=dtype, device="cuda")
        emb = 0.3 * E.double()[ids.long()]
        for a in (None, add):
            K.embed_norm(z(E).cuda(), ids.cuda(), 0.3, z(w).cuda(), width, 1e-4, x, h, add=None if a is None else z(a).cuda(), centered=centered)
            want = emb if a is None else emb + a.double()
            assert _err(x[:, :width], want) < 1e-6 and _err(h[:, :width], norm(want, w.double(), 1e-4)) < tol
        for more in (False, True):
            y = (rnd(M, width) - 2.0).to(dtype)
            before = torch.empty_like(x) if more else None
            x0 = x.double().cpu()[:, :width]
            kw = dict(add=z(add).cuda(), embedding=(z(E).cuda(), ids.cuda(), 0.3), before=before) if more else {}
            K.residual_norm(z(y).cuda(), x, z(wo).cuda(), z(wn).cuda(), width, 1e-4, h, centered=centered, **kw)
            want = x0 + norm(y.double(), wo.double(), 1e-4)
            if more:
                assert _err(before[:, :width], want) < 1e-5
                want = want + emb + add.double()
            assert _err(x[:, :width], want) < 1e-5 and _err(h[:, :width], norm(want, wn.double(), 1e-4)) < tol
        assert float(h[:, width:].float().abs().sum()) == 0 and float(x[:, width:].abs().sum()) == 0
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,F,Kd", [(1, 64, 128), (5, 320, 192), (40, 1000 // 8 * 8, 64), (200, 192, 256), (1100, 512, 128), (1025, 320, 64), (3000, 256, 192)])
def test_xielu_product(dtype, M, F, Kd):
    """The activation in the epilogue of every form of the product, both signs and large arguments."""
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(M)
    x, w = torch.randn(M, Kd, generator=g).to(dtype), (3 * torch.randn(F, Kd, generator=g) / math.sqrt(Kd)).to(dtype)
    w[0] *= 8
    pq = torch.tensor([0.7, -0.4], dtype=torch.float64)
    up, low = float(O.softplus(pq)[0]), 0.5 + float(O.softplus(pq)[1])
    out = torch.full((M, F + 64), 5.0, dtype=dtype, device="cuda")
    K.xielu_linear(x.cuda(), w.cuda(), up, low, out=out[:, :F])
    z = x.double() @ w.double().T
    if dtype == BF16:
        z = z.float().to(BF16).double()
    want = O.xielu(z, pq)
    err = (out[:, :F].double().cpu() - want).abs() / (want.abs() + 0.05)
    # (a sum that rounds to the neighbouring 16-bit number moves the result by some more of them)
    assert float(err.max()) < (1e-4 if dtype == F32 else 4e-2) and float((err > 1e-2).double().mean()) < (1e-9 if dtype == F32 else 2e-3)
    assert bool((out[:, F:] == 5.0).all())
    check_ok()


# T, heads, key heads, dim, window, block
TIED = [(150, 4, 2, 40, 19, 5), (300, 16, 8, 128, 64, 16), (200, 3, 3, 18, 3, 1), (260, 8, 1, 64, 16, 4), (190, 5, 1, 7, 11, 21), (210, 6, 2, 200, 50, 12),
        (170, 1, 1, 8, 1, 2), (140, 2, 2, 136, 130, 3), (330, 12, 4, 96, 100, 40)]


def _tied_case(case, dtype, peaked, pooled, factors, seed=0):
    """Random queries and keys in a shuffled paged cache; block means written by the kernel that appends keys."""
    from tah_b200.engine.kv_cache import LayerKV
    from tah_b200.ops import cuda as K
    T, nh, G, dim, size, block = case
    dk = _pad(dim, 8)
    g = torch.Generator().manual_seed(seed + T)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k = rnd(T, nh, dim), rnd(T, G, dim)
    if peaked:
        u = torch.nn.functional.normalize(rnd(dim), dim=0) * math.sqrt(dim)
        q, k = 0.2 * q + 1.5 * u, 0.3 * k
        for j in {0, 15, 16, 63, 64, 77, 127, 128, T - 1}:
            if j < T:
                k[j] = (3.0 if j % 2 else -3.0) * u + 0.5 * rnd(G, dim)
    q, k = q.to(dtype), k.to(dtype)
    n_pages = (T + 15) // 16
    perm = torch.randperm(n_pages + 3, generator=g)[:n_pages].to(torch.int32)
    pt = perm.view(1, -1).contiguous().cuda()
    slot = _i32(int(perm[t // 16]) * 16 + t % 16 for t in range(T))
    pool = torch.zeros(n_pages + 3, G * 16 * dk, dtype=dtype, device="cuda")
    S = LayerKV(block=block).pool_rows(16)
    means = torch.zeros(n_pages + 3, G * S * dk, dtype=dtype, device="cuda")
    km = torch.full((T, G * dk + 64), 3.0, dtype=dtype)
    km[:, :G * dk] = _padt(k, dk).flatten(1)
    pos, row = _i32(range(T)), _i32([0] * T)
    km = km.cuda()
    at = 0
    for c in (37, 2, 1, T - 40):                           # in portions: the keys of a block come from several steps
        s = slice(at, at + c)
        K.tied_keys(km[s], pool, slot[s], pos[s], row[s], pt, G, dk, 16, means, block, S)
        at += c
    qm = torch.zeros(T, nh * dk + 64, dtype=dtype)
    qm[:, :nh * dk] = _padt(q, dk).flatten(1)
    fac = torch.rand(n_pages + 3, 16, generator=g) + 0.3
    per_key = torch.stack([fac[int(perm[t // 16]), t % 16] for t in range(T)])
    kw = dict(nq=nh, nkv=G, dk=dk, dv=dk, page_size=16, window=size, keep_first=0, tied=True)
    if pooled:
        kw.update(pooled=means, block=block, pool_rows=S)
    if factors:
        kw.update(factor=fac.cuda())
    return dict(q=q.double(), k=k.double(), qm=qm.cuda(), pool=pool, pt=pt, perm=perm, means=means, S=S, per_key=per_key.double(), kw=kw, pos=pos, row=row,
                n_pages=n_pages, slot=slot, g=g)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", TIED)
def test_block_means(dtype, case):
    """Means of complete blocks in the places the rule gives, whichever steps brought their keys; nothing else is written."""
    T, nh, G, dim, size, block = case
    c, dk = _tied_case(case, dtype, False, True, False), _pad(dim, 8)
    want = O.block_means(c["k"], block)
    rows = c["means"].cpu().double().view(-1, G, c["S"], dk)
    touched = torch.zeros(rows.shape[0], c["S"], dtype=torch.bool)
    for b in range(T // block):
        p, o = int(c["perm"][b // c["S"]]), b % c["S"]
        touched[p, o] = True
        assert float((rows[p, :, o, :dim] - want[b]).abs().max()) < (1e-6 if dtype == F32 else 1.5e-2) * float(want.abs().max())
        assert float(rows[p, :, o, dim:].abs().sum()) == 0
    assert float(rows.permute(0, 2, 1, 3)[~touched].abs().sum()) == 0
    cache = c["pool"].cpu().double().view(-1, G, 16, dk)
    for t in range(T):
        assert torch.equal(cache[int(c["perm"][t // 16]), :, t % 16, :dim], c["k"][t])
    check_ok()


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode", "tiles"])
@pytest.mark.parametrize("case", TIED)
@pytest.mark.parametrize("peaked", [False, True])
@pytest.mark.parametrize("form", ["blocks", "biased", "bare"])
def test_tied_attention(kernel, case, peaked, form):
    """Values that are the keys: with pooled blocks, with key factors and slopes and a gate of every element, with neither."""
    from tah_b200.ops import cuda as K
    T, nh, G, dim, size, block = case
    dtype, dk = F32 if kernel == "plain32" else BF16, _pad(dim, 8)
    c = _tied_case(case, dtype, peaked, form == "blocks", form == "biased")
    kw, scale = dict(c["kw"], scale=1.0 / math.sqrt(dim), out_scale=0.7), 1.0 / math.sqrt(dim)
    k, q = c["k"], c["q"]
    want = 0.7 * O.attention_core(q, k * c["per_key"].view(-1, 1, 1) if form == "biased" else k, k, scale, size, block if form == "blocks" else None,
                                  O.slopes(nh) if form == "biased" else None)
    gate = None
    if form == "biased":
        gt = torch.randn(T, nh, dim, generator=c["g"]).to(dtype)
        want = want * torch.sigmoid(gt.double())
        gate = torch.zeros(T, nh * dk + 64, dtype=dtype)
        gate[:, 64:] = _padt(gt, dk).flatten(1)
        gate = gate.cuda()
        kw["slope"] = torch.tensor(O.slopes(nh)).float().cuda() * (1.0 if kernel.startswith("plain") else LOG2E)
    tol = 3e-5 if dtype == F32 else 2e-2
    wide = lambda s: {} if gate is None else dict(wide_gate=gate[s, 64:])
    sl = slice(0, nh * dk)

    def compare(out, rows):
        got = out.double().cpu().view(len(rows), nh, dk)[..., :dim]
        assert float(_row_err(got, want[rows]).max()) < tol, _row_err(got, want[rows])

    if kernel.startswith("plain"):
        out = torch.full((T, nh * dk), 7.0, dtype=dtype, device="cuda")
        K.window_attn_plain(c["qm"][:, sl], out, c["pool"], c["pt"], c["pos"], c["row"], **wide(slice(None)), **kw)
        compare(out, list(range(T)))
    elif kernel == "decode":
        rows = sorted({p for p in (0, 1, 2, 15, 16, 17, 63, 64, 77, 78, size - 1, size, size + 1, size + block - 1, size + block, size + 2 * block, 127, 128,
                                   129, T - 2, T - 1) if 0 <= p < T})
        at, zero = _i32(rows), _i32([0] * len(rows))
        for split in (1, 3):
            out, ws = torch.full((len(rows), nh * dk), 7.0, dtype=dtype, device="cuda"), torch.empty(len(rows) * nh * split * (dk + 2), device="cuda")
            g = {} if gate is None else dict(wide_gate=gate[rows].contiguous()[:, 64:])
            K.window_attn_decode(c["qm"][rows].contiguous()[:, sl], out, c["pool"], c["pt"], at, zero, n_split=split, ws=ws, **g, **kw)
            compare(out, rows)
    else:
        for a, b in ((0, T), (37, T), (T - 2, T), (100, 129)):
            n, t0 = b - a, list(range(0, b - a, 128))
            more = {}
            if form == "blocks":
                seen = max(0, b - size) // block
                src = [int(c["perm"][j // c["S"]]) * c["S"] + j % c["S"] if j < seen else -1 for j in range(_pad(seen, 16))]
                src = [int(c["perm"][0]) * c["S"]] * 16 + src                    # a page of another row in front
                m = K.pool_gather(c["means"], _i32(src), G, dk, c["S"], torch.full((len(src), G * dk), 9.0, dtype=dtype, device="cuda"))
                more = dict(pooled=m, pool_base=_i32([1] * len(t0)))
            out = torch.full((n, nh * dk), 7.0, dtype=dtype, device="cuda")
            K.window_attn_tiles(c["qm"][a:b, sl], out, c["pool"], c["pt"], _i32(range(a, b)), _i32([0] * n), _i32(t0), _i32(min(128, n - x) for x in t0),
                                c["pool"].shape[0], **wide(slice(a, b)), **dict(kw, **more))
            compare(out, list(range(a, b)))
    check_ok()


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode", "tiles"])
def test_slopes_and_element_gates_beside_separate_values(kernel):
    """The same distance bias and gate in a layer with keys and values of their own."""
    from tah_b200.ops import cuda as K
    T, nh, G, dim, vdim, size = 200, 6, 2, 40, 24, 70
    dtype, dk, dv = F32 if kernel == "plain32" else BF16, 40, 24
    g = torch.Generator().manual_seed(1)
    q, k, v, gt = (torch.randn(T, h, d, generator=g).to(dtype) for h, d in ((nh, dim), (G, dim), (G, vdim), (nh, vdim)))
    want = O.attention_core(q.double(), k.double(), v.double(), 0.3, size, None, O.slopes(nh)) * torch.sigmoid(gt.double())
    pages = (T + 15) // 16
    pad = lambda t: torch.nn.functional.pad(t, (0, 0, 0, 0, 0, pages * 16 - T)).view(pages, 16, G, -1).transpose(1, 2).reshape(pages, -1)
    pool = torch.cat([pad(k), pad(v)], 1).contiguous().cuda()
    pt, qm, gm = _i32(range(pages)).view(1, -1), q.flatten(1).contiguous().cuda(), gt.flatten(1).contiguous().cuda()
    unit = 1.0 if kernel.startswith("plain") else LOG2E
    kw = dict(nq=nh, nkv=G, dk=dk, dv=dv, page_size=16, scale=0.3, window=size, keep_first=0, slope=torch.tensor(O.slopes(nh)).float().cuda() * unit, wide_gate=gm)
    out = torch.zeros(T, nh * dv, dtype=dtype, device="cuda")
    a = (qm, out, pool, pt, _i32(range(T)), _i32([0] * T))
    if kernel.startswith("plain"):
        K.window_attn_plain(*a, **kw)
    elif kernel == "decode":
        K.window_attn_decode(*a, n_split=2, ws=torch.empty(T * nh * 2 * (dv + 2), device="cuda"), **kw)
    else:
        K.window_attn_tiles(*a, _i32([0, 128]), _i32([128, 72]), pages, **kw)
    assert float(_row_err(out.double().cpu().view(T, nh, dv), want).max()) < (3e-5 if dtype == F32 else 2e-2)
    check_ok()


def test_forms_that_no_kernel_has_are_refused():
    from tah_b200.ops import cuda as K
    z = lambda *s: torch.zeros(*s, dtype=BF16, device="cuda")
    q, out, pool, pt, one = z(1, 16), z(1, 16), z(1, 256), _i32([0]).view(1, 1), _i32([0])
    kw = dict(nq=1, nkv=1, dk=16, dv=16, page_size=16, scale=1.0, window=4, keep_first=0)
    f = torch.ones(1, 16, device="cuda")
    for bad in (dict(pooled=pool, block=4, pool_rows=4), dict(factor=f), dict(tied=True, softcap=3.0), dict(tied=True, pooled=pool, block=4, pool_rows=3),
                dict(tied=True, pooled=pool, block=4, pool_rows=2), dict(tied=True, pooled=pool, block=4, pool_rows=4, factor=f),
                dict(tied=True, slope=f, bias=f)):
        for fn in (K.window_attn_plain, K.window_attn_decode):
            with pytest.raises(RuntimeError):
                fn(q, out, pool, pt, one, one, **dict(kw, **bad))
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("nq,G,dim", [(4, 2, 40), (16, 8, 128), (3, 1, 18), (5, 5, 7), (6, 1, 200)])
def test_norms_over_all_heads(dtype, nq, G, dim):
    from tah_b200.ops import cuda as K
    M, dk = 21, _pad(dim, 8)
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, wq, wk = (2 * rnd(M, nq, dim)).to(dtype), (0.3 * rnd(M, G, dim)).to(dtype), 1 + 0.2 * rnd(nq, dim), 1 + 0.2 * rnd(G, dim)
    proj = torch.full((M, (nq + G) * dk + 24), 2.0, dtype=dtype)
    proj[:, :(nq + G) * dk] = _padt(torch.cat([q, k], 1), dk).flatten(1)
    proj = proj.cuda()
    slot = torch.randperm(64, generator=g)[:M].to(torch.int32)
    slot[3] = -1
    pool, fac = torch.full((4, G * 16 * dk), 8.0, dtype=dtype, device="cuda"), torch.full((4, 16), 8.0, device="cuda")
    out = torch.empty(M, nq * dk, dtype=dtype, device="cuda")
    folded = _padt(wq.view(G, nq // G, dim) * wk.view(G, 1, dim), dk).reshape(-1).contiguous().cuda()
    K.norm_all(proj[:, :nq * dk], proj[:, nq * dk:(nq + G) * dk], folded, out, pool, fac, slot.cuda(), nq=nq, nkv=G, dk=dk, dim=dim, page_size=16, eps=1e-3)
    # scores of normed queries and keys, from what the kernel left
    qn = O.rms_norm(q.double().flatten(1), wq.double().flatten(), 1e-3).view(M, nq, dim)
    kn = O.rms_norm(k.double().flatten(1), wk.double().flatten(), 1e-3).view(M, G, dim)
    ok = [t for t in range(M) if slot[t] >= 0]
    rows = pool.cpu().double().view(4, G, 16, dk).transpose(1, 2).reshape(64, G, dk)
    keys = rows[slot[ok].long()]
    assert torch.equal(keys[..., :dim], k.double()[ok]) and float(keys[..., dim:].abs().sum()) == 0
    f = fac.cpu().double().flatten()[slot[ok].long()]
    o = out.double().cpu().view(M, nq, dk)
    owner = torch.arange(nq) // (nq // G)
    got = torch.einsum("thd,shd->ths", o[..., :dim], keys[:, owner][..., :dim]) * f
    assert _err(got, torch.einsum("thd,shd->ths", qn, kn[ok][:, owner])) < (1e-5 if dtype == F32 else 1e-2)
    assert float(o[..., dim:].abs().sum()) == 0
    idle = [s for s in range(64) if s not in slot.tolist()]
    assert bool((rows[idle] == 8.0).all()) and bool((fac.cpu().flatten()[idle] == 8.0).all())
    check_ok()


# lengths of portions side by side, width
GRU = [([1], 72), ([150], 224), ([64, 5, 260, 2], 40), ([129, 63], 13), ([1500, 17], 320), ([700], 2)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("form", ["scan", "segments", "steps"])
@pytest.mark.parametrize("case", GRU)
@pytest.mark.parametrize("fresh", [True, False])
def test_min_gru(dtype, form, case, fresh):
    """Portions side by side from an empty and from a given state: outputs and the state they leave.  Gates from wide open to shut."""
    from tah_b200.ops import cuda as K
    lens, D = case
    d, n = _pad(D, 8), sum(lens)
    g = torch.Generator().manual_seed(n)
    rnd = lambda *s: torch.randn(*s, generator=g)
    z, u, gate = (4 * rnd(n, D) - 3).to(dtype), (3 * rnd(n, D)).to(dtype), rnd(n, D).to(dtype)
    z[1::7], u[2::5] = 40.0, -60.0                           # sigmoids at both ends
    z[3::11] = -45.0
    zb, xb = rnd(D), rnd(D)
    S0 = [torch.zeros(D, dtype=torch.float64) if fresh else rnd(D).double() for _ in lens]
    want, states, at = [], [], 0
    for c, s in zip(lens, S0):
        o, s = O.min_gru_core(z.double()[at:at + c] + zb.double(), u.double()[at:at + c] + xb.double(), s)
        want.append(o)
        states.append(s)
        at += c
    want = 0.6 * torch.cat(want) * gate.double() * torch.sigmoid(gate.double())
    proj = torch.full((n, 3 * d + 40), 3.0, dtype=dtype)
    proj[:, 16:16 + 3 * d] = torch.cat([_padt(t, d) for t in (z, u, gate)], 1)
    proj = proj.cuda()[:, 16:]
    out = torch.full((n, d + 24), 5.0, dtype=dtype, device="cuda")
    rows = torch.randperm(len(lens) + 2, generator=g)[:len(lens)]
    S = torch.full((len(lens) + 2, d), float("nan") if fresh else 0.0, device="cuda")
    if not fresh:
        for r, s in zip(rows, S0):
            S[r, :D] = s.float().cuda()
    keep = S.clone()
    off = 0 if fresh else 500
    pos, row = _i32(off + t for c in lens for t in range(c)), _i32(int(r) for r, c in zip(rows, lens) for _ in range(c))
    starts = [sum(lens[:i]) for i in range(len(lens))]
    a = lambda s: (proj[s], _padt(zb, d).cuda(), _padt(xb, d).cuda(), out[s, 8:8 + d], (S,), pos[s], row[s], 0.6)
    if form == "steps":
        live, idle = _i32([5]), _i32([-1])
        for t in range(min(120, max(lens))):
            for s, c in zip(starts, lens):
                if t < c:
                    K.min_gru_step(*a(slice(s + t, s + t + 1)), slot=live)
        before = S.clone()
        K.min_gru_step(*a(slice(0, 1)), slot=idle)                           # an idle row keeps its state
        assert torch.equal(before.nan_to_num(), S.nan_to_num())
        done = [s + t for s, c in zip(starts, lens) for t in range(min(120, c))]
    else:
        split = 1 if form == "scan" else 5
        ws = torch.full((len(lens) * split * 2 * d,), float("nan"), device="cuda")
        K.min_gru_scan(*a(slice(None)), seq_start=_i32(starts), seq_len=_i32(lens), n_split=split, ws=ws)
        done = list(range(n))
    got = out[:, 8:8 + D].double().cpu()[done]
    tol = 2e-5 if dtype == F32 else 6e-3
    assert float(((got - want[done]).abs() / (want[done].abs() + 0.02 * float(want.abs().max()))).max()) < tol
    assert bool((out[:, :8] == 5.0).all()) and bool((out[:, 8 + d:] == 5.0).all())
    if form != "steps" or max(lens) <= 120:
        for r, s in zip(rows, states):
            assert _err(S[r, :D], s) < 1e-5                                  # the recurrence is 32-bit, whatever the activations are
    others = [r for r in range(len(lens) + 2) if r not in rows.tolist()]
    assert torch.equal(S[others].nan_to_num(7.0), keep[others].nan_to_num(7.0))
    check_ok()


LATENT = [  # T, heads, rot, kv_rank, window
    (150, 3, 12, 72, 23), (300, 16, 64, 512, 48), (260, 36, 16, 192, 97), (140, 1, 2, 8, 1), (200, 20, 64, 64, 150), (300, 5, 72, 320, 64),
]


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode"])
@pytest.mark.parametrize("case", LATENT)
def test_windowed_latent_attention(kernel, case):
    """Single tokens against the cached rows themselves, keys that stand out on both sides of the window's end, no sink."""
    from tah_b200.ops import cuda as K
    T, nh, r, R, size = case
    dtype = F32 if kernel == "plain32" else BF16
    Rp, rw = _pad(R, 64), _pad(r, 64)
    g = torch.Generator().manual_seed(R)
    rnd = lambda *s: torch.randn(*s, generator=g)
    u = torch.nn.functional.normalize(rnd(R + r), dim=0) * math.sqrt(R + r)
    q, kk = 0.2 * rnd(T, nh, R + r) + 1.5 * u, 0.3 * rnd(T, 1, R + r)
    rows = sorted({p for p in (0, 1, 15, 16, 47, 48, 63, 64, 95, 96, 127, 128, size - 1, size, size + 1, T - 2, T - 1) if 0 <= p < T})
    for p in rows[::2]:
        for j in (p - size, p - size + 1):
            if j >= 0:
                kk[j] = (3.0 if j % 2 else -3.0) * u + 0.5 * rnd(R + r)
    q, kk = q.to(dtype).double(), kk.to(dtype).double()
    scale = 1.0 / math.sqrt(R + r)
    want = O.attention_core(q, kk, kk[..., :R], scale, size)
    n_pages = (T + 15) // 16
    perm = torch.randperm(n_pages + 3, generator=g)[:n_pages]
    pool = torch.zeros(n_pages + 3, 16, Rp + rw)
    for t in range(T):
        pool[perm[t // 16], t % 16, :R], pool[perm[t // 16], t % 16, Rp:Rp + r] = kk[t, 0, :R].float(), kk[t, 0, R:].float()
    pool = pool.view(n_pages + 3, -1).to("cuda", dtype)
    L = K.HeadLists(len(rows), nh, dtype, "cuda")
    ql = torch.zeros(nh, L.npad, Rp + rw)
    ql[:, :len(rows), :R], ql[:, :len(rows), Rp:Rp + r] = q[rows, :, :R].transpose(0, 1).float(), q[rows, :, R:].transpose(0, 1).float()
    ql = ql.view(-1, Rp + rw).to("cuda", dtype)
    pt = perm.to("cuda", torch.int32).view(1, -1).contiguous()
    at, zero = _i32(rows), _i32([0] * len(rows))
    for split in (1, 2, 4) if kernel == "decode" else (1,):
        out = torch.full((L.rows, Rp), 7.0, dtype=dtype, device="cuda")
        kw = dict(Rp=Rp, rw=rw, page_size=16, scale=scale, window=size)
        if kernel == "decode":
            K.latent_attn_decode(ql, out, pool, pt, at, zero, L, n_split=split, ws=torch.empty(len(rows) * nh * split * (Rp + 2), device="cuda"), **kw)
        else:
            K.latent_attn_plain(ql, out, pool, pt, at, zero, L, **kw)
        got = out.double().cpu().view(nh, L.npad, Rp)[:, :len(rows)].transpose(0, 1)
        assert float(_row_err(got[..., :R], want[rows]).max()) < (3e-5 if dtype == F32 else 2e-2), split
    v, o = torch.randn(L.rows, 64, device="cuda").to(dtype), torch.zeros(len(rows), nh * 24, dtype=dtype, device="cuda")
    K.latent_gate(v, L, None, o, 24)                       # back to token rows without a gate
    assert torch.equal(o.view(len(rows), nh, 24), v.view(nh, L.npad, 64)[:, :len(rows), :24].transpose(0, 1))
    check_ok()


# ------------------------------------------------------------------------------------
# the model through the engine's step function
# ------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(H.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompt_portions_and_single_tokens(tmp_path, name, dtype):
    cfg, sd, d = H.make(tmp_path, name)
    T = 210 if name in ("tiles", "wide") else 150
    toks = H.tokens(cfg, T)
    layers = []
    want = O.forward(cfg, sd, toks, layers_out=layers)
    e = engine(d, dtype)
    seen = []
    e.layer_hook = lambda i, x: seen.append(x.clone())
    whole = run_portions(e, toks, [T])
    e.layer_hook = None
    assert len(seen) == len(layers)
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
@pytest.mark.parametrize("kind", list(H.EDGES))
@pytest.mark.parametrize("size,pool,place", [(24, 5, 41), (24, 5, 0), (16, 16, 15), (64, 4, 63), (33, 12, 64), (48, 1, 16), (100, 7, 127)])
def test_edges_of_windows_and_blocks(tmp_path, dtype, kind, size, pool, place):
    """One key that every query finds: seen inside the window, gone behind its end, seen again in its block's mean, in a prompt, in
    portions that are cut at those places and in decoding."""
    special, T = 7, 260
    cfg = H.EDGES[kind](size, pool)
    sd = H.stand_out(cfg, O.random_model(cfg, 3), special, H.STRENGTH[kind])
    d = os.path.join(str(tmp_path), "ckpt")
    H.write_checkpoint(d, cfg, sd)
    toks = [t if t != special else special + 1 for t in H.tokens(cfg, T, 3)]
    toks[place] = special
    want = O.forward(cfg, sd, toks)
    e = engine(d, dtype)
    last, block = place + size, place // pool * pool + pool - 1 + size     # first query behind the window, first that sees the block
    cuts = sorted({c for c in (place, place + 1, last - 1, last, last + 1, block, block + 1) if 0 < c < T})
    pieces = [b - a for a, b in zip([0] + cuts, cuts + [T])]
    first = max(2, last - 5)
    for portions in ([T], pieces, [2] * (T // 2), [first] + [1] * min(60, T - first) + ([T - first - 60] if T - first > 60 else [])):
        assert H.close(run_portions(e, toks, portions), want, dtype), portions[:4]
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_mixed_batches_and_reused_pages_and_slots(tmp_path, dtype, name, monkeypatch):
    """Requests of unequal lengths in shared steps, in a pool that only holds a few of them, rows handed on, latents of a few pages
    expanded at a time; every request's logits equal those of the request alone."""
    from tah_b200.engine import StepEntry, hybrid
    monkeypatch.setattr(hybrid, "LATENT_PAGES", 6)
    cfg, sd, d = H.make(tmp_path, name, seed=1)
    g = torch.Generator().manual_seed(11)
    reqs = [H.tokens(cfg, n, seed=20 + i) for i, n in enumerate([90, 1, 37, 64, 130, 2, 17, 175, 50])]
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
    """More than a thousand tokens in a step (wide token tiles of the products, segments of the recurrence), unequal requests, latent
    expansions in several launches."""
    from tah_b200.engine import StepEntry, hybrid
    cfg, sd, d = H.make(tmp_path, "tiles", seed=9)
    reqs = [H.tokens(cfg, n, 60 + n) for n in (1150, 200, 260, 131)]
    want = [O.forward(cfg, sd, t) for t in reqs]
    for pages in (hybrid.LATENT_PAGES, 30):
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


def test_guard_pages_stay_untouched(tmp_path, monkeypatch):
    """Pages behind the pools, those of block means and key factors included, keep their pattern over portions, decoding and reuse."""
    monkeypatch.setenv("TAH_B200_CANARY", "2")
    for name in ("mixed", "odd"):
        cfg, sd, d = H.make(os.path.join(str(tmp_path), name), name)
        toks = H.tokens(cfg, 128)
        e = engine(d, BF16, rows=1, pool=128)
        for portions in ([128], [60] + [1] * 68, [2] * 64):
            run_portions(e, toks, portions)
        assert e.kv.guard_pages == 2 and e.kv.check_guards()
    check_ok()


@pytest.mark.parametrize("page", [8, 32])
def test_plain_kernels_in_bf16(tmp_path, page):
    """Other page sizes take the plain kernels; the pooled rows of a page follow its size."""
    cfg, sd, d = H.make(tmp_path, "mixed")
    toks = H.tokens(cfg, 100)
    e = engine(d, BF16, page_size=page)
    assert e.plain and H.close(run_portions(e, toks, [60, 1, 1, 38]), O.forward(cfg, sd, toks), BF16)
    check_ok()


def test_sizes_beyond_the_tensor_core_kernels(tmp_path):
    """Latents and heads that fit neither the decode kernel nor the portion kernel."""
    cfg = H.config([(H.latent(heads=2, dim=250, rot_dim=16, vdim=24, kv_rank=1300, scale=0.06, size=40), 88),
                    (H.latent(heads=2, dim=40, rot_dim=8, vdim=264, kv_rank=64, size=70), None), H.attn(heads=2, kv_heads=1, dim=256, scale=0.06)])
    cfg, sd, d = H.make(tmp_path, cfg)
    toks = H.tokens(cfg, 140)
    e = engine(d, BF16)
    assert [getattr(b.mixer, "w_exp", 0) is None for b in e.w.layers] == [True, True, False] and not e.w.layers[0].mixer.on_tensor_cores
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
