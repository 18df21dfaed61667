"""Gunuvik on the GPU: every mechanism against a plain statement of it, and the engine's steps, ticks and scheduler."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from tests import gunuvik_helpers as H
from tests.oracle import gunuvik_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16
LOG2E = 1.0 / math.log(2.0)


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


# ------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------
def _pad8(n):
    return (n + 7) // 8 * 8


def _paged(k, v, dtype, page=16, seed=0):
    """Scatter ``k [T, G, dk]``, ``v [T, G, dv]`` into a shuffled paged pool; returns (pool, page table [1, n])."""
    T, G, dk = k.shape
    dv = v.shape[2]
    n = (T + page - 1) // page
    total = n + 3
    g = torch.Generator().manual_seed(seed)
    perm = torch.randperm(total, generator=g)[:n]
    pool = torch.zeros(total, G * page * (dk + dv))
    for t in range(T):
        pg = pool[perm[t // page]]
        pg[:G * page * dk].view(G, page, dk)[:, t % page] = k[t]
        pg[G * page * dk:].view(G, page, dv)[:, t % page] = v[t]
    return pool.to("cuda", dtype), perm.to("cuda", torch.int32).view(1, -1).contiguous()


def _attn_case(T, nq, G, dim, vdim, window, keep, far, rel_rows, dtype, seed=0, peaks=()):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v = rnd(T, nq, dim), rnd(T, G, dim), rnd(T, G, vdim)
    if peaks:
        # all queries and the chosen keys share a direction, so that a chosen key dominates wherever it is visible
        u = torch.nn.functional.normalize(rnd(dim), dim=0) * math.sqrt(dim)
        q, k = 0.2 * q + 1.5 * u, 0.3 * k
        for n, j in enumerate(peaks):
            k[j] = 1.2 * u
            v[j] = 6.0 * torch.randn(G, vdim, generator=g)
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    rel, sink, gate = rnd(rel_rows, nq).double(), (1.0 + rnd(nq)).double(), rnd(T, nq).to(dtype).double()
    scale = 1.3 / math.sqrt(dim)
    own = torch.arange(nq) // (nq // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, own]) * scale + O.distance_bias(T, rel, far)
    w = O.sink_softmax(s, O.window_mask(T, window, keep), sink)
    want = torch.einsum("hij,jhd->ihd", w, v[:, own]) * torch.sigmoid(gate).unsqueeze(-1)
    return q, k, v, rel, sink, gate, scale, want


ATTN = [  # T, heads, kv heads, dim, vdim, window, keep, far, rel rows
    (150, 4, 2, 40, 24, 19, 3, 45, 14),
    (300, 3, 1, 64, 128, 64, 17, 250, 16),
    (260, 4, 4, 128, 64, 129, 1, 64, 32),
    (140, 6, 1, 16, 8, 16, 0, 20, 8),
    (200, 2, 2, 128, 128, None, 0, 100, 12),
    (170, 5, 1, 200, 136, 50, 70, 90, 10),
    (130, 8, 1, 72, 80, 1, 5, 33, 7),
]


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode", "tiles"])
@pytest.mark.parametrize("case", ATTN)
@pytest.mark.parametrize("peaked", [False, True])
def test_windowed_attention_kernels(kernel, case, peaked):
    from tah_b200.engine.hybrid import NO_WINDOW, distance_table
    from tah_b200.ops import cuda as K
    T, nq, G, dim, vdim, window, keep, far, rel_rows = case
    dtype = F32 if kernel == "plain32" else BF16
    # keys at the window's edges of the probed queries, at page borders, around the end of the kept part
    W = window or T
    probes = sorted({p for p in (T - 1, T - 2, T // 2, 127, 128, W, W + 1, keep, 15, 16, 64) if 0 <= p < T})
    peaks = sorted({j for j in (keep - 1, keep, T - 1 - W, T - W, T // 2 - W, T // 2 - W + 1, 15, 16, 63, 64, 128) if 0 <= j < T}) if peaked else ()
    q, k, v, rel, sink, gate, scale, want = _attn_case(T, nq, G, dim, vdim, window, keep, far, rel_rows, dtype, 3, peaks)
    dk, dv = _pad8(dim), _pad8(vdim)
    padded = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1])).float()
    pool, pt = _paged(padded(k, dk), padded(v, dv), dtype)
    unit = 1.0 if kernel.startswith("plain") else LOG2E
    kw = dict(nq=nq, nkv=G, dk=dk, dv=dv, page_size=16, scale=scale, window=NO_WINDOW if window is None else window,
              keep_first=keep, bias=(distance_table(rel, far) * unit).cuda(), sink=(sink.float() * unit).cuda())
    gate_d = gate.to("cuda", dtype)
    tol = 3e-5 if dtype == F32 else 2e-2
    top = float(want.abs().max())
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")

    def compare(out, rows):
        got = out.double().cpu().view(len(rows), nq, dv)
        assert float((got[..., :vdim] - want[rows]).abs().max()) <= tol * top
        assert float(got[..., vdim:].abs().max() if dv > vdim else 0.0) == 0.0

    if kernel == "tiles":
        # portions that start at several offsets: whole, in the middle of a page, the last two tokens
        for a, b in ((0, T), (37, T), (T - 2, T), (100, 129)):
            n = b - a
            qd = padded(q[a:b], dk).reshape(n, nq * dk).to("cuda", dtype)
            out = torch.zeros(n, nq * dv, dtype=dtype, device="cuda")
            t0 = list(range(0, n, 128))
            K.window_attn_tiles(qd, out, pool, pt, i32(range(a, b)), i32([0] * n), i32(t0), i32([min(128, n - x) for x in t0]),
                                pool.shape[0], gate=gate_d[a:b], **kw)
            compare(out, list(range(a, b)))
    else:
        rows = list(range(T)) if kernel.startswith("plain") else probes
        n = len(rows)
        qd = padded(q[rows], dk).reshape(n, nq * dk).to("cuda", dtype)
        args = (pool, pt, i32(rows), i32([0] * n))
        if kernel == "decode":
            for split in (1, 3):
                out = torch.zeros(n, nq * dv, dtype=dtype, device="cuda")
                ws = torch.empty(n * nq * split * (dv + 2), device="cuda")
                K.window_attn_decode(qd, out, *args, gate=gate_d[rows].contiguous(), n_split=split, ws=ws, **kw)
                compare(out, rows)
        else:
            out = torch.zeros(n, nq * dv, dtype=dtype, device="cuda")
            K.window_attn_plain(qd, out, *args, gate=gate_d[rows].contiguous(), **kw)
            compare(out, rows)
    check_ok()


def test_attention_options_absent():
    """No bias, no sink, no gate: ordinary causal softmax attention."""
    from tah_b200.engine.hybrid import NO_WINDOW
    from tah_b200.ops import cuda as K
    T, nq, G, d = 90, 4, 2, 32
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(T, h, d, generator=g).to(BF16) for h in (nq, G, G))
    own = torch.arange(nq) // 2
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double()[:, own]) * 0.2
    want = torch.einsum("hij,jhd->ihd", s.masked_fill(~O.window_mask(T, None, 0), -math.inf).softmax(-1), v.double()[:, own])
    pool, pt = _paged(k.float(), v.float(), BF16)
    kw = dict(nq=nq, nkv=G, dk=d, dv=d, page_size=16, scale=0.2, window=NO_WINDOW, keep_first=0)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    qd = q.reshape(T, -1).cuda()
    for run in ("plain", "decode", "tiles"):
        out = torch.zeros(T, nq * d, dtype=BF16, device="cuda")
        args = (qd, out, pool, pt, i32(range(T)), i32([0] * T))
        if run == "plain":
            K.window_attn_plain(*args, **kw)
        elif run == "decode":
            K.window_attn_decode(*args, **kw)
        else:
            K.window_attn_tiles(*args, i32([0]), i32([T]), pool.shape[0], **kw)
        assert float((out.double().cpu().view(T, nq, d) - want).abs().max()) < 2e-2 * float(want.abs().max())
    check_ok()


@pytest.mark.parametrize("heads,dim,vdim,cap", [(3, 24, 56, 9.0), (1, 13, 19, 4.0), (2, 128, 256, 15.0), (2, 64, 64, 30.0), (1, 72, 200, 6.0)])
@pytest.mark.parametrize("kernel", ["recurrent32", "recurrent", "chunks"])
@pytest.mark.parametrize("shift", [0.0, -6.0, 6.0])
def test_mlstm_kernels(kernel, heads, dim, vdim, cap, shift):
    """Recurrent and chunkwise kernels against the token-by-token cell; ``shift`` moves the gates so that the running
    maximum comes from the start value, from decayed old tokens or from new ones."""
    from tah_b200.ops import cuda as K
    T = 300
    dtype = F32 if kernel == "recurrent32" else BF16
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v, og = (rnd(T, heads, d).to(dtype) for d in (dim, dim, vdim, vdim))
    z = rnd(T, 2 * heads)
    z[:, :heads] = 3 * z[:, :heads] + shift
    z[:, heads:] = 2 * z[:, heads:] + 3.0 - shift / 2
    z[T // 2, heads:] = -40.0                                  # one token forgets almost everything
    z[T // 3, :heads] = 25.0                                   # one token takes over the running maximum
    nw = 1.0 + 0.2 * rnd(heads * vdim)
    eps = 1e-5
    want = []
    for h in range(heads):
        li = cap * torch.tanh(z[:, h].double() / cap)
        lf = torch.nn.functional.logsigmoid(cap * torch.tanh(z[:, heads + h].double() / cap))
        want.append(O.mlstm_cell(q[:, h].double() * dim ** -0.5, k[:, h].double(), v[:, h].double(), li, lf))
    want = O.rms_norm(torch.stack(want, 1), eps) * nw.double().view(heads, vdim) * torch.sigmoid(og.double())
    dk, dv = _pad8(dim), _pad8(vdim)
    pad = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1])).reshape(T, -1)
    F = (2 * dk + 2 * dv) * heads
    x = torch.zeros(T, (F + 63) // 64 * 64, dtype=dtype)
    x[:, :F] = torch.cat([pad(q, dk), pad(k, dk), pad(v, dv), pad(og, dv)], 1)
    x, zd = x.cuda(), z.cuda()
    nwp = torch.nn.functional.pad(nw.view(heads, vdim), (0, dv - vdim)).reshape(-1).cuda()
    kw = dict(heads=heads, dk=dk, dv=dv, dim=dim, vdim=vdim, cap=cap, eps=eps)
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")
    rows = 3
    for portions in ((300,), (128, 128, 44), (2, 3, 120, 1, 174), (100, 200)):
        # a slot full of garbage: a sequence at position 0 must not read it
        state = tuple(torch.full((rows, *s), 7.0, device="cuda") for s in ((heads, dk, dv), (heads, dk), (heads,)))
        out = torch.zeros(T, heads * dv, dtype=dtype, device="cuda")
        at = 0
        for c in portions:
            sl = slice(at, at + c)
            pos, row = i32(range(at, at + c)), i32([1] * c)
            args = (x[sl], zd[sl].contiguous(), nwp, out[sl], state, pos, row)
            if kernel != "chunks" or c == 1:
                K.mlstm_recurrent(*args, seq_start=i32([0]), seq_len=i32([c]), **kw)
            else:
                st = list(range(0, c, 128))
                K.mlstm_chunks(*args, chunk_start=i32(st), chunk_len=i32([min(128, c - a) for a in st]), seq_chunk0=i32([0]),
                               seq_chunks=i32([len(st)]), ws=torch.full((K.mlstm_chunk_ws_floats(len(st), heads, dk, dv),), 3.0, device="cuda"), **kw)
            at += c
        got = out.double().cpu().view(T, heads, dv)[..., :vdim]
        # errors relative to each token's own output size
        err = (got - want).abs().amax(-1) / want.abs().amax(-1).clamp(min=1e-3)
        assert float(err.max()) < (2e-4 if dtype == F32 else 2e-2), (portions, float(err.max()))
        assert float(state[0][0].min()) == 7.0 and float(state[0][2].min()) == 7.0      # other slots untouched
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_norm_and_small_kernels(dtype):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == F32 else 1e-2
    for width, ld, M in ((77, 128, 5), (136, 192, 33), (2048, 2048, 9), (5000, 5056, 3)):
        z = lambda t: torch.nn.functional.pad(t, (0, ld - width))
        E, w, w2 = rnd(50, width).to(dtype), rnd(width), rnd(width)
        ids = torch.randint(0, 50, (M,), generator=g).to(torch.int32)
        x, h = torch.empty(M, ld, device="cuda"), torch.empty(M, ld, dtype=dtype, device="cuda")
        K.embed_norm(z(E).cuda(), ids.cuda(), 3.5, z(w).cuda(), width, 1e-4, x, h)
        ref = E.double()[ids.long()] * 3.5
        assert torch.allclose(x.cpu().double()[:, :width], ref, rtol=1e-6, atol=1e-6)
        want = O.rms_norm(ref, 1e-4, w.double())
        assert float((h.cpu().double()[:, :width] - want).abs().max()) < tol * float(want.abs().max())
        y = rnd(M, width).to(dtype)
        K.residual_norm(z(y).cuda(), x, z(w2).cuda(), z(w).cuda(), width, 1e-4, h)
        ref = ref + O.rms_norm(y.double(), 1e-4, w2.double())
        assert torch.allclose(x.cpu().double()[:, :width], ref, rtol=1e-5, atol=1e-5)
        want = O.rms_norm(ref, 1e-4, w.double())
        assert float((h.cpu().double()[:, :width] - want).abs().max()) < tol * float(want.abs().max())
    for M in (1, 3, 200):
        for K_, F in ((128, 2), (192, 34), (2048, 16)):
            x, w, b = rnd(M, K_).to(dtype), rnd(F, K_).to(dtype), rnd(F)
            got = K.few_linear(x.cuda(), w.cuda(), b.cuda())
            assert torch.allclose(got.cpu().double(), x.double() @ w.double().T + b.double(), rtol=1e-4, atol=2e-4)
    if dtype == F32:
        x, w = rnd(37, 192), rnd(2 * 70, 192)
        assert torch.allclose(K.linear(x.cuda(), w.cuda()).cpu().double(), x.double() @ w.double().T, rtol=1e-4, atol=1e-4)
        gu = x.double() @ w.double().T
        want = O.silu(gu[:, :70]) * gu[:, 70:]
        assert torch.allclose(K.swiglu_linear(x.cuda(), w.cuda()).cpu().double(), want, rtol=1e-4, atol=1e-3)
        lg = rnd(4, 301).cuda()
        best, cum = torch.zeros(4, dtype=torch.int32, device="cuda"), torch.zeros_like(lg)
        K.logits_post(lg, cum, None, best)
        assert torch.equal(best.long(), lg.argmax(-1)) and torch.equal(cum, lg)
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_projection_bias_norm_and_cache_write(dtype):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g)
    M, nq, G, dim, vdim, page = 21, 3, 2, 20, 33, 16
    dk, dv = _pad8(dim), _pad8(vdim)
    padh = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1]))
    q, k, v = rnd(M, nq, dim).to(dtype), rnd(M, G, dim).to(dtype), rnd(M, G, vdim).to(dtype)
    bq, bk, bv, wq, wk = rnd(nq, dim), rnd(G, dim), rnd(G, vdim), rnd(dim), rnd(dim)
    qkv = torch.cat([padh(q, dk).reshape(M, -1), padh(k, dk).reshape(M, -1), padh(v, dv).reshape(M, -1), torch.zeros(M, 8, dtype=dtype)], 1).cuda()
    bias = torch.cat([padh(bq, dk).reshape(-1), padh(bk, dk).reshape(-1), padh(bv, dv).reshape(-1), torch.zeros(8)]).cuda()
    slot = torch.randperm(64, generator=g)[:M].to(torch.int32)
    slot[4] = -1
    pool = torch.zeros(4, G * page * (dk + dv), dtype=dtype, device="cuda")
    out = torch.zeros(M, nq * dk, dtype=dtype, device="cuda")
    K.qkv_post(qkv, bias, padh(wq, dk).cuda(), padh(wk, dk).cuda(), out, pool, slot.cuda(), nq, G, dk, dv, dim, page, 1e-3)
    tol = 1e-5 if dtype == F32 else 1e-2
    want = O.rms_norm(q.double() + bq.double(), 1e-3, wq.double())
    assert float((out.cpu().double().view(M, nq, dk)[..., :dim] - want).abs().max()) < tol * float(want.abs().max())
    kw_, vw = O.rms_norm(k.double() + bk.double(), 1e-3, wk.double()), v.double() + bv.double()
    pc = pool.cpu().double()
    for t in range(M):
        s = int(slot[t])
        if s < 0:
            continue
        pg = pc[s // page]
        kt = pg[:G * page * dk].view(G, page, dk)[:, s % page]
        vt = pg[G * page * dk:].view(G, page, dv)[:, s % page]
        assert float((kt[:, :dim] - kw_[t]).abs().max()) < tol * float(kw_.abs().max())
        assert float((vt[:, :vdim] - vw[t]).abs().max()) < tol * float(vw.abs().max())
    before = pool.clone()                                     # queries only: the cache of another layer stays as it is
    K.qkv_post(qkv, bias, padh(wq, dk).cuda(), None, out, pool, slot.cuda(), nq, 0, dk, dv, dim, page, 1e-3)
    assert torch.equal(before, pool)
    check_ok()


# ------------------------------------------------------------------------------------
# the model through the engine's step function
# ------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(H.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompt_portions_and_single_tokens(tmp_path, name, dtype):
    cfg, sd, d = H.make(tmp_path, name)
    T = 210 if name == "tiles" else 150
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
        assert err < (2e-5 if dtype == F32 else 6e-2), (i, err)
    assert H.close(whole, want, dtype)
    for portions in ([1] * T, [2] * (T // 2), [3, 1, 64, 1, 2, T - 71], [17] * (T // 17) + [T % 17], [T - 40] + [1] * 40, [16, 16, 48, T - 80],
                     [128, T - 128]):
        portions = [p for p in portions if p]
        got = run_portions(e, toks, portions)
        assert H.close(got, want, dtype), portions[:4]
    assert e.kv.pages_in_use(0) == 0
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_and_reused_pages_and_slots(tmp_path, dtype):
    """Requests of unequal lengths in shared steps, in a pool that only holds a few of them, rows handed on; every
    request's logits equal those of the request alone."""
    from tah_b200.engine import StepEntry
    cfg, sd, d = H.make(tmp_path, "mixed", seed=1)
    g = torch.Generator().manual_seed(11)
    lengths = [90, 1, 37, 64, 130, 2, 17, 75, 50]
    reqs = [H.tokens(cfg, n, seed=20 + i) for i, n in enumerate(lengths)]
    want = [O.forward(cfg, sd, t) for t in reqs]
    e = engine(d, dtype, rows=3, pool=288)
    live, at, queue, got = {}, {}, list(range(len(reqs))), [[] for _ in reqs]
    rows_used = set()
    while queue or live:
        held = lambda: sum((len(reqs[r]) + 15) // 16 * 16 for r in live)
        while queue and len(live) < 3 and held() + (len(reqs[queue[0]]) + 15) // 16 * 16 <= 288:
            r = queue.pop(0)
            live[r], at[r] = e.admit(), 0
            rows_used.add(live[r])
        entries, who = [], []
        for r in list(live):
            if len(live) > 1 and torch.rand((), generator=g) < 0.25:
                continue                                           # left out of this step
            n = int(torch.tensor([1, 1, 2, 5, 16, 31, 60])[torch.randint(0, 7, (), generator=g)])
            n = min(n, len(reqs[r]) - at[r])
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
    """bf16: the same portion of the same request gives the same logits, up to a last-bit rounding here and there, on
    other pages, in another row and beside other requests."""
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


def test_large_steps_and_grouped_chunk_launches(tmp_path, monkeypatch):
    """More than a thousand tokens in a step (the GEMM's two-tile form), and a step whose recurrent chunks need several
    launches; the portions of unequal requests side by side."""
    from tah_b200.engine import StepEntry, hybrid
    cfg, sd, d = H.make(tmp_path, "tiles", seed=9)
    reqs = [H.tokens(cfg, n, 60 + n) for n in (1150, 200, 260, 131)]
    want = [O.forward(cfg, sd, t) for t in reqs]
    for limit in (hybrid.MEMORY_CHUNKS, 3):
        monkeypatch.setattr(hybrid, "MEMORY_CHUNKS", limit)
        e = engine(d, BF16, rows=4, pool=2048)
        rows = [e.admit() for _ in reqs]
        a = e.step([StepEntry(r, t[:len(t) - 70], range(len(t) - 70)) for r, t in zip(rows, reqs)]).float().cpu()
        b = e.step([StepEntry(r, t[len(t) - 70:], range(70)) for r, t in zip(rows, reqs)]).float().cpu()
        at = 0
        for i, w in enumerate(want):
            n = len(reqs[i]) - 70
            assert H.close(torch.cat([a[at:at + n], b[70 * i:70 * i + 70]]), w, BF16), (limit, i)
            at += n
    check_ok()


def test_pool_exhaustion_is_an_error_and_leaves_the_cache_usable(tmp_path):
    from tah_b200.engine import StepEntry
    from tah_b200.ops import cuda as K
    cfg, sd, d = H.make(tmp_path, "mixed")
    toks = H.tokens(cfg, 200)
    e = engine(d, F32, rows=2, pool=96)
    row = e.admit()
    e.step([StepEntry(row, toks[:50], ())])
    e.step([StepEntry(row, toks[50:200], ())])
    torch.cuda.synchronize()
    with pytest.raises(K.KernelTimeout):
        K.check_status()
    e.release(row)
    assert e.kv.pages_in_use(0) == 0
    got = run_portions(e, toks[:90], [60, 30])
    assert H.close(got, O.forward(cfg, sd, toks[:90]), F32)


# ------------------------------------------------------------------------------------
# generation through generate() and serve()
# ------------------------------------------------------------------------------------
def _greedy(cfg, sd, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, sd, toks)[-1].argmax()))
    return toks[len(prompt):]


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
    n_new = 60
    for _ in range(2):                                  # the second call replays the captured tick
        res = e.generate(ids, mask, max_new_tokens=n_new)
        for p, out in zip(prompts, res.tokens):
            assert len(out) == n_new
            assert _tokens_follow(cfg, sd, p, out, 1e-4 if dtype == F32 else 0.15)


def test_long_decoding_crosses_windows_and_pages(tmp_path):
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
    e = make_engine(load_model(d, F32, "cuda"), max_rows=3)
    prompts = [H.tokens(cfg, n, 40 + i) for i, n in enumerate([30, 3, 71, 12, 1, 44, 25])]
    for _ in range(2):
        res, stats = e.serve([torch.tensor(p) for p in prompts], max_new_tokens=20, portion=16, check_every=4)
        assert stats["admitted"] == 7 and stats["mixed_steps"] > 7 and stats["tokens"] == 140
        for p, out in zip(prompts, res):
            assert _tokens_follow(cfg, sd, p, out, 1e-4)
        assert e.kv.pages_in_use(0) == 0
    # an EOS ends a request early, and its place goes to the next one
    eos = res[2][5]
    res2, _ = e.serve([torch.tensor(p) for p in prompts], max_new_tokens=20, portion=16, check_every=4, eos_token_id=eos)
    for a, b in zip(res, res2):
        assert b == (a[:a.index(eos)] if eos in a else a)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_sampling(tmp_path, dtype):
    from tah_b200.engine import get_engine
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, "mixed", seed=6)
    e = get_engine(load_model(d, dtype, "cuda"), max_rows=4)
    ids = torch.tensor([H.tokens(cfg, 12, 1), H.tokens(cfg, 12, 2)])
    for kw in (dict(top_k=5), dict(top_k=0, top_p=0.9), dict(top_k=20, min_p=0.05)):
        a = e.generate(ids, None, max_new_tokens=12, do_sample=True, temperature=0.8, seed=7, **kw).tokens
        b = e.generate(ids, None, max_new_tokens=12, do_sample=True, temperature=0.8, seed=7, **kw).tokens
        c = e.generate(ids, None, max_new_tokens=12, do_sample=True, temperature=0.8, seed=8, **kw).tokens
        assert a == b and a != c and all(0 <= t < cfg["vocab"] for r in a for t in r)
    res, _ = e.serve([ids[0], ids[1], ids[0, :5]], max_new_tokens=9, rows=2, do_sample=True, top_k=3, seed=1)
    assert [len(r) for r in res] == [9, 9, 9]
    # top_k = 1 is greedy (the samplers see bf16 logits: in the 32-bit mode a near tie may fall the other way)
    if dtype == F32:
        return
    g = e.generate(ids, None, max_new_tokens=12).tokens
    assert e.generate(ids, None, max_new_tokens=12, do_sample=True, top_k=1, seed=3).tokens == g


def test_trace_replay_program(tmp_path):
    cfg, sd, d = H.make(tmp_path, "odd", seed=7)
    a, b = H.tokens(cfg, 40, 1), H.tokens(cfg, 9, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:25], want=[24])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[8, 0]), dict(id="a", tokens=a[25:26], want=[0])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=a[26:30], want=[])], end=[]),
             dict(step=3, entries=[dict(id="c", tokens=b[:2], want=[1]), dict(id="a", tokens=a[30:], want=[9])], end=["a", "c"])]
    out = os.path.join(str(tmp_path), "out")
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out, "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        assert not os.path.exists(os.path.join(out, "2.f32"))
        la, lb = O.forward(cfg, sd, a), O.forward(cfg, sd, b)
        for step, want in ((0, la[24:25]), (1, torch.stack([lb[8], lb[0], la[25]])), (3, torch.stack([lb[1], la[39]]))):
            raw = torch.frombuffer(bytearray(open(os.path.join(out, f"{step}.f32"), "rb").read()), dtype=torch.float32)
            assert H.close(raw.view(-1, cfg["vocab"]), want, getattr(torch, dtype))
            os.unlink(os.path.join(out, f"{step}.f32"))


def test_playground_command_line_and_evaluation_backend(tmp_path):
    from tah_b200.evaluate.backends import setup_backend
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

    class Ids:                                             # a tokenizer whose texts are token ids
        eos_token_id = None
        encode = staticmethod(lambda s: [int(t) for t in s.split()])
        decode = staticmethod(lambda ids: " ".join(map(str, ids)))

    model, infer = setup_backend("engine", dict(dtype="float32", max_new_tokens=8, batch_size=4), d, Ids())
    for rows_n in (1, 2):
        got = infer.serve_all([Ids.decode(p) for p in prompts], rows_n)
        assert [Ids.encode(t) for t, _ in got] == rows
