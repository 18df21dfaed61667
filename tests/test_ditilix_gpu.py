"""Ditilix on the GPU: every mechanism against a plain statement of it, and the engine's steps, ticks and scheduler."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from tests import ditilix_helpers as H
from tests.oracle import ditilix_oracle as O

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
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _pad8(n):
    return (n + 7) // 8 * 8


def _paged(k, v, dtype, page=16):
    """Scatter ``k [T, G, dk]``, ``v [T, G, dv]`` into a shuffled paged pool; returns (pool, page table [1, n])."""
    T, G, dk = k.shape
    dv = v.shape[2]
    n = (T + page - 1) // page
    perm = torch.randperm(n + 3, generator=torch.Generator().manual_seed(0))[:n]
    pool = torch.zeros(n + 3, G * page * (dk + dv))
    for t in range(T):
        pg = pool[perm[t // page]]
        pg[:G * page * dk].view(G, page, dk)[:, t % page] = k[t]
        pg[G * page * dk:].view(G, page, dv)[:, t % page] = v[t]
    return pool.to("cuda", dtype), perm.to("cuda", torch.int32).view(1, -1).contiguous()


# ------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------
ATTN = [  # T, heads, kv heads, dim, vdim, cap, temperature, size of the scores
    (150, 4, 2, 40, 24, 3.0, (0.4, 23), 1.0),
    (300, 3, 1, 64, 128, 20.0, (0.3, 100), 4.0),       # arguments of the cap well inside (-1, 1)
    (260, 4, 4, 128, 64, 1.5, (0.9, 1), 3.0),          # saturated scores
    (140, 6, 1, 16, 8, 5.0, None, 5.0),                # arguments on both sides of 1
    (200, 2, 2, 128, 128, None, (0.5, 17.5), 1.0),     # no cap
    (170, 5, 1, 200, 136, 8.0, (0.2, 64), 2.0),
    (130, 8, 1, 72, 80, 30.0, (0.7, 128), 1.0),
]


@pytest.mark.parametrize("kernel", ["plain32", "plain", "decode", "tiles"])
@pytest.mark.parametrize("case", ATTN)
@pytest.mark.parametrize("peaked", [False, True])
def test_capped_attention_kernels(kernel, case, peaked):
    from tah_b200.engine.hybrid import NO_WINDOW
    from tah_b200.ops import cuda as K
    T, nq, G, dim, vdim, cap, temp, size = case
    dtype = F32 if kernel == "plain32" else BF16
    g = torch.Generator().manual_seed(4)
    rnd = lambda *s: torch.randn(*s, generator=g)
    q, k, v = rnd(T, nq, dim), rnd(T, G, dim), rnd(T, G, vdim)
    if peaked:
        # keys that stand out, far away, at page and tile borders: each dominates what sees it
        u = torch.nn.functional.normalize(rnd(dim), dim=0) * math.sqrt(dim)
        q, k = 0.2 * q + 1.5 * u, 0.3 * k
        for j in (0, 15, 16, 63, 64, 127, 128, T - 1):
            k[j] = 3.0 * u
            v[j] = 6.0 * rnd(G, vdim)
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    scale = size / math.sqrt(dim)
    qt = q if temp is None else q * O.query_temperature(range(T), *temp).view(T, 1, 1)
    want = O.attention_core(qt, k, v, scale, cap)
    dk, dv = _pad8(dim), _pad8(vdim)
    padded = lambda t, d: torch.nn.functional.pad(t, (0, d - t.shape[-1])).float()
    pool, pt = _paged(padded(k, dk), padded(v, dv), dtype)
    kw = dict(nq=nq, nkv=G, dk=dk, dv=dv, page_size=16, scale=scale, window=NO_WINDOW, keep_first=0, softcap=cap, q_temp=temp)
    tol = 3e-5 if dtype == F32 else 2e-2

    def queries(rows):                               # inside a wider matrix, as a projection leaves them
        m = torch.full((len(rows), nq * dk + 64), 3.0, device="cuda", dtype=dtype)
        m[:, :nq * dk] = padded(q[rows], dk).reshape(len(rows), -1).to("cuda", dtype)
        return m[:, :nq * dk]

    def compare(out, rows):
        got = out.double().cpu().view(len(rows), nq, dv)
        err = (got[..., :vdim] - want[rows]).abs().amax((1, 2)) / want[rows].abs().amax((1, 2)).clamp(min=0.3 * float(want.abs().max()))
        assert float(err.max()) <= tol
        assert float(got[..., vdim:].abs().max() if dv > vdim else 0.0) == 0.0

    if kernel == "tiles":
        for a, b in ((0, T), (37, T), (T - 2, T), (100, 129)):
            n, t0 = b - a, list(range(0, b - a, 128))
            out = torch.zeros(n, nq * dv, dtype=dtype, device="cuda")
            K.window_attn_tiles(queries(list(range(a, b))), out, pool, pt, _i32(range(a, b)), _i32([0] * n), _i32(t0),
                                _i32([min(128, n - x) for x in t0]), pool.shape[0], **kw)
            compare(out, list(range(a, b)))
    else:
        rows = list(range(T)) if kernel.startswith("plain") else sorted({p for p in (0, 1, 15, 16, 17, 63, 64, 99, 127, 128, 129, T - 2, T - 1) if p < T})
        n = len(rows)
        args = (pool, pt, _i32(rows), _i32([0] * n))
        for split in (1, 3) if kernel == "decode" else (1,):
            out = torch.zeros(n, nq * dv, dtype=dtype, device="cuda")
            if kernel == "decode":
                K.window_attn_decode(queries(rows), out, *args, n_split=split, ws=torch.empty(n * nq * split * (dv + 2), device="cuda"), **kw)
            else:
                K.window_attn_plain(queries(rows), out, *args, **kw)
            compare(out, rows)
    check_ok()


def test_score_cap_of_every_size():
    """One key per query: cap * tanh(s / cap) from tiny to saturated arguments shows in the weight against a key of score 0."""
    from tah_b200.engine.hybrid import NO_WINDOW
    from tah_b200.ops import cuda as K
    T, d, cap = 128, 64, 4.0
    q = torch.zeros(T, 1, d)
    q[:, 0, 0] = torch.linspace(-4.0, 4.0, T) ** 3 / 4
    k, v = torch.zeros(T, 1, d), torch.zeros(T, 1, d)
    k[0, 0, 0], v[0, 0, :] = 1.0, 1.0
    q, k, v = (t.to(BF16).double() for t in (q, k, v))
    want = O.attention_core(q, k, v, 1.0, cap)[:, 0, 0]
    pool, pt = _paged(k.float(), v.float(), BF16)
    out = torch.zeros(T, d, dtype=BF16, device="cuda")
    K.window_attn_tiles(q.view(T, d).to("cuda", BF16), out, pool, pt, _i32(range(T)), _i32([0] * T), _i32([0]), _i32([T]), pool.shape[0],
                        nq=1, nkv=1, dk=d, dv=d, page_size=16, scale=1.0, window=NO_WINDOW, keep_first=0, softcap=cap)
    err = (out[:, 0].double().cpu() - want).abs() / want
    assert float(err.max()) < 1.2e-2
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_positions_and_grouped_norms(dtype):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == F32 else 1e-2
    # parts of whole 128-column blocks, parts that no vector or warp respects, single columns, one part
    for width, ld, groups, M in ((512, 512, 4, 5), (2048, 2048, 2, 3), (77, 128, 7, 9), (132, 192, 6, 4), (96, 128, 96, 2), (90, 128, 1, 3),
                                 (5000, 5056, 8, 2), (384, 384, 3, 40)):
        z = lambda t: torch.nn.functional.pad(t, (0, ld - width))
        E, w, w2 = rnd(50, width).to(dtype), rnd(width), rnd(width)
        ids = torch.randint(0, 50, (M,), generator=g).to(torch.int32)
        pos = torch.randint(0, 70000, (M,), generator=g).to(torch.int32)
        pos[0] = 0
        x, h = torch.empty(M, ld, device="cuda"), torch.empty(M, ld, dtype=dtype, device="cuda")
        K.embed_norm(z(E).cuda(), ids.cuda(), 1.0, z(w).cuda(), width, 1e-4, x, h, groups=groups, pos=pos.cuda(),
                     freq=K.sinusoid_frequencies(width, device="cuda"))
        ref = E.double()[ids.long()] + O.sinusoid(pos.tolist(), width)
        assert float((x.cpu().double()[:, :width] - ref).abs().max()) < 2e-6
        want = O.group_rms_norm(ref, groups, 1e-4, w.double())
        assert float((h.cpu().double()[:, :width] - want).abs().max()) < tol * float(want.abs().max())
        assert float(h[:, width:].float().abs().sum()) == 0 and float(x[:, width:].abs().sum()) == 0
        y, ye = rnd(M, width).to(dtype), rnd(11, width).to(dtype)
        slot = torch.randint(0, 11, (M, 3), generator=g).to(torch.int32)
        for ex in (False, True):
            K.residual_add_norm(z(y).cuda(), x, 0.7, z(w2).cuda(), width, groups, 1e-4, h, z(ye).cuda() if ex else None, slot.cuda() if ex else None)
            ref = ref + 0.7 * (y.double() + (ye.double()[slot.long()].sum(1) if ex else 0.0))
            assert float((x.cpu().double()[:, :width] - ref).abs().max()) < 1e-5
            want = O.group_rms_norm(ref, groups, 1e-4, w2.double())
            assert float((h.cpu().double()[:, :width] - want).abs().max()) < tol * float(want.abs().max())
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_activations(dtype):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-5 if dtype == F32 else 1e-2
    act = torch.tensor([0.7, -0.3, 0.5, 0.2])
    for n, M in ((45, 3), (320, 5), (1000, 2), (4096, 3), (9216, 2), (17000, 2)):
        cols = (n + 63) // 64 * 64
        z = (1.5 * rnd(M, n)).to(dtype)
        wide = torch.zeros(M, cols + 128, dtype=dtype, device="cuda")
        wide[:, 64:64 + n] = z.cuda()
        out = torch.zeros(M, cols + 64, dtype=dtype, device="cuda")
        K.poly_norm(wide[:, 64:64 + cols], act.cuda(), n, 1e-3, out[:, 64:])
        want = O.poly_norm(z.double(), act.double(), 1e-3)
        assert float((out[:, 64:64 + n].cpu().double() - want).abs().max()) < tol * float(want.abs().max())
        assert float(out[:, :64].float().abs().sum()) == 0
    for n, M in ((24, 7), (64, 300), (768, 9)):
        gu = (2 * rnd(M, n, 2)).to(dtype)
        w, gate = torch.rand(M, generator=g), rnd(M, 5)
        out = torch.zeros(M, n, dtype=dtype, device="cuda")
        K.clamped_glu(gu.view(M, -1).cuda(), 1.3, out)
        want = O.clamped_glu(gu[..., 0].double(), gu[..., 1].double(), 1.3)
        assert float((out.cpu().double() - want).abs().max()) < tol * float(want.abs().max())
        K.clamped_glu(gu.view(M, -1).cuda(), 0.6, out, in_scale=w.cuda(), gate=gate.cuda()[:, 2])
        ww = w.double().view(M, 1)
        want = O.clamped_glu(ww * gu[..., 0].double(), ww * gu[..., 1].double(), 0.6) * torch.sigmoid(gate[:, 2:3].double())
        assert float((out.cpu().double() - want).abs().max()) < tol * float(want.abs().max())
    check_ok()


@pytest.mark.parametrize("M,E,top", [(1, 8, 1), (1, 5, 5), (7, 37, 3), (300, 9, 1), (256, 64, 8), (4200, 5, 2), (33, 1000, 4), (5000, 64, 6)])
@pytest.mark.parametrize("skew", [False, True])
def test_router_and_expert_lists(M, E, top, skew):
    """Chosen experts, weights and lists; a second launch finds clean counters.  ``skew``: nearly all tokens pick one expert."""
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(M + E)
    for bn in (16, 64):
        L = K.ExpertLists(M, E, top, BF16, "cuda", bn=bn)
        for rep in range(2):
            z = 2 * torch.randn(M, E + 1, generator=g)
            if skew:
                z[:, E // 2] += 6.0
            K.moe_route(z.cuda(), L)
            h = torch.randn(M, 64, generator=g).to(BF16)
            x = K.moe_gather(h.cuda(), L, torch.empty(L.rows, 64, dtype=BF16, device="cuda"))
            s = torch.sigmoid(z[:, :E])
            want = s.topk(top, -1)
            got = L.expert.cpu().long()
            assert torch.equal(got.sort(-1).values, want.indices.sort(-1).values)
            assert torch.allclose(L.weight.cpu(), s.gather(1, got), rtol=1e-6)
            slot, nb, blk = L.slot.cpu().long(), int(L.n_blocks), L.blk_expert.cpu().long()
            assert slot.unique().numel() == M * top and int(slot.max()) < nb * bn
            assert torch.equal(blk[slot // bn], got)                           # every row lies in a block of its expert
            count = torch.bincount(got.flatten(), minlength=E)
            assert nb == int(((count + bn - 1) // bn).sum()) <= L.max_blocks
            assert torch.equal(x.cpu()[slot], h[:, None].expand(M, top, 64))
            assert torch.equal(L.row_weight.cpu()[slot], L.weight.cpu())
            assert int(L.count.abs().sum()) == 0
    check_ok()


@pytest.mark.parametrize("M,F", [(5, 65), (2048, 65), (3001, 130), (2500, 33)])
def test_router_logits(M, F):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(0)
    x, w = torch.randn(M, 192, generator=g).to(BF16), torch.randn(F, 192, generator=g).to(BF16)
    got = K.few_linear(x.cuda(), w.cuda(), None).cpu().double()
    assert float((got - x.double() @ w.double().T).abs().max()) < 1e-4
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,E,top,width,ff,bn", [(3, 5, 2, 128, 64, 16), (40, 3, 1, 192, 128, 32), (150, 9, 2, 64, 192, 64), (700, 4, 2, 320, 64, 128),
                                                 (900, 2, 1, 128, 320, 256), (2500, 7, 3, 256, 128, None), (1, 300, 4, 64, 64, None)])
def test_grouped_products(dtype, M, E, top, width, ff, bn):
    from tah_b200.ops import cuda as K
    g = torch.Generator().manual_seed(M)
    rnd = lambda *s: torch.randn(*s, generator=g)
    L = K.ExpertLists(M, E, top, dtype, "cuda", bn=bn if dtype == BF16 else None)
    h = rnd(M, width).to(dtype)
    w_gu, w_down = (rnd(E, 2 * ff, width) / math.sqrt(width)).to(dtype), (rnd(E, width, ff) / math.sqrt(ff)).to(dtype)
    z = rnd(M, E).cuda()
    K.moe_route(z, L)
    e = lambda c: torch.full((L.rows, c), float("nan"), dtype=dtype, device="cuda")
    x = K.moe_gather(h.cuda(), L, e(width))                        # rows behind a list's end stay what they were
    act = K.moe_glu_linear(x, w_gu.cuda(), 0.9, L, e(ff))
    y = K.moe_linear(act, w_down.cuda(), L, e(width))
    slot, which, wt = L.slot.cpu().long(), L.expert.cpu().long(), L.weight.cpu().double()
    sel = list(range(M)) if M <= 200 else torch.randperm(M, generator=g)[:200].tolist()
    gu = torch.einsum("tjfk,tk->tjf", w_gu.double()[which[sel]], h.double()[sel]) * wt[sel].unsqueeze(-1)
    want = O.clamped_glu(gu[..., 0::2], gu[..., 1::2], 0.9)
    tol = 2e-5 if dtype == F32 else 1e-2
    got = act.cpu().double()[slot[sel]]
    assert float((got - want).abs().max()) < tol * float(want.abs().max())
    want = torch.einsum("tjwf,tjf->tjw", w_down.double()[which[sel]], got)
    assert float((y.cpu().double()[slot[sel]] - want).abs().max()) < tol * float(want.abs().max())
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
        got = run_portions(e, toks, [p for p in portions if p])
        assert H.close(got, want, dtype), portions[:4]
    assert e.kv.pages_in_use(0) == 0
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("place", [0, 1, 15, 16, 63, 64, 127, 130])
def test_a_far_key_is_found(tmp_path, dtype, place):
    """One key that every later query finds, through layers with keys of their own and one that shares them: in a prompt, in
    portions and in decoding, wherever the key lies."""
    cfg = H.CONFIGS["far"]()
    special, T = 7, 300
    sd = H.stand_out(cfg, O.random_model(cfg, 3), special, layers=(0, 1))
    d = os.path.join(str(tmp_path), "ckpt")
    H.write_checkpoint(d, cfg, sd)
    plain = [t if t != special else special + 1 for t in H.tokens(cfg, T, 3)]
    toks = list(plain)
    toks[place] = special
    want = O.forward(cfg, sd, toks)
    # it is this key that the last tokens answer to
    assert float(H.row_errors(O.forward(cfg, sd, plain)[-40:], want[-40:]).min()) > 0.3
    e = engine(d, dtype)
    for portions in ([T], [100, 100, 60] + [1] * 40, [place + 2, 2, T - place - 4]):
        assert H.close(run_portions(e, toks, portions), want, dtype), portions[:3]
    check_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_and_reused_pages_and_slots(tmp_path, dtype):
    """Requests of unequal lengths in shared steps, in a pool that only holds a few of them, rows handed on; every
    request's logits equal those of the request alone."""
    from tah_b200.engine import StepEntry
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
def test_large_steps(tmp_path, dtype):
    """More than a thousand tokens in a step (wide token tiles of the dense and the grouped products), unequal requests."""
    from tah_b200.engine import StepEntry
    cfg, sd, d = H.make(tmp_path, "tiles", seed=9)
    reqs = [H.tokens(cfg, n, 60 + n) for n in (1150, 200, 260, 131)]
    want = [O.forward(cfg, sd, t) for t in reqs]
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
    assert H.close(run_portions(e, toks[:90], [60, 30]), O.forward(cfg, sd, toks[:90]), F32)


def test_plain_attention_path_in_bf16(tmp_path, monkeypatch):
    """Other page sizes take the plain attention kernel, with the same routed experts."""
    cfg, sd, d = H.make(tmp_path, "mixed")
    toks = H.tokens(cfg, 100)
    e = engine(d, BF16, page_size=8)
    assert e.plain and H.close(run_portions(e, toks, [60, 1, 1, 38]), O.forward(cfg, sd, toks), BF16)
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
    e = make_engine(load_model(d, F32, "cuda"), max_rows=3)
    prompts = [H.tokens(cfg, n, 40 + i) for i, n in enumerate([30, 3, 71, 12, 1, 44, 25])]
    for _ in range(2):
        res, stats = e.serve([torch.tensor(p) for p in prompts], max_new_tokens=20, portion=16, check_every=4)
        assert stats["admitted"] == 7 and stats["mixed_steps"] > 7 and stats["tokens"] == 140
        assert all(_tokens_follow(cfg, sd, p, out, 1e-4) for p, out in zip(prompts, res))
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
        a, b, c = (e.generate(ids, None, max_new_tokens=12, do_sample=True, temperature=0.8, seed=s, **kw).tokens for s in (7, 7, 8))
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
