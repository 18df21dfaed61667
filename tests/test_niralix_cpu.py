"""Niralix without a GPU: configuration, checkpoints, registry, weight layout, and that the comparisons have teeth."""
import copy
import json
import os

import pytest
import torch

from tests import niralix_helpers as H
from tests.oracle import niralix_oracle as O


def _public(d):
    with open(os.path.join(d, "config.json")) as fh:
        return json.load(fh)


def test_config_round_trip_and_shapes(tmp_path):
    from tah_b200.models.niralix import NiralixConfig, NiralixForCausalLM
    for name in H.CONFIGS:
        cfg, sd, d = H.make(os.path.join(str(tmp_path), name), name)
        m = NiralixForCausalLM.from_pretrained(d)
        c = m.config
        assert {k: tuple(v.shape) for k, v in sd.items()} == c.tensor_shapes()
        assert c.to_dict() == _public(d)
        again = NiralixConfig.from_dict(c.to_dict())
        assert [type(l.mixer) for l in again.layers] == [type(l.mixer) for l in c.layers] and [l.ff for l in again.layers] == [l.ff for l in c.layers]
        assert (again.streams, again.logit_scale, again.rms_norm_eps) == (cfg["streams"], cfg["logit_scale"], cfg["norm"]["eps"])
        assert all(torch.equal(m.tensor(k), v) for k, v in sd.items())
        out = os.path.join(str(tmp_path), name, "again")
        m.save_pretrained(out, max_shard_bytes=20000)
        m2 = NiralixForCausalLM.from_pretrained(out, dtype=torch.float32)
        assert all(torch.equal(m2.tensor(k), v.float()) for k, v in sd.items())


def test_wrong_checkpoints_and_configurations_are_refused(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models.niralix import NiralixConfig
    cfg, sd, d = H.make(tmp_path, "mixed")
    for change in (lambda s: s.pop("l1.mlp.e3.up"), lambda s: s.update({"l0.mix.vmix": torch.tensor(0.5)}), lambda s: s.pop("l2.hc1.mix"),
                   lambda s: s.update({"l1.mix.sink": torch.zeros(4)}), lambda s: s.update(head=s["embed"].clone())):
        bad = dict(sd)
        change(bad)
        H.write_checkpoint(str(tmp_path / "bad"), cfg, bad)
        with pytest.raises(ValueError):
            load_model(str(tmp_path / "bad"))
    for path, value in ((("layers", 0, "type"), "mlstm"), (("layers", 0, "mlp", "kind"), "swiglu"), (("layers", 0, "mixer", "kv_heads"), 3),
                        (("layers", 1, "mlp", "router", "top"), 6), (("layers", 2, "mixer", "rot", "dims"), 42), (("layers", 2, "mixer", "rot", "dims"), 7),
                        (("layers", 4, "mixer", "vdim"), 16), (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 3, "mixer", "tau"), 0.0)):
        c = copy.deepcopy(cfg)
        at = c
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            NiralixConfig.from_dict(c)


def test_registry(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models import registry as R
    from tah_b200.ops.build import CSRC, GROUPS
    cfg, sd, d = H.make(tmp_path, "odd")
    f = R.family_of_config(R.read_config(d))
    assert f.name == "niralix" and R.family_of_model(load_model(d)).name == "niralix"
    with pytest.raises(RuntimeError):                            # no silent CPU path
        R.make_engine(load_model(d))
    assert all(os.path.exists(os.path.join(CSRC, s + ".cu")) for s in GROUPS[f.sources])


def test_presets():
    from tah_b200.models import niralix_preset
    from tah_b200.models.niralix import NiralixConfig
    for name in ("niralix-1.7b", "niralix-moe", "niralix-tiny"):
        c = niralix_preset(name)
        assert NiralixConfig.from_dict(c.to_dict()).layers == c.layers
    with pytest.raises(KeyError):
        niralix_preset("niralix-unknown")


def test_random_init_reaches_every_tensor():
    from tah_b200.models import NiralixForCausalLM, niralix_preset
    m = NiralixForCausalLM(niralix_preset("niralix-tiny"), dtype=torch.float32).init_random(1)
    zero = [n for n in m.config.tensor_shapes() if float(m.tensor(n).abs().sum()) == 0]
    assert all(n.endswith((".norm1", ".norm2", "final.norm", ".q.b", ".k.b", ".v.b", ".o.b", ".sink")) for n in zero)


@pytest.mark.parametrize("rot", [dict(dims=24, base=1e6, scaling=dict(factor=8.0, original=1024, fast=20.0, slow=2.0)), dict(dims=2, base=5.0),
                                 dict(dims=64, base=1e4, scaling=dict(factor=2.0, original=16, fast=64.0, slow=32.0)),
                                 dict(dims=128, base=1e4, scaling=dict(factor=1.5, original=100000, fast=2.0, slow=0.001))])
def test_rotary_frequencies(rot):
    from tah_b200.models.niralix import _rotary
    got, want = _rotary(rot, False).frequencies(), O.rotary_frequencies(rot)
    assert torch.allclose(torch.tensor(got[0], dtype=torch.float64), torch.tensor(want[0], dtype=torch.float64), rtol=1e-14)
    assert got[1] == pytest.approx(want[1], rel=1e-14)


@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_weight_layout(tmp_path, name):
    """The stacked and padded matrices give the projections of the plain statement, and the absorbed and the expanded form of
    latent attention its scores and values."""
    from tah_b200.engine.hybrid_weights import GLALayer, HybridWeights, LatentLayer, MixtureLayer
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, name)
    w = HybridWeights(load_model(d, torch.float32), torch.float32, plain=False)
    W, S = cfg["width"], cfg["streams"]
    assert torch.allclose(w.final_norm[:W], (1 + sd["final.norm"].float()) * cfg["logit_scale"]) and float(w.final_norm[W:].abs().sum()) == 0
    assert torch.equal(w.head[:w.vocab, :W], sd["embed"].float()) and torch.equal(w.hc_in0, sd["l0.hc1.in"].float())
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g)
    h = torch.zeros(3, w.Wp)
    h[:, :W] = rnd(3, W)
    near = lambda a, b: torch.allclose(a, b, atol=2e-4, rtol=1e-4)
    reads = []                                                    # in-vectors in the order of the sublayers
    for i, l in enumerate(cfg["layers"]):
        reads += [sd[f"l{i}.hc{q}.in"].float() for q in ((1,) if l["mlp"] is None else (1, 2))]
    reads, k = reads[1:] + [torch.ones(S)], 0
    for i, (b, l) in enumerate(zip(w.layers, cfg["layers"])):
        p, m, mix, mlp = f"l{i}.", b.mixer, l["mixer"], l["mlp"]
        for q, hc in ((1, b.hc1), (2, b.hc2)):
            if q == 2 and mlp is None:
                assert hc is None and b.norm2 is None
                continue
            assert torch.equal(hc, torch.cat([sd[p + f"hc{q}.mix"].float().flatten(), sd[p + f"hc{q}.out"].float(), reads[k]]))
            k += 1
        lin = lambda n: h[:, :W] @ sd[p + "mix." + n].float().T
        proj, nh, dv = h @ m.w_in.T, mix["heads"], mix["vdim"]
        cut = lambda c, heads, dp, dd: proj[:, c:c + heads * dp].view(3, heads, dp)[..., :dd].reshape(3, -1)
        assert m.w_in.shape[0] % 64 == 0 and m.w_o.shape[1] % 64 == 0
        if isinstance(m, LatentLayer):
            R, r, dim = mix["kv_rank"], mix["rot_dim"], mix["dim"]
            assert near(proj[:, :mix["q_rank"]], lin("dq")) and near(cut(m.g_col, nh, m.dv, dv), lin("g"))
            assert near(torch.cat([proj[:, m.c_col:m.c_col + R], proj[:, m.r_col:m.r_col + r]], 1), lin("dkv"))
            assert float(proj[:, mix["q_rank"]:m.Qp].abs().sum()) == 0 and float(proj[:, m.c_col + R:m.r_col].abs().sum()) == 0
            cq, c, kr = rnd(3, mix["q_rank"]), rnd(3, R), rnd(3, r)
            q = torch.nn.functional.pad(cq, (0, m.Qp - cq.shape[1])) @ m.w_uq.T
            want_q = (cq @ sd[p + "mix.uq"].float().T).view(3, nh, dim + r)
            q = q[:, :nh * m.dk].view(3, nh, m.dk)
            assert near(q[..., :dim + r], want_q) and float(q[..., dim + r:].abs().sum()) == 0
            row = torch.zeros(3, m.w_abs.shape[1])
            row[:, :R], row[:, m.Rp:m.Rp + r] = c, kr
            key = torch.cat([(c @ sd[p + "mix.uk"].float().T).view(3, nh, dim), kr[:, None].expand(3, nh, r)], -1)
            val = (c @ sd[p + "mix.uv"].float().T).view(3, nh, dv)
            qa = torch.einsum("hlk,thk->thl", m.w_abs, torch.nn.functional.pad(q, (0, m.w_abs.shape[2] - m.dk)))
            assert near(torch.einsum("thl,sl->ths", qa, row), torch.einsum("thd,shd->ths", want_q, key))
            assert near(torch.einsum("hvr,tr->thv", m.w_uv, row[:, :m.Rp])[..., :dv], val)
            kv = row @ m.w_exp.T
            assert near(kv[:, :nh * m.dk].view(3, nh, m.dk)[..., :dim + r], key)
            assert near(kv[:, nh * m.dk:nh * (m.dk + m.dv)].view(3, nh, m.dv)[..., :dv], val)
            assert torch.allclose(m.sink_log2 * 0.6931471805599453, m.sink)
        elif isinstance(m, GLALayer):
            at = 0
            for n, dp, dd in (("q", m.dk, mix["dim"]), ("k", m.dk, mix["dim"]), ("v", m.dv, dv), ("g", m.dv, dv)):
                assert near(cut(at, nh, dp, dd), lin(n))
                at += nh * dp
            z = (h @ m.w_a1.T @ m.w_a2.T + m.b_a2).view(3, nh, m.dk)[..., :mix["dim"]].reshape(3, -1)
            assert near(z, lin("a1") @ sd[p + "mix.a2"].float().T + sd[p + "mix.a2.b"].float())
        else:
            G = mix["kv_heads"]
            pb = proj + m.b_in
            for n, c, heads, dp, dd in (("q", 0, nh, m.dk, mix["dim"]), ("k", m.kv_col, G, m.dk, mix["dim"]), ("v", m.kv_col + G * m.dk, G, m.dv, dv)):
                assert near(pb[:, c:c + heads * dp].view(3, heads, dp)[..., :dd].reshape(3, -1), lin(n) + sd[p + "mix." + n + ".b"].float())
            assert torch.equal(m.o_bias[:W], sd[p + "mix.o.b"].float())
            first = next((j for j, x in enumerate(cfg["layers"]) if x["mixer"].get("v_mix")), None)
            assert m.v_keeps == (i == first) and (m.v_lambda is not None) == (bool(mix["v_mix"]) and i != first)
        o = rnd(3, nh, dv)
        cat = torch.zeros(3, m.w_o.shape[1])
        cat[:, :nh * m.dv].view(3, nh, m.dv)[..., :dv] = o
        assert near((cat @ m.w_o.T)[:, :W], o.reshape(3, -1) @ sd[p + "mix.o"].float().T)
        if isinstance(b.ff, MixtureLayer):
            n = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                gu = (h @ b.ff.w_gu[e].T).view(3, -1, 2)
                assert near(gu[:, :n, 0], h[:, :W] @ sd[f"{p}mlp.e{e}.gate"].float().T) and near(gu[:, :n, 1], h[:, :W] @ sd[f"{p}mlp.e{e}.up"].float().T)
                assert torch.equal(b.ff.w_down[e, :W, :n], sd[f"{p}mlp.e{e}.down"].float())


@pytest.mark.parametrize("n,heads", [(1, 3), (16, 1), (17, 5), (64, 16), (300, 2)])
def test_head_lists(n, heads):
    from tah_b200.ops.cuda import HeadLists
    for dtype in (torch.bfloat16, torch.float32):
        L = HeadLists(n, heads, dtype, "cpu")
        assert L.npad >= n and L.npad % L.bn == 0 and L.rows == heads * L.npad == int(L.n_blocks) * L.bn
        assert L.blk_expert.tolist() == [r // L.npad for r in range(0, L.rows, L.bn)]


def test_latent_key_splits():
    from types import SimpleNamespace as NS
    from tah_b200.engine.hybrid import latent_splits
    m = lambda h, tc=True: NS(on_tensor_cores=tc, spec=NS(heads=h, window=None))
    assert latent_splits(m(16), 0) == 1 and latent_splits(m(16, False), 4) == 1 and latent_splits(m(16), 1) > 8
    assert all(1 <= latent_splits(m(h), n) <= 16 for h in (1, 16, 17, 128) for n in (1, 7, 64, 256, 1024))


def test_portions_fall_into_launches(monkeypatch):
    """Cache pages of the latent expansions: every portion's pages once, in order, launches within the limit."""
    from types import SimpleNamespace as NS
    from tah_b200.engine import hybrid
    from tah_b200.engine.hybrid_weights import LatentLayer
    monkeypatch.setattr(hybrid, "LATENT_PAGES", 10)
    table = torch.randperm(200, generator=torch.Generator().manual_seed(0)).view(5, 40).to(torch.int32)
    lens = torch.tensor([70, 16, 161, 0, 33], dtype=torch.int32)
    latent = LatentLayer.__new__(LatentLayer)
    latent.spec, latent.w_exp = NS(window=None), True
    eng = NS(device="cpu", page_size=16, plain=False, kv=NS(page_table=[table], len=[lens], max_pages=[40]), w=NS(parts=lambda: [latent]))
    eng._latent_plan = lambda *a: hybrid.HybridEngine._latent_plan(eng, *a)
    plan = hybrid._Plan()
    rows, counts, tiles = [4, 0, 2, 1], [2, 70, 150, 16], [1, 1, 2, 1]
    hybrid.HybridEngine._portion_plan(eng, plan, rows, counts, tiles, 3 + sum(counts))
    need = {4: 3, 0: 5, 2: 11, 1: 1}
    launches, where = plan.latent[None]
    assert [(a, b, len(s)) for a, b, s in launches] == [(0, 2, 8), (2, 4, 11), (4, 5, 1)] and plan.latent_pages == 11
    flat = torch.cat([table[r, :need[r]] for r in rows])
    assert torch.equal(torch.cat([s for _, _, s in launches]), flat)
    assert where[:, 0].tolist() == [0, 3, 0, 0] and where[2, :11].tolist() == list(range(11))
    assert plan.portion_of.tolist() == [0] * 3 + [0] * 2 + [1] * 70 + [2] * 150 + [3] * 16


def _changed(cfg, sd, toks, edit_cfg=None, edit_sd=None):
    c, s = copy.deepcopy(cfg), dict(sd)
    if edit_cfg:
        edit_cfg(c)
    if edit_sd:
        edit_sd(s)
    return O.forward(c, s, toks)


def test_plain_statement_is_sensitive_to_every_mechanism():
    """A mistake in any mechanism moves some logits of the test models by far more than the comparison tolerance."""
    cfg = H.CONFIGS["mixed"]()
    sd = O.random_model(cfg, 0)
    toks = H.tokens(cfg, 90)
    base = O.forward(cfg, sd, toks)
    mix = lambda i, **kw: lambda c: c["layers"][i]["mixer"].update(kw)
    rot = lambda i, **kw: lambda c: c["layers"][i]["mixer"]["rot"].update(kw)
    yarn = lambda i, **kw: lambda c: c["layers"][i]["mixer"]["rot"]["scaling"].update(kw)
    scale = lambda name, f: lambda s: s.update({name: s[name] * f})
    zero = lambda name: lambda s: s.update({name: torch.zeros_like(s[name])})
    swap = lambda a, b: lambda s: s.update({a: s[b], b: s[a]})
    turn = lambda name: lambda s: s.update({name: s[name].T.contiguous()})
    cases = {
        "score scale": (mix(2, scale=0.29), None), "latent scale": (mix(1, scale=0.26), None), "rotation base": (rot(2, base=950.0), None),
        "rotated dims": (rot(2, dims=18), None), "latent rotation": (rot(1, base=600.0), None), "scaling": (rot(2, scaling=None), None),
        "scaling factor": (yarn(2, factor=3.2), None), "fast": (yarn(2, fast=3.0), None), "slow": (yarn(2, slow=0.1), None),
        "original": (yarn(2, original=100), None), "mixed values": (mix(4, v_mix=False), None), "mixed from the first": (mix(0, v_mix=True), lambda s: s.update({"l0.mix.vmix": s["l2.mix.vmix"]})),
        "lambda": (None, scale("l4.mix.vmix", 1.1)), "query bias": (None, zero("l2.mix.q.b")), "key bias": (None, zero("l2.mix.k.b")),
        "value bias": (None, zero("l2.mix.v.b")), "output bias": (None, zero("l2.mix.o.b")), "sink": (None, zero("l1.mix.sink")),
        "latent gate": (None, scale("l1.mix.g", 0.9)), "query latent norm": (None, scale("l1.mix.dq.norm", 1.02)), "latent norm": (None, scale("l1.mix.dkv.norm", 1.02)),
        "tau": (mix(3, tau=6.3), None), "decay bias": (None, scale("l3.mix.a2.b", 0.9)), "decay features": (None, scale("l3.mix.a1", 0.9)),
        "gla norm": (None, scale("l3.mix.norm", 1.02)), "gla gate": (None, scale("l3.mix.g", 0.95)), "eps": (lambda c: c["norm"].update(eps=3e-3), None),
        "logit factor": (lambda c: c.update(logit_scale=0.71), None), "one expert less": (lambda c: c["layers"][1]["mlp"]["router"].update(top=1), None),
        "router": (None, scale("l1.mlp.router", 0.9)), "gate and up": (None, swap("l1.mlp.e0.gate", "l1.mlp.e0.up")),
        "experts": (None, swap("l1.mlp.e0.down", "l1.mlp.e1.down")), "norm weight": (None, scale("l3.norm1", 1.2)), "final norm": (None, scale("final.norm", 1.2)),
        "from and to": (None, turn("l2.hc1.mix")), "streams out": (None, scale("l3.hc2.out", 1.05)), "streams in": (None, swap("l3.hc1.in", "l3.hc2.in")),
    }
    for name, (ec, es) in cases.items():
        err = float(H.row_errors(_changed(cfg, sd, toks, ec, es), base).max())
        assert err > 20 * H.TOL[torch.float32], (name, err)


def test_layouts_of_the_rotation_differ():
    x = torch.randn(5, 2, 12, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    rot = dict(dims=8, base=50.0)
    a, b = O.rotate(x, range(5), rot, True), O.rotate(x, range(5), rot, False)
    assert float((a - b)[1:, :, :8].abs().max()) > 0.1 and torch.equal(a[..., 8:], x[..., 8:]) and torch.equal(a[0], x[0])
    assert torch.allclose((a * a).sum(-1), (x * x).sum(-1))                       # a rotation


def test_random_models_have_no_close_routing():
    for name in ("mixed", "tiles", "far"):
        cfg = H.CONFIGS[name]()
        assert O.router_margin(cfg, O.random_model(cfg, 0), H.tokens(cfg, 60)) > 0.1


def test_steep_models_cover_both_forms_of_the_chunk_product():
    """Running log decays of a 128-token chunk below the range of the factored product in some channels, inside in others."""
    cfg = H.CONFIGS["steep"]()
    sd, seen, keep = O.random_model(cfg, 0), [], O.gla_decay

    def watch(z, tau):
        a = keep(z, tau)
        seen.append(torch.log(a[:128]).sum(0).flatten())
        return a
    O.gla_decay = watch
    try:
        O.forward(cfg, sd, H.tokens(cfg, 130))
    finally:
        O.gla_decay = keep
    total = torch.cat(seen)
    assert int((total < -60).sum()) > 20 and int((total > -60).sum()) > 20 and float(total.min()) < -200 and float(total.max()) > -3
