"""Pidenex without a GPU: configuration, checkpoints, registry, weight layout, cache geometry, and that the comparisons have teeth."""
import copy
import json
import os
from types import SimpleNamespace as NS

import pytest
import torch

from tests import pidenex_helpers as H
from tests.oracle import pidenex_oracle as O


def _public(d):
    with open(os.path.join(d, "config.json")) as fh:
        return json.load(fh)


def test_config_round_trip_and_shapes(tmp_path):
    from tah_b200.models.pidenex import PidenexConfig, PidenexForCausalLM
    for name in H.CONFIGS:
        cfg, sd, d = H.make(os.path.join(str(tmp_path), name), name)
        m = PidenexForCausalLM.from_pretrained(d)
        c = m.config
        assert {k: tuple(v.shape) for k, v in sd.items()} == c.tensor_shapes()
        assert c.to_dict() == _public(d)
        again = PidenexConfig.from_dict(c.to_dict())
        assert again.layers == c.layers and again.loop == c.loop
        assert (again.embedding_scale, again.rms_norm_eps) == (cfg["embedding"]["scale"], cfg["norm"]["eps"])
        assert c.layer_runs() == O.layer_order(cfg)
        assert all(torch.equal(m.tensor(k), v) for k, v in sd.items())
        out = os.path.join(str(tmp_path), name, "again")
        m.save_pretrained(out, max_shard_bytes=20000)
        m2 = PidenexForCausalLM.from_pretrained(out, dtype=torch.float32)
        assert all(torch.equal(m2.tensor(k), v.float()) for k, v in sd.items())


def test_layer_runs():
    from tah_b200.models.layered import LayeredConfig, LoopSpec
    runs = lambda n, *loop: LayeredConfig(1, 1, 1.0, 1e-6, [None] * n, loop=LoopSpec(*loop) if loop else None).layer_runs()
    assert runs(3) == [(0, None), (1, None), (2, None)]
    assert runs(4, 1, 3, 2) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert runs(2, 0, 1, 3) == [(0, 0), (0, 1), (0, 2), (1, None)] and runs(1, 0, 1, 1) == [(0, 0)]


def test_wrong_checkpoints_and_configurations_are_refused(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models.pidenex import PidenexConfig
    cfg, sd, d = H.make(tmp_path, "mixed")
    for change in (lambda s: s.pop("l1.mix.left.k.norm"), lambda s: s.update({"l0.mix.v": s["l0.mix.k"].clone()}), lambda s: s.pop("loop.step"),
                   lambda s: s.update({"l1.mix.right.z.b": torch.zeros(4)}), lambda s: s.update({"l3.norm1.b": s["l3.norm1"].clone()})):
        bad = dict(sd)
        change(bad)
        H.write_checkpoint(str(tmp_path / "bad"), cfg, bad)
        with pytest.raises(ValueError):
            load_model(str(tmp_path / "bad"))
    for path, value in ((("layers", 0, "type"), "mlstm"), (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mixer", "kv_heads"), 3),
                        (("layers", 0, "mixer", "vdim"), 24), (("layers", 1, "mixer", "left", "vdim"), 16), (("layers", 0, "mixer", "mask", "pool"), 0),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 2, "mixer", "mask", "size"), 0), (("layers", 2, "mixer", "rot", "dims"), 10),
                        (("loop", "stop"), 1), (("loop", "stop"), 5), (("loop", "times"), 0)):
        c = copy.deepcopy(cfg)
        at = c
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            PidenexConfig.from_dict(c)


def test_registry(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models import registry as R
    from tah_b200.ops.build import CSRC, GROUPS
    cfg, sd, d = H.make(tmp_path, "odd")
    f = R.family_of_config(R.read_config(d))
    assert f.name == "pidenex" and R.family_of_model(load_model(d)).name == "pidenex"
    with pytest.raises(RuntimeError):                            # no silent CPU path
        R.make_engine(load_model(d))
    assert all(os.path.exists(os.path.join(CSRC, s + ".cu")) for s in GROUPS[f.sources])


def test_presets_and_random_init():
    from tah_b200.models import PidenexForCausalLM, pidenex_preset
    from tah_b200.models.pidenex import PidenexConfig
    for name, runs in (("pidenex-1.7b", 28), ("pidenex-flat", 28), ("pidenex-tiny", 6)):
        c = pidenex_preset(name)
        assert PidenexConfig.from_dict(c.to_dict()).layers == c.layers and len(c.layer_runs()) == runs
    with pytest.raises(KeyError):
        pidenex_preset("pidenex-unknown")
    m = PidenexForCausalLM(pidenex_preset("pidenex-tiny"), dtype=torch.float32).init_random(1)
    assert [n for n in m.config.tensor_shapes() if float(m.tensor(n).abs().sum()) == 0] == ["l1.mix.right.x.b"]


@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_weight_layout(tmp_path, name):
    """The stacked and padded matrices give the projections of the plain statement; the queries carry the weights of both norms over
    all heads."""
    from tah_b200.engine.hybrid_weights import BranchesLayer, HybridWeights, LatentLayer
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, name)
    w = HybridWeights(load_model(d, torch.float32), torch.float32, plain=False)
    W = cfg["width"]
    f = lambda n: sd[n].float()
    assert torch.equal(w.final_norm[:W], f("final.norm")) and torch.equal(w.head[:w.vocab, :W], f("head"))
    for r, (i, t) in zip(w.runs, O.layer_order(cfg)):
        assert r.layer == i and r.embedding == bool(t) and (r.add is None) == (t is None)
        if t is not None:
            assert torch.equal(r.add[:W], f("loop.step")[t]) and float(r.add[W:].abs().sum()) == 0
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g)
    h = torch.zeros(3, w.Wp)
    h[:, :W] = rnd(3, W)
    near = lambda a, b: torch.allclose(a, b, atol=2e-4, rtol=1e-4)
    for i, (b, l) in enumerate(zip(w.layers, cfg["layers"])):
        p, m, mix, mlp = f"l{i}.", b.mixer, l["mixer"], l["mlp"]
        lin = lambda n: h[:, :W] @ f(p + "mix." + n).T
        proj = h @ m.w_in.T
        assert m.w_in.shape[0] % 64 == 0 and m.w_o.shape[1] % 64 == 0
        assert torch.equal(b.out1[:W], f(p + "norm1b")) and (b.norm2 is None) == (mlp is None)
        if isinstance(m, LatentLayer):
            R, r = mix["kv_rank"], mix["rot_dim"]
            assert near(proj[:, :mix["q_rank"]], lin("dq")) and m.g_col is None and m.sink is None
            assert near(torch.cat([proj[:, m.c_col:m.c_col + R], proj[:, m.r_col:m.r_col + r]], 1), lin("dkv"))
            a, dv = m, m.dv
        else:
            x, a, sub = ("left.", m.left, mix["left"]) if isinstance(m, BranchesLayer) else ("", m, mix)
            nh, G, dim, dv = sub["heads"], sub["kv_heads"], sub["dim"], a.dv
            cut = lambda c, heads: proj[:, c:c + heads * a.dk].view(3, heads, a.dk)[..., :dim].reshape(3, -1)
            assert a.nkv == G and near(cut(0, nh), lin(x + "q")) and near(cut(a.kv_col, G), lin(x + "k"))
            if x:
                n = a.norm_w.view(nh, a.dk)
                wq, wk = f(p + "mix.left.q.norm").view(nh, dim), f(p + "mix.left.k.norm").view(G, dim)
                assert torch.equal(n[:, :dim], torch.stack([wq[j] * wk[j // (nh // G)] for j in range(nh)])) and float(n[:, dim:].abs().sum()) == 0
                assert near(cut(a.wide_col, nh), lin("left.g")) and a.out_scale == mix["left_scale"]
                assert torch.allclose(a.slope * 0.6931471805599453, torch.tensor(O.slopes(nh)), rtol=1e-6)
                r, D = m.right, mix["right"]["width"]
                for k, n in enumerate(("z", "x", "g")):
                    at = r.in_col + k * r.d
                    assert near(proj[:, at:at + D], lin("right." + n)) and float(proj[:, at + D:at + r.d].abs().sum()) == 0
                assert torch.equal(r.zb[:D], f(p + "mix.right.z.b")) and torch.equal(r.xb[:D], f(p + "mix.right.x.b"))
                assert r.out_scale == mix["right_scale"] and all(c % 8 == 0 for c in (r.in_col, r.out_col, a.wide_col, a.kv_col))
        sub = mix.get("left", mix)
        o = rnd(3, sub["heads"], sub["vdim"])
        cat = torch.zeros(3, m.w_o.shape[1])
        cat[:, :sub["heads"] * dv].view(3, sub["heads"], dv)[..., :sub["vdim"]] = o
        want = o.reshape(3, -1) @ f(p + ("mix.left.o" if "left" in mix else "mix.o")).T
        if "left" in mix:
            s = rnd(3, mix["right"]["width"])
            cat[:, m.right.out_col:m.right.out_col + s.shape[1]] = s
            want = want + s @ f(p + "mix.right.o").T
        assert near((cat @ m.w_o.T)[:, :W], want)
        if mlp is not None:
            F, z = mlp["ff"], torch.linspace(-6, 6, 50, dtype=torch.float64)
            assert torch.equal(b.w_up[:F, :W], f(p + "mlp.up")) and torch.equal(b.w_down[:W, :F], f(p + "mlp.down"))
            got = torch.where(z > 0, b.ff.up * z * z, b.ff.low * (torch.expm1(z) - z)) + z / 2
            assert torch.allclose(got, O.xielu(z, sd[p + "mlp.act"].double()), atol=1e-12)


@pytest.mark.parametrize("page", [8, 16])
@pytest.mark.parametrize("block", [1, 2, 3, 5, 7, 8, 12, 16, 17, 40, 100])
def test_a_row_owns_the_page_of_a_block_that_is_complete(page, block):
    from tah_b200.engine.kv_cache import LayerKV
    S = LayerKV(2, 8, 0, block=block).pool_rows(page)
    assert S & (S - 1) == 0 and 1 <= S <= page and LayerKV(2, 8, 0).pool_rows(page) == 0
    for b in range(200):
        assert b // S <= (b * block + block - 1) // page


def test_cache_geometry(monkeypatch):
    from tah_b200.engine.kv_cache import CacheGeometry, LayerKV, PagedKVCache
    monkeypatch.setenv("TAH_B200_CANARY", "2")
    kv = PagedKVCache(CacheGeometry.per_layer([LayerKV(2, 24, 0, block=5), LayerKV(3, 8, 0, factor=True), None, LayerKV(1, 16, 8)]), 2, 100, 1,
                      device="cpu", pool_tokens=90)
    assert kv.n_pages == [6] and [None if t is None else tuple(t.shape) for t in kv.pool[0]] == [(8, 768), (8, 384), None, (8, 384)]
    assert [None if t is None else tuple(t.shape) for t in kv.pooled[0]] == [(8, 2 * 4 * 24), None, None, None]
    assert [None if t is None else tuple(t.shape) for t in kv.factors[0]] == [None, (8, 16), None, None]
    assert kv.check_guards() and kv.bytes() == 2 * 8 * (768 + 384 + 384 + 192) + 4 * 8 * 16
    kv.pooled[0][0][6, 0] = 1.0
    assert not kv.check_guards()


def test_portion_plan(monkeypatch):
    """Pooled rows and latent pages of the portions of a step: what is seen, and nothing of other rows."""
    from tah_b200.engine import hybrid
    from tah_b200.engine.hybrid_weights import AttentionLayer, LatentLayer
    att = lambda size, pool: AttentionLayer(NS(window=size, pool=pool, heads=1, kv_heads=1), 8, 8, 1, None, None, 8)
    lat = LatentLayer.__new__(LatentLayer)
    lat.spec, lat.w_exp = NS(window=40), True
    table = torch.randperm(200, generator=torch.Generator().manual_seed(0)).view(5, 40).to(torch.int32)
    lens = torch.tensor([70, 16, 361, 0, 133], dtype=torch.int32)
    eng = NS(device="cpu", page_size=16, plain=False, kv=NS(page_table=[table], len=[lens], max_pages=[40]),
             w=NS(parts=lambda: [att(30, 5), lat, att(30, 5), att(100, 16), att(9, None)]))
    eng._latent_plan = lambda *a: hybrid.HybridEngine._latent_plan(eng, *a)
    plan = hybrid._Plan()
    rows, counts, tiles = [4, 0, 2, 1], [2, 70, 150, 16], [1, 1, 2, 1]
    hybrid.HybridEngine._portion_plan(eng, plan, rows, counts, tiles, 3 + sum(counts))
    assert set(plan.pooled) == {(30, 5), (100, 16)}
    for (size, block), (src, base) in plan.pooled.items():
        S, at = {5: 4, 16: 1}[block], 0
        for e, (r, k) in enumerate(zip(rows, tiles)):
            seen = sum(b * block + block - 1 <= int(lens[r]) - 1 - size for b in range(400))
            assert base[sum(tiles[:e]):sum(tiles[:e]) + k].tolist() == [at] * k
            got = src[16 * at:16 * (at + (seen + 15) // 16)].tolist()
            assert got == [int(table[r, b // S]) * S + b % S if b < seen else -1 for b in range(len(got))]
            at += (seen + 15) // 16
        assert src.numel() == 16 * at
    assert plan.pooled_rows == max(s.numel() for s, _ in plan.pooled.values())
    launches, where = plan.latent[40]
    src = torch.cat([s for _, _, s in launches])
    for e, (r, c) in enumerate(zip(rows, counts)):
        lo = max(0, int(lens[r]) - c - 39)
        for j in range(lo // 64 * 4, (int(lens[r]) + 15) // 16):
            assert int(src[where[e, j]]) == int(table[r, j])
    assert src.numel() < sum((int(lens[r]) + 15) // 16 for r in rows) and plan.portion_of.tolist()[3:] == sum(([e] * c for e, c in enumerate(counts)), [])


def test_key_and_time_splits():
    from tah_b200.engine.hybrid import gru_splits, latent_splits
    gru = lambda d, n, longest: gru_splits(NS(d=d), n, longest)
    assert gru(2048, 1, 8192) > 4 and gru(2048, 64, 1024) == 1 and gru(72, 1, 200) == 1 and gru(8, 1, 100000) == 32
    m = lambda w: NS(on_tensor_cores=True, spec=NS(heads=16, window=w))
    assert latent_splits(m(40), 1) < latent_splits(m(None), 1)


def _changed(cfg, sd, toks, edit_cfg=None, edit_sd=None):
    c, s = copy.deepcopy(cfg), dict(sd)
    if edit_cfg:
        edit_cfg(c)
    if edit_sd:
        edit_sd(s)
    return O.forward(c, s, toks)


def test_plain_statement_is_sensitive_to_every_mechanism(monkeypatch):
    """A mistake in any mechanism moves some logits of the test models by far more than the comparison tolerance."""
    cfg = H.CONFIGS["mixed"]()
    sd = O.random_model(cfg, 0)
    toks = H.tokens(cfg, 90)
    base = O.forward(cfg, sd, toks)
    at = lambda i, *path: lambda c: c["layers"][i]["mixer"] if not path else c["layers"][i]["mixer"][path[0]]
    mix = lambda i, *path, **kw: lambda c: at(i, *path)(c).update(kw)
    scale = lambda name, f: lambda s: s.update({name: s[name] * f})
    zero = lambda name: lambda s: s.update({name: torch.zeros_like(s[name])})
    cases = {
        "score scale": (mix(0, scale=0.21), None), "window": (mix(0, "mask", size=20), None), "blocks": (mix(0, "mask", pool=4), None),
        "no blocks": (mix(3, "mask", pool=None), None), "latent scale": (mix(2, scale=0.21), None), "latent window": (mix(2, "mask", size=22), None),
        "rotation base": (mix(2, "rot", base=520.0), None), "latent norms": (None, scale("l2.mix.dkv.norm", 1.02)),
        "query latent norm": (None, scale("l2.mix.dq.norm", 1.05)), "left window": (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=18), None),
        "left score scale": (mix(1, "left", scale=0.31), None), "left scale": (mix(1, left_scale=0.82), None), "right scale": (mix(1, right_scale=1.12), None),
        "query norm": (None, scale("l1.mix.left.q.norm", 1.02)), "key norm": (None, scale("l1.mix.left.k.norm", 1.02)),
        "gate": (None, scale("l1.mix.left.g", 0.95)), "update bias": (None, scale("l1.mix.right.z.b", 0.95)), "input bias": (None, scale("l1.mix.right.x.b", 0.95)),
        "update gate": (None, scale("l1.mix.right.z", 0.98)), "right gate": (None, scale("l1.mix.right.g", 0.98)), "eps": (lambda c: c["norm"].update(eps=3e-3), None),
        "embedding scale": (lambda c: c["embedding"].update(scale=0.72), None), "one pass less": (lambda c: c["loop"].update(times=2), None),
        "pass vector": (None, zero("loop.step")), "activation": (None, scale("l1.mlp.act", 1.05)), "norm weight": (None, scale("l3.norm1", 1.2)),
        "output norm": (None, scale("l3.norm1b", 1.02)), "second output norm": (None, scale("l1.norm2b", 1.02)),
    }
    for name, (ec, es) in cases.items():
        err = float(H.row_errors(_changed(cfg, sd, toks, ec, es), base).max())
        assert err > 20 * H.TOL[torch.float32], (name, err)
    # mistakes that no number of the configuration expresses
    keep = {n: getattr(O, n) for n in ("slopes", "block_mask", "block_means", "layer_norm", "biased_attention", "min_gru_core", "layer_order")}

    def normed_values(h, mix, p, s, eps):
        T, G, d = h.shape[0], mix["kv_heads"], mix["dim"]
        q = O.rms_norm(h @ s[p + "q"].T, s[p + "q.norm"], eps).view(T, mix["heads"], d)
        k = O.rms_norm(h @ s[p + "k"].T, s[p + "k.norm"], eps).view(T, G, d)
        o = O.attention_core(q, k, k, mix["scale"], mix["mask"]["size"], None, O.slopes(mix["heads"]))
        return (o.reshape(T, -1) * torch.sigmoid(h @ s[p + "g"].T)) @ s[p + "o"].T
    faults = {
        "slopes": lambda heads: [2.0 ** (-8.0 * h / heads) for h in range(heads)],
        "block_mask": lambda T, size, pool: keep["block_mask"](T, size + 1, pool),
        "block_means": lambda k, pool: keep["block_means"](k, pool) * pool / (pool + 1),
        "layer_norm": lambda x, w, eps: O.rms_norm(x, w, eps),
        "biased_attention": normed_values,
        "min_gru_core": lambda z, u, state=None: keep["min_gru_core"](z, u.clamp(min=-0.5), state),
        "layer_order": lambda c: [(i, t if t else None) for i, t in keep["layer_order"](c)],
    }
    for name, fault in faults.items():
        monkeypatch.setattr(O, name, fault)
        assert float(H.row_errors(O.forward(cfg, sd, toks), base).max()) > 20 * H.TOL[torch.float32], name
        monkeypatch.setattr(O, name, keep[name])


@pytest.mark.parametrize("kind", list(H.EDGES))
def test_a_key_that_stands_out_shows_every_edge(kind):
    """The models of the edge tests: the key changes every logit of the tokens that see it, and a window or a block rule that is one
    token off changes those at the edge by more than 16-bit rounding."""
    size, pool, place, T, special = 24, 5, 41, 110, 7
    cfg = H.EDGES[kind](size, pool)
    sd = H.stand_out(cfg, O.random_model(cfg, 3), special, H.STRENGTH[kind])
    plain = [t if t != special else special + 1 for t in H.tokens(cfg, T, 3)]
    toks = list(plain)
    toks[place] = special
    err = lambda a, b: H.row_errors(a, b)
    full, without = O.forward(cfg, sd, toks), O.forward(cfg, sd, plain)
    seen = [i for i in range(place + 1, T) if i - place < size or kind == "attention" and place // pool * pool + pool - 1 <= i - size]
    e = err(without, full)
    assert float(e[seen].min()) > 0.15, e[seen].min()
    if kind != "parallel":
        assert float(e[[i for i in range(T) if i < place or i > place and i not in seen]].max()) < 1e-12
    for d in (-1, 1):
        c = H.EDGES[kind](size + d, pool)
        at = place + size - 1 if d < 0 else place + size
        assert float(err(O.forward(c, sd, toks), full)[at]) > 0.15
    if kind == "attention":
        first = place // pool * pool + pool - 1 + size                      # the first query that sees the key's block
        assert first > place + size and first in seen and first - 1 not in seen
