"""Ditilix without a GPU: configuration, checkpoints, registry, weight layout, and that the comparisons have teeth."""
import copy
import os

import pytest
import torch

from tests import ditilix_helpers as H
from tests.oracle import ditilix_oracle as O


def test_config_round_trip_and_shapes(tmp_path):
    from tah_b200.models.ditilix import DitilixConfig, DitilixForCausalLM
    for name in H.CONFIGS:
        cfg, sd, d = H.make(os.path.join(str(tmp_path), name), name)
        c = DitilixConfig.from_pretrained(d)
        assert {k: tuple(v.shape) for k, v in sd.items()} == c.tensor_shapes()
        again = DitilixConfig.from_dict(c.to_dict())
        assert c.to_dict() == cfg and again.layers == c.layers
        assert (again.norm_groups, again.residual_mult, again.logit_scale) == (cfg["norm"]["groups"], cfg["residual_mult"], cfg["logit_scale"])
        m = DitilixForCausalLM.from_pretrained(d)
        assert all(torch.equal(m.tensor(k), v) for k, v in sd.items())
        out = os.path.join(str(tmp_path), name, "again")
        m.save_pretrained(out, max_shard_bytes=20000)
        m2 = DitilixForCausalLM.from_pretrained(out, dtype=torch.float32)
        assert all(torch.equal(m2.tensor(k), v.float()) for k, v in sd.items())


def test_wrong_checkpoints_and_configurations_are_refused(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models.ditilix import DitilixConfig
    cfg, sd, d = H.make(tmp_path, "mixed")
    for change in (lambda s: s.pop("l1.mlp.e3.up"), lambda s: s.update({"l3.mix.k": s["l0.mix.k"].clone()}),
                   lambda s: s.update({"l0.mlp.act": torch.zeros(3)}), lambda s: s.pop("l1.mlp.shared.sg")):
        bad = dict(sd)
        change(bad)
        H.write_checkpoint(str(tmp_path / "bad"), cfg, bad)
        with pytest.raises(ValueError):
            load_model(str(tmp_path / "bad"))
    for path, value in ((("layers", 0, "type"), "mlstm"), (("layers", 0, "mlp", "kind"), "swiglu"), (("layers", 2, "mixer", "kv_from"), 2),
                        (("layers", 3, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "vdim"), 8), (("layers", 0, "mixer", "kv_heads"), 3),
                        (("layers", 1, "mlp", "router", "top"), 6), (("norm", "groups"), 5), (("layers", 0, "mixer", "softcap"), 0.0),
                        (("layers", 0, "mixer", "q_temp", "every"), 0)):
        c = copy.deepcopy(cfg)
        at = c
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            DitilixConfig.from_dict(c)


def test_registry(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models import registry as R
    from tah_b200.ops.build import CSRC, GROUPS
    cfg, sd, d = H.make(tmp_path, "odd")
    f = R.family_of_config(R.read_config(d))
    assert f.name == "ditilix" and R.family_of_model(load_model(d)).name == "ditilix"
    with pytest.raises(RuntimeError):                            # no silent CPU path
        R.make_engine(load_model(d))
    for name in ("ditilix", "gunuvik"):
        fam = next(x for x in R._FAMILIES if x.name == name)
        assert all(os.path.exists(os.path.join(CSRC, s + ".cu")) for s in GROUPS[fam.sources])


def test_presets():
    from tah_b200.models import ditilix_preset
    from tah_b200.models.ditilix import DitilixConfig
    for name in ("ditilix-1.7b", "ditilix-moe", "ditilix-tiny"):
        c = ditilix_preset(name)
        assert DitilixConfig.from_dict(c.to_dict()).layers == c.layers
    with pytest.raises(KeyError):
        ditilix_preset("ditilix-unknown")


@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_weight_layout(tmp_path, name):
    """The stacked, padded and interleaved matrices give the projections and sublayer sums of the plain statement."""
    from tah_b200.engine.hybrid_weights import HybridWeights, MixtureLayer, PolyNormLayer
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, name)
    w = HybridWeights(load_model(d, torch.float32), torch.float32, plain=True)
    W = cfg["width"]
    assert torch.allclose(w.final_norm[:W], sd["final.norm"].float() * cfg["logit_scale"]) and float(w.final_norm[W:].abs().sum()) == 0
    g = torch.Generator().manual_seed(0)
    h = torch.zeros(3, w.Wp)
    h[:, :W] = torch.randn(3, W, generator=g)
    for i, (b, l) in enumerate(zip(w.layers, cfg["layers"])):
        p, m, mix, mlp = f"l{i}.", b.mixer, l["mixer"], l["mlp"]
        lin = lambda n: h[:, :W] @ sd[p + n].float().T
        proj = h @ m.w_in.T
        assert m.w_in.shape[0] % 64 == 0 and m.w_o.shape[1] % 64 == 0
        q = proj[:, :mix["heads"] * m.dk].view(3, mix["heads"], m.dk)
        assert torch.allclose(q[..., :mix["dim"]].reshape(3, -1), lin("mix.q"), atol=1e-4) and float(q[..., mix["dim"]:].abs().sum()) == 0
        if m.nkv:
            v = proj[:, m.kv_col + m.nkv * m.dk:][:, :m.nkv * m.dv].view(3, m.nkv, m.dv)
            assert torch.allclose(v[..., :mix["vdim"]].reshape(3, -1), lin("mix.v"), atol=1e-4)
        cat, want = torch.full((3, m.w_o.shape[1]), 1.5), torch.zeros(3, W)     # padding columns must not matter
        o = torch.randn(3, mix["heads"], mix["vdim"], generator=g)
        cat[:, :mix["heads"] * m.dv].view(3, mix["heads"], m.dv)[..., :mix["vdim"]] = o
        want = o.reshape(3, -1) @ sd[p + "mix.o"].float().T
        if isinstance(b.ff, PolyNormLayer):
            f, n = b.ff, mlp["ff"]
            assert torch.allclose(proj[:, f.in_col:f.in_col + n], lin("mlp.up"), atol=1e-4)
            a = torch.randn(3, n, generator=g)
            cat[:, f.out_col:f.out_col + n] = a
            want = want + a @ sd[p + "mlp.down"].float().T
        if isinstance(b.ff, MixtureLayer):
            f, n = b.ff, mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                gu = (h @ f.w_gu[e].T).view(3, -1, 2)
                assert torch.allclose(gu[:, :n, 0], lin(f"mlp.e{e}.gate"), atol=1e-4) and torch.allclose(gu[:, :n, 1], lin(f"mlp.e{e}.up"), atol=1e-4)
                assert float(gu[:, n:].abs().sum()) == 0
                assert torch.equal(f.w_down[e, :W, :n], sd[f"{p}mlp.e{e}.down"].float())
            assert torch.allclose((h @ f.w_router.T)[:, :mlp["router"]["experts"]], lin("mlp.router"), atol=1e-4)
            if f.shared is not None:
                s, n = f.shared, mlp["shared"]["ff"]
                gu = proj[:, s.in_col:s.in_col + 2 * s.cols].view(3, -1, 2)
                assert torch.allclose(gu[:, :n, 0], lin("mlp.shared.gate"), atol=1e-4)
                assert torch.allclose((h @ f.w_router.T)[:, -1:], lin("mlp.shared.sg"), atol=1e-4)
                a = torch.randn(3, n, generator=g)
                cat[:, s.out_col:s.out_col + n] = a
                want = want + a @ sd[p + "mlp.shared.down"].float().T
        got = cat @ m.w_o.T
        assert torch.allclose(got[:, :W], want, atol=1e-3) and float(got[:, W:].abs().sum()) == 0


def test_engine_refuses_combinations_without_kernels(tmp_path):
    from tah_b200.engine.hybrid_weights import HybridWeights
    from tah_b200.models import load_model
    from tah_b200.models.layered import SwiGLUSpec
    m = load_model(H.make(tmp_path, "mixed")[2], torch.float32)
    m.config.layers[0].ff = SwiGLUSpec(88)
    with pytest.raises(NotImplementedError):
        HybridWeights(m, torch.float32, plain=True)


@pytest.mark.parametrize("width", [6, 77, 132, 2048])
def test_sinusoid_frequencies(width):
    from tah_b200.ops.cuda import sinusoid_frequencies
    f = sinusoid_frequencies(width)
    exact = torch.tensor([10000.0 ** (-2.0 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64)
    assert f.shape == (2, (width + 1) // 2) and float(((f[0].double() + f[1].double()) / exact - 1).abs().max()) < 1e-13


@pytest.mark.parametrize("bn", [16, 64, 256])
def test_expert_lists_hold_every_distribution(bn):
    """The block capacity covers the worst distribution of tokens over experts."""
    from tah_b200.ops.cuda import ExpertLists
    g = torch.Generator().manual_seed(0)
    for M, E, top in ((1, 8, 1), (5, 3, 2), (300, 7, 3), (40, 64, 8), (1000, 5, 1), (17, 1000, 4)):
        L = ExpertLists(M, E, top, torch.bfloat16, "cpu", bn=bn)
        n = M * top
        spread = [n - min(E, n) + 1] + [1] * (min(E, n) - 1)             # one expert takes nearly all, the others one each
        cases = [[n], spread]
        for _ in range(20):
            cases.append(torch.bincount(torch.randint(0, E, (n,), generator=g), minlength=E).tolist())
        assert all(sum((c + bn - 1) // bn for c in case) <= L.max_blocks for case in cases)


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
    mlp = lambda i, k, **kw: lambda c: c["layers"][i]["mlp"][k].update(kw)
    scale = lambda name, f: lambda s: s.update({name: s[name] * f})
    swap = lambda a, b: lambda s: s.update({a: s[b], b: s[a]})

    def act(k):
        def f(s):
            a = s["l0.mlp.act"].clone()
            a[k] *= 1.1
            s["l0.mlp.act"] = a
        return f

    cases = {
        "score scale": (mix(1, scale=0.29), None), "cap": (mix(0, softcap=3.3), None), "no cap": (mix(1, softcap=None), None),
        "temperature": (mix(0, q_temp=dict(coef=0.38, every=23)), None), "temperature step": (mix(0, q_temp=dict(coef=0.4, every=24)), None),
        "shared keys": (mix(2, kv_from=0), None), "eps": (lambda c: c["norm"].update(eps=3e-3), None),
        "norm groups": (lambda c: c["norm"].update(groups=3), None), "residual factor": (lambda c: c.update(residual_mult=0.81), None),
        "logit factor": (lambda c: c.update(logit_scale=0.61), None), "expert limit": (mlp(1, "expert", limit=0.95), None),
        "shared limit": (mlp(1, "shared", limit=0.75), None), "one expert less": (mlp(1, "router", top=1), None),
        "router": (None, scale("l1.mlp.router", 0.9)), "shared gate": (None, scale("l1.mlp.shared.sg", 0.5)),
        "gate and up": (None, swap("l1.mlp.e0.gate", "l1.mlp.e0.up")), "experts": (None, swap("l1.mlp.e0.down", "l1.mlp.e1.down")),
        "norm weight": (None, scale("l3.norm1", 1.02)), "final norm": (None, scale("final.norm", 1.02)),
        **{f"activation {k}": (None, act(k)) for k in range(4)},
    }
    for name, (ec, es) in cases.items():
        err = float(H.row_errors(_changed(cfg, sd, toks, ec, es), base).max())
        assert err > 20 * H.TOL[torch.float32], (name, err)


def test_random_models_have_no_close_routing():
    for name in ("mixed", "tiles", "far"):
        cfg = H.CONFIGS[name]()
        assert O.router_margin(cfg, O.random_model(cfg, 0), H.tokens(cfg, 60)) > 0.1


def test_weight_on_the_input_is_not_a_weight_on_the_output():
    """The router's score inside the expert (through its clamps and gates) differs from the score behind it."""
    g = torch.Generator().manual_seed(0)
    h = torch.randn(4, 8, generator=g, dtype=torch.float64)
    sd = {k: torch.randn(6, 8, generator=g, dtype=torch.float64) for k in ("e0.gate", "e0.up")}
    sd["e0.down"] = torch.randn(8, 6, generator=g, dtype=torch.float64)
    sd["router"] = torch.randn(1, 8, generator=g, dtype=torch.float64)
    got = O.mixture(h, dict(router=dict(top=1), expert=dict(limit=0.8)), "", sd)
    w = torch.sigmoid(h @ sd["router"].T)
    assert torch.allclose(got, O.expert(w * h, "e0.", sd, 0.8))
    assert float((got - w * O.expert(h, "e0.", sd, 0.8)).abs().max()) > 0.1
