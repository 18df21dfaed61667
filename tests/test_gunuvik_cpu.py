"""Gunuvik without a GPU: configuration, checkpoints, registry, cache geometry, and that the comparisons have teeth."""
import copy
import json
import os

import pytest
import torch

from tests import gunuvik_helpers as H
from tests.oracle import gunuvik_oracle as O


def test_config_round_trip_and_shapes(tmp_path):
    from tah_b200.models.gunuvik import GunuvikConfig, GunuvikForCausalLM
    for name in H.CONFIGS:
        cfg, sd, d = H.make(os.path.join(str(tmp_path), name), name)
        c = GunuvikConfig.from_pretrained(d)
        for l in c.layers:
            if l.mixer.kind == "attention":
                l.mixer.rel_rows = cfg["_rel_rows"]
        assert {k: tuple(v.shape) for k, v in sd.items()} == c.tensor_shapes()
        again = GunuvikConfig.from_dict(c.to_dict())
        for l in again.layers:
            if l.mixer.kind == "attention":
                l.mixer.rel_rows = cfg["_rel_rows"]
        assert again.layers == c.layers and again.hidden_size == c.hidden_size and again.rms_norm_eps == c.rms_norm_eps
        m = GunuvikForCausalLM.from_pretrained(d)
        assert all(torch.equal(m.tensor(k), v) for k, v in sd.items())
        out = os.path.join(str(tmp_path), name, "again")
        m.save_pretrained(out, max_shard_bytes=20000)                 # sharded on the way out, whole on the way in
        m2 = GunuvikForCausalLM.from_pretrained(out, dtype=torch.float32)
        assert all(torch.equal(m2.tensor(k), v.float()) for k, v in sd.items())


def test_wrong_checkpoints_and_configurations_are_refused(tmp_path):
    from tah_b200.models import load_model
    from tah_b200.models.gunuvik import GunuvikConfig
    cfg, sd, d = H.make(tmp_path, "mixed")
    for change in (lambda s: s.pop("l0.ls1"), lambda s: s.update({"l0.extra": torch.zeros(1)}),
                   lambda s: s.update({"l2.mix.k": torch.zeros(4, 4)}), lambda s: s.update({"head": torch.zeros(3, cfg["width"])})):
        bad = dict(sd)
        change(bad)
        H.write_checkpoint(str(tmp_path / "bad"), cfg, bad)
        with pytest.raises(ValueError):
            load_model(str(tmp_path / "bad"))
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mlp"), dict(kind="experts", ff=8)),
                        (("layers", 2, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), 2),
                        (("layers", 2, "mixer", "vdim"), 8), (("layers", 0, "mixer", "kv_heads"), 3)):
        c = copy.deepcopy(cfg)
        at = c
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            GunuvikConfig.from_dict(c)


def test_registry(tmp_path):
    from tah_b200.models import registry as R
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, "odd")
    assert R.family_of_config(R.read_config(d)).name == "gunuvik"
    assert R.family_of_config({"model_type": "qwen3"}).name == "qwen3-tah"
    assert R.family_of_config({"architectures": ["Qwen3ForCausalLM"]}).name == "qwen3-tah"
    with pytest.raises(ValueError):
        R.family_of_config({"architecture": "Unheard"})
    assert R.family_of_model(load_model(d)).name == "gunuvik"
    with pytest.raises(TypeError):
        R.family_of_model(object())
    with pytest.raises(RuntimeError):                            # no silent CPU path
        R.make_engine(load_model(d))
    from tests.helpers import tiny_tah
    assert R.family_of_model(tiny_tah()).name == "qwen3-tah"
    R.register_family(R.Family("probe", lambda c: c.get("architecture") == "Probe", lambda *a: "model", lambda m: m == "model",
                               lambda m, **k: ("engine", m)))
    try:
        assert R.make_engine(R.family_of_config({"architecture": "Probe"}).load("x", None, None)) == ("engine", "model")
    finally:
        R._FAMILIES[:] = [f for f in R._FAMILIES if f.name != "probe"]


@pytest.mark.parametrize("rows,far", [(6, 9), (14, 45), (32, 240), (16, 128), (9, 77), (20, 64), (2, 5), (64, 4096)])
def test_distance_table(rows, far):
    from tah_b200.engine.hybrid import distance_table
    rel = torch.randn(rows, 3)
    t = distance_table(rel, far)
    assert t.shape == (3, far + 1)
    for n in range(0, far + 1, max(1, far // 400)):
        assert torch.equal(t[:, n], rel[O.distance_bucket(n, rows, far)])
    for n in (far, far + 1, 10 * far):
        assert O.distance_bucket(n, rows, far) == rows - 1
    with pytest.raises(ValueError):
        distance_table(rel, rows // 2)


def test_weight_layout_pads_with_zeros(tmp_path):
    """Padded rows, columns and head dims of the kernel-ready weights are zero and the rest is where it belongs."""
    from tah_b200.engine.hybrid import AttentionLayer, HybridWeights
    from tah_b200.models import load_model
    cfg, sd, d = H.make(tmp_path, "odd")
    w = HybridWeights(load_model(d, torch.float32), torch.float32, plain=True)
    W = cfg["width"]
    for i, (b, l) in enumerate(zip(w.layers, cfg["layers"])):
        m, mix = b.mixer, l["mixer"]
        q = m.w_in[:mix["heads"] * m.dk].view(mix["heads"], m.dk, -1)
        assert torch.equal(q[:, :mix["dim"], :W], sd[f"l{i}.mix.q"].float().view(mix["heads"], mix["dim"], W))
        assert float(q[:, mix["dim"]:].abs().sum()) == 0 and float(q[:, :, W:].abs().sum()) == 0
        o = m.w_o[:W, :mix["heads"] * m.dv].view(W, mix["heads"], m.dv)
        assert torch.equal(o[:, :, :mix["vdim"]].reshape(W, -1), sd[f"l{i}.mix.o"].float())
        assert float(m.w_o.abs().sum()) == pytest.approx(float(sd[f"l{i}.mix.o"].float().abs().sum()), rel=1e-4)
        if isinstance(m, AttentionLayer):
            assert torch.equal(m.w_in[m.gate_col:m.gate_col + mix["heads"], :W], sd[f"l{i}.mix.g"].float())


def test_cache_geometry_per_layer():
    from tah_b200.engine.kv_cache import CacheGeometry, LayerKV, PagedKVCache, RecurrentState
    geo = CacheGeometry.per_layer([LayerKV(2, 40, 24), None, LayerKV(shared_with=0), LayerKV(1, 8, 16)])
    kv = PagedKVCache(geo, rows=3, max_tokens_per_row=100, n_depths=1, device="cpu", dtype=torch.float32, pool_tokens=96)
    assert kv.n_pages == [6] and kv.max_pages == [8]
    assert kv.layer_pool(0, 0).shape == (6, 2 * 16 * 64) and kv.layer_pool(0, 2) is kv.layer_pool(0, 0)
    assert kv.layer_pool(0, 1) is None and kv.layer_pool(0, 3).shape == (6, 16 * 24)
    assert kv.bytes() == 4 * 6 * 16 * (2 * 64 + 24)
    slots = kv.assign_rows(0, torch.tensor([1]), torch.tensor([40]))
    assert slots.unique().numel() == 40 and kv.pages_in_use(0) == 3
    with pytest.raises(RuntimeError):
        kv.assign_rows(0, torch.tensor([2]), torch.tensor([60]))
    assert kv.free_rows(torch.tensor([1])) == 3 and kv.pages_in_use(0) == 0
    for bad in ([LayerKV(shared_with=0)], [None, LayerKV(shared_with=0)], [LayerKV(1, 8, 8), LayerKV(shared_with=0), LayerKV(shared_with=1)]):
        with pytest.raises(ValueError):
            CacheGeometry.per_layer(bad)
    st = RecurrentState([None, [(2, 8, 16), (2, 8), (2,)]], rows=3, device="cpu")
    assert st.layers[0] is None and [tuple(t.shape) for t in st.layers[1]] == [(3, 2, 8, 16), (3, 2, 8), (3, 2)]
    assert st.bytes() == 4 * 3 * (2 * 8 * 16 + 2 * 8 + 2)


def test_guard_pages_of_per_layer_pools(monkeypatch):
    from tah_b200.engine.kv_cache import CacheGeometry, LayerKV, PagedKVCache
    monkeypatch.setenv("TAH_B200_CANARY", "2")
    for geo in (CacheGeometry.per_layer([LayerKV(1, 8, 16), None, LayerKV(2, 8, 8)]), CacheGeometry(2, 2, 64)):
        kv = PagedKVCache(geo, 2, 40, 1, device="cpu", dtype=torch.bfloat16)
        assert kv.check_guards()
        kv.layer_pool(0, 0)[kv.n_pages[0]].view(-1)[0] = 1.0
        assert not kv.check_guards()


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

    def mix(i, **kw):
        return lambda c: c["layers"][i]["mixer"].update(kw)

    def mask(i, **kw):
        return lambda c: c["layers"][i]["mixer"]["mask"].update(kw)

    def scale(name, f):
        return lambda s: s.update({name: s[name] * f})

    def swap(a, b):
        return lambda s: s.update({a: s[b], b: s[a]})

    cases = {
        "window": (mask(0, size=18), None), "window of the sharing layer": (mask(2, size=12), None),
        "kept tokens": (mask(3, keep_first=4), None), "no kept tokens": (mask(0, keep_first=0), None),
        "score scale": (mix(0, scale=0.2), None), "far end": (mix(3, bias_max=44), None),
        "gate cap": (mix(1, gate_cap=8.0), None), "eps": (lambda c: c["norm"].update(eps=1e-3), None),
        "embedding scale": (lambda c: c["embedding"].update(scale=4.0), None),
        "sink": (None, scale("l0.mix.sink", 0.0)), "distance bias": (None, scale("l2.mix.rel", 0.0)),
        "head gate": (None, scale("l3.mix.g", 0.0)), "key bias": (None, scale("l0.mix.k.b", 0.0)),
        "value bias": (None, scale("l0.mix.v.b", 0.0)), "layer scale": (None, scale("l1.ls1", 1.02)),
        "q and k norm": (None, swap("l0.mix.q.norm", "l0.mix.k.norm")), "output norm": (None, swap("l0.norm1", "l0.norm1b")),
        "feed-forward norm": (None, swap("l0.norm2", "l0.norm2b")), "i and f": (None, swap("l1.mix.i", "l1.mix.f")),
        "gate bias": (None, scale("l1.mix.f.b", 0.9)), "memory norm": (None, scale("l4.mix.norm", 0.9)),
        "memory gate": (None, scale("l4.mix.g", 0.0)), "gate and up": (None, swap("l0.mlp.gate", "l0.mlp.up")),
    }
    for name, (ec, es) in cases.items():
        err = float(H.row_errors(_changed(cfg, sd, toks, ec, es), base).max())
        assert err > 20 * H.TOL[torch.float32], (name, err)


def test_statement_of_the_running_maximum():
    """The cell against the unstabilised sums in double precision: the running maximum starts at zero, which shows in
    the normaliser of the first tokens when the input gates are small."""
    g = torch.Generator().manual_seed(0)
    T, dk, dv = 24, 5, 3
    q, k, v = (torch.randn(T, d, generator=g, dtype=torch.float64) for d in (dk, dk, dv))
    li, lf = torch.randn(T, generator=g, dtype=torch.float64) - 4.0, -torch.rand(T, generator=g, dtype=torch.float64)
    got = O.mlstm_cell(q, k, v, li, lf)
    m = 0.0
    for t in range(T):
        m = max(float(lf[t]) + m, float(li[t]))
        w = torch.stack([li[s] + lf[s + 1:t + 1].sum() for s in range(t + 1)]).exp()
        num = (w * (k[:t + 1] @ q[t])) @ v[:t + 1]
        den = (w * (k[:t + 1] @ q[t])).sum()
        e = torch.exp(torch.tensor(-m, dtype=torch.float64))
        want = num * e / (torch.maximum((den * e).abs(), e) + 1e-6)
        assert torch.allclose(got[t], want, rtol=1e-9, atol=1e-12)


def test_trace_replay_bookkeeping(tmp_path):
    """Rows are handed out at a request's first entry and given back at its end; logits go to one file per step."""
    from tah_b200.engine import trace

    class Fake:
        device = "cpu"

        def __init__(self):
            self.free, self.log = [1, 0], []

        def admit(self):
            return self.free.pop()

        def release(self, row):
            self.free.append(row)
            self.log.append(("release", row))

        def step(self, entries):
            self.log.append([(e.row, list(e.tokens), list(e.want)) for e in entries])
            return torch.arange(sum(len(e.want) for e in entries) * 4, dtype=torch.float32).view(-1, 4)

    from tah_b200.ops import cuda as K
    keep, K.check_status = K.check_status, lambda d=None: None
    try:
        eng, said = Fake(), []
        lines = [json.dumps(x) for x in (
            dict(step=0, entries=[dict(id="x", tokens=[1, 2], want=[1]), dict(id="y", tokens=[3], want=[0])], end=["x"]),
            dict(step=1, entries=[dict(id="z", tokens=[4], want=[])], end=["y", "z"]), dict(step=2, entries=[], end=[]))]
        trace.replay(lines, eng, str(tmp_path), said.append)
    finally:
        K.check_status = keep
    assert said == ["done 0", "done 1", "done 2"] and sorted(eng.free) == [0, 1]
    assert eng.log[0] == [(0, [1, 2], [1]), (1, [3], [0])] and eng.log[2] == [(0, [4], [])]
    assert os.path.getsize(tmp_path / "0.f32") == 32 and not os.path.exists(tmp_path / "1.f32")
