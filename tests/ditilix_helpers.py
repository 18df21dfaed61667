"""Small Ditilix configurations, checkpoints of random weights, and comparison helpers for the tests."""
import os

import torch

from tests.gunuvik_helpers import TOL, row_errors, tokens, write_checkpoint  # noqa: F401
from tests.oracle import ditilix_oracle as O


def attn(heads=4, kv_heads=2, dim=40, vdim=24, scale=0.21, softcap=3.0, temp=(0.4, 23), kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if softcap is not None:
        m["softcap"] = softcap
    if temp is not None:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=72, limit=0.9, shared=(40, 0.7)):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))
    if shared is not None:
        m["shared"] = dict(ff=shared[0], limit=shared[1])
    return m


def config(layers, vocab=203, width=132, groups=6, eps=3e-5, residual=0.8, logit=0.6):
    return dict(architecture="Ditilix", vocab=vocab, width=width, residual_mult=residual, logit_scale=logit,
                norm=dict(eps=eps, groups=groups), layers=[dict(type="attention", mixer=m, mlp=f) for m, f in layers])


CONFIGS = {
    # every kind of feed-forward, none at all, and layers that read another layer's keys with queries of their own
    "mixed": lambda: config([(attn(), dense()), (attn(scale=0.3, softcap=5.0), moe()), (attn(temp=(0.9, 7), kv_from=1), moe(ff=33)),
                             (attn(kv_from=0), None), (attn(heads=2, kv_heads=2, dim=24, vdim=40), moe(shared=None))]),
    # odd sizes, one key head for all, one per query head, many experts, no temperature, no cap, a mixture in front
    "odd": lambda: config([(attn(heads=3, kv_heads=1, dim=18, vdim=33, temp=None), moe(experts=37, top=3, ff=13, shared=(19, 1.3))),
                           (attn(heads=5, kv_heads=5, dim=7, vdim=9, scale=0.5, softcap=None, temp=(0.2, 1)), dense(45)),
                           (attn(heads=3, kv_heads=1, dim=18, vdim=33, softcap=1.5, kv_from=0), dense(51))],
                          vocab=151, width=77, groups=7),
    # head sizes of whole 64-column tiles, norm parts of whole 128-column blocks, one expert per token
    "tiles": lambda: config([(attn(heads=4, kv_heads=2, dim=128, vdim=64, scale=0.09, softcap=6.0), moe(experts=9, top=1, ff=64, shared=(64, 1.0))),
                             (attn(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.125, temp=(0.3, 64)), dense(320)),
                             (attn(heads=4, kv_heads=2, dim=128, vdim=64, scale=0.11, softcap=4.0, kv_from=0), moe(experts=9, top=1, ff=128))],
                            vocab=320, width=384, groups=3),
    # a high score cap, so that one key among hundreds can win
    "far": lambda: config([(attn(softcap=9.0), moe()), (attn(dim=64, vdim=64, scale=0.15, softcap=10.0), dense()),
                           (attn(softcap=8.0, kv_from=0), moe())], width=160, groups=4),
    # one norm group, a residual and a logit factor of one, all experts chosen
    "ones": lambda: config([(attn(heads=6, kv_heads=1, dim=72, vdim=16), moe(experts=2, top=2, ff=24, limit=2.0, shared=(8, 0.3))),
                            (attn(heads=1, kv_heads=1, dim=200, vdim=136, scale=0.1), dense(16))],
                           vocab=97, width=96, groups=1, residual=1.0, logit=1.0),
}


def make(tmp_path, name_or_cfg, seed=0):
    """``(cfg, weights, checkpoint dir)`` of random weights."""
    cfg = CONFIGS[name_or_cfg]() if isinstance(name_or_cfg, str) else name_or_cfg
    sd = O.random_model(cfg, seed)
    d = os.path.join(str(tmp_path), f"ckpt{seed}")
    write_checkpoint(d, cfg, sd)
    return cfg, sd, d


def close(got, want, dtype, tol=None):
    """Every row of logits within the rounding of ``dtype``."""
    return bool((row_errors(got, want) <= (tol or TOL[dtype])).all())


def stand_out(cfg, sd, token, layers=(0,)):
    """Make ``token`` a key that every query finds, in the given layers: all embeddings share a component that the query
    projections turn into a direction, and the key projections turn the token's own embedding into the same direction."""
    g = torch.Generator().manual_seed(99)
    W, E = cfg["width"], 0
    for l in cfg["layers"]:
        if l["mlp"] is not None and l["mlp"]["kind"] == "moe":
            E = l["mlp"]["router"]["experts"]
    sd = {k: v.double() for k, v in sd.items()}
    b, u = torch.randn(W, generator=g, dtype=torch.float64), torch.randn(W, generator=g, dtype=torch.float64)
    b[:E] = u[:E] = 0.0
    u -= (u @ b) / (b @ b) * b
    sd["embed"] = sd["embed"] + b
    sd["embed"][token, E:] = 3.0 * u[E:]
    for i in layers:
        m, p = cfg["layers"][i]["mixer"], f"l{i}.mix."
        c = torch.randn(m["dim"], generator=g, dtype=torch.float64)
        c *= 2.5 / c.norm() / (m["scale"] ** 0.5)
        sd[p + "q"] = 0.3 * sd[p + "q"] + torch.outer(c.repeat(m["heads"]), b) / (b @ b) * 1.5
        sd[p + "k"] = 0.3 * sd[p + "k"] + torch.outer(c.repeat(m["kv_heads"]), u) / (u @ u)
        sd[p + "o"] = 1.5 * sd[p + "o"]
    for k in sd:
        if k.endswith("router"):
            sd[k][:, E:] = 0.0                    # the shared component of the embeddings must not decide the routing
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}
