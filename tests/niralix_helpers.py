"""Small Niralix configurations, checkpoints of random weights, and comparison helpers for the tests."""
import copy
import os

import torch

from tests import gunuvik_helpers
from tests.gunuvik_helpers import TOL, row_errors, tokens  # noqa: F401
from tests.oracle import niralix_oracle as O

YARN = dict(factor=3.0, original=64, fast=6.0, slow=0.5)


def attn(heads=4, kv_heads=2, dim=40, vdim=24, scale=0.21, rot=(20, 900.0), yarn=YARN, v_mix=True):
    r = dict(dims=rot[0], base=rot[1])
    if yarn is not None:
        r["scaling"] = dict(yarn)
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=r, v_mix=v_mix)


def latent(heads=3, dim=24, rot_dim=12, vdim=40, q_rank=56, kv_rank=72, scale=0.25, base=500.0):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                rot=dict(dims=rot_dim, base=base))


def gla(heads=3, dim=24, vdim=56, tau=6.0, bias=2.0):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau, _bias=bias)


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=72):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def layer(mixer, mlp):
    kind = "gla" if "tau" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return dict(type=kind, mixer=mixer, mlp=mlp)


def config(layers, vocab=203, width=136, eps=3e-5, streams=3, logit=0.7, rank=12):
    return dict(architecture="Niralix", vocab=vocab, width=width, streams=streams, logit_scale=logit, norm=dict(eps=eps),
                layers=[layer(m, f) for m, f in layers], _rank=rank)


CONFIGS = {
    # every mixer and feed-forward, none at all, values mixed from a layer that is not the first
    "mixed": lambda: config([(attn(v_mix=False), dense()), (latent(), moe()), (attn(scale=0.3), None), (gla(), moe(ff=33)),
                             (attn(rot=(12, 70.0), yarn=None), dense(45)), (latent(heads=5, kv_rank=40, rot_dim=6), None),
                             (gla(heads=2, dim=40, vdim=16, tau=3.0, bias=4.0), dense())]),
    # odd sizes, one stream, one key head for all and one per query head, many experts, decay features that need padding
    "odd": lambda: config([(latent(heads=5, dim=7, rot_dim=10, vdim=9, q_rank=21, kv_rank=19, scale=0.5), dense(51)),
                           (attn(heads=3, kv_heads=1, dim=18, vdim=33, rot=(6, 30.0)), moe(experts=37, top=3, ff=13)),
                           (gla(heads=1, dim=13, vdim=19, tau=1.0), None),
                           (attn(heads=5, kv_heads=1, dim=7, vdim=33, scale=0.5, rot=(2, 5.0), yarn=None), dense(45))],
                          vocab=151, width=77, streams=1, rank=5),
    # sizes of whole 64-column tiles, more heads than a decode block, whole heads rotated, one expert per token
    "tiles": lambda: config([(attn(heads=4, kv_heads=4, dim=128, vdim=64, scale=0.09, rot=(128, 1e4)), moe(experts=9, top=1, ff=64)),
                             (latent(heads=36, dim=64, rot_dim=64, vdim=64, q_rank=128, kv_rank=192, scale=0.09), dense(320)),
                             (gla(heads=2, dim=128, vdim=256, tau=16.0), moe(experts=9, top=1, ff=128)),
                             (latent(heads=20, dim=128, rot_dim=64, vdim=128, q_rank=64, kv_rank=512, scale=0.08), None)],
                            vocab=320, width=384, streams=2, rank=16),
    # decays from nearly none to nearly all of the state within a chunk
    "steep": lambda: config([(gla(tau=0.7, bias=0.0), dense()), (gla(heads=2, dim=32, vdim=64, tau=2.0, bias=-1.0), dense()),
                             (gla(heads=4, dim=72, vdim=24, tau=12.0, bias=4.0), dense())], streams=2),
    # a key that stands out can win among hundreds
    "far": lambda: config([(attn(), moe()), (latent(), dense()), (attn(dim=64, scale=0.15, rot=(24, 1e4)), moe())], width=160, streams=2),
    # a single head, all experts chosen, five streams
    "ones": lambda: config([(attn(heads=1, kv_heads=1, dim=200, vdim=136, scale=0.1, rot=(64, 1e3)), moe(experts=2, top=2, ff=24)),
                            (latent(heads=1, dim=136, rot_dim=2, vdim=8, q_rank=8, kv_rank=8), moe(experts=2, top=2, ff=16))],
                           vocab=97, width=96, streams=5, logit=1.0),
}


def write_checkpoint(path, cfg, sd):
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        l["mixer"].pop("_bias", None)
    gunuvik_helpers.write_checkpoint(path, c, sd)


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


def stand_out(cfg, sd, token, layers=(0, 1)):
    """Make ``token`` a key that every query finds at any distance, in the given attention and latent-attention layers: all
    embeddings share a component that the queries turn into a direction of the unrotated dims, and the keys turn the token's
    own embedding into the same direction."""
    g = torch.Generator().manual_seed(99)
    W, E = cfg["width"], 0
    for l in cfg["layers"]:
        if l["mlp"] is not None and l["mlp"]["kind"] == "moe":
            E = l["mlp"]["router"]["experts"]
    sd = {k: v.double() for k, v in sd.items()}
    rnd = lambda n: torch.randn(n, generator=g, dtype=torch.float64)
    b, u = rnd(W), rnd(W)
    b[:E] = u[:E] = 0.0
    u -= (u @ b) / (b @ b) * b
    sd["embed"] = sd["embed"] + b
    sd["embed"][token, E:] = 3.0 * u[E:]
    for i in layers:
        mix, p = cfg["layers"][i]["mixer"], f"l{i}.mix."
        if cfg["layers"][i]["type"] == "attention":
            c = rnd(mix["dim"])
            c[:mix["rot"]["dims"]] = 0.0
            c *= 3.0 / c.norm() / (mix["scale"] ** 0.5)
            sd[p + "q"] = 0.3 * sd[p + "q"] + torch.outer(c.repeat(mix["heads"]), b) / (b @ b) * 1.5
            sd[p + "k"] = 0.3 * sd[p + "k"] + torch.outer(c.repeat(mix["kv_heads"]), u) / (u @ u)
        else:
            H, d, r = mix["heads"], mix["dim"], mix["rot_dim"]
            c = rnd(d)
            c *= 1.2 / c.norm() / (mix["scale"] ** 0.5)
            sd[p + "dq"][0], sd[p + "dkv"][0] = 8.0 * b / (b @ b) ** 0.5, 8.0 * u / (u @ u) ** 0.5
            sd[p + "uq"] *= 0.3
            sd[p + "uq"].view(H, d + r, -1)[:, :d, 0] = c
            sd[p + "uk"] *= 0.3
            sd[p + "uk"].view(H, d, -1)[:, :, 0] = c
        sd[p + "o"] = 1.5 * sd[p + "o"]
    for k in sd:
        if k.endswith("router"):
            sd[k][:, E:] = 0.0                    # the shared component of the embeddings must not decide the routing
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}
