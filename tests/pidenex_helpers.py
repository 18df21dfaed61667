"""Small Pidenex configurations, checkpoints of random weights, and comparison helpers for the tests."""
import os

import torch

from tests import gunuvik_helpers
from tests.gunuvik_helpers import TOL, row_errors, tokens  # noqa: F401
from tests.oracle import pidenex_oracle as O


def attn(heads=4, kv_heads=2, dim=40, scale=0.2, size=19, pool=5):
    mask = dict(size=size) if pool is None else dict(size=size, pool=pool)
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=mask)


def latent(heads=3, dim=24, rot_dim=12, vdim=40, q_rank=56, kv_rank=72, scale=0.2, base=500.0, size=23):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                rot=dict(dims=rot_dim, base=base), mask=dict(size=size))


def both(heads=4, kv_heads=2, dim=24, scale=0.3, size=17, D=72, left=0.8, right=1.1):
    return dict(left=attn(heads, kv_heads, dim, scale, size, None), right=dict(width=D), left_scale=left, right_scale=right)


def layer(mixer, ff=88):
    kind = "parallel" if "left" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return dict(type=kind, mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


def config(layers, vocab=203, width=136, eps=3e-5, scale=0.7, loop=None):
    c = dict(architecture="Pidenex", vocab=vocab, width=width, embedding=dict(scale=scale), norm=dict(eps=eps),
             layers=[layer(*l) if isinstance(l, tuple) else layer(l) for l in layers])
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # every mixer, with and without feed-forward, a loop in the middle
    "mixed": lambda: config([attn(), (both(), 72), (latent(), None), attn(heads=6, kv_heads=1, dim=32, size=33, pool=7, scale=0.15)],
                            loop=(1, 3, 3)),
    # odd sizes, one key head for all and one per query head, blocks of one token, longer than a page and longer than the window,
    # a loop from the first layer
    "odd": lambda: config([attn(heads=3, kv_heads=3, dim=18, size=3, pool=1, scale=0.4), (both(heads=5, kv_heads=1, dim=7, size=9, D=13), 45),
                           (attn(heads=5, kv_heads=1, dim=7, size=11, pool=21, scale=0.5), None),
                           (latent(heads=5, dim=7, rot_dim=10, vdim=9, q_rank=21, kv_rank=19, scale=0.5, size=1), 51),
                           (both(heads=1, kv_heads=1, dim=33, size=1, D=2, left=1.0, right=0.3), None)],
                          vocab=151, width=77, loop=(0, 2, 2)),
    # sizes of whole 64-column tiles, windows of pages and of tiles, many heads, a loop to the last layer
    "tiles": lambda: config([attn(heads=4, kv_heads=2, dim=128, size=64, pool=16, scale=0.09), (both(heads=8, kv_heads=4, dim=64, size=129, D=192), 320),
                             (latent(heads=20, dim=64, rot_dim=64, vdim=64, q_rank=128, kv_rank=192, scale=0.09, size=80), 128),
                             (attn(heads=16, kv_heads=2, dim=64, size=16, pool=4, scale=0.12), None)],
                            vocab=320, width=384, eps=1e-6, loop=(2, 4, 2)),
    # heads beyond the narrow tiles, a loop of one layer, a loop of everything once, groups of three and of six heads
    "wide": lambda: config([(attn(heads=6, kv_heads=2, dim=200, size=50, pool=12, scale=0.07), 130), (both(heads=6, kv_heads=1, dim=136, size=70, D=320), None),
                            (latent(heads=18, dim=136, rot_dim=40, vdim=112, q_rank=64, kv_rank=136, scale=0.08, size=100), None)],
                           vocab=97, width=200, loop=(1, 2, 4)),
    # no loop, no feed-forward, windows that a prompt does not reach the end of
    "plain": lambda: config([(attn(size=500, pool=9), None), (both(size=400), None), (latent(size=300), None)], scale=1.0),
}


def write_checkpoint(path, cfg, sd):
    gunuvik_helpers.write_checkpoint(path, cfg, sd)


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


def stand_out(cfg, sd, token, strength=1.0):
    """Make ``token`` a key that every query finds wherever it is seen: all embeddings share a component that the queries turn into
    one direction, and the keys turn the token's own embedding into the same direction."""
    g = torch.Generator().manual_seed(99)
    rnd = lambda n: torch.randn(n, generator=g, dtype=torch.float64)
    W = cfg["width"]
    sd = {k: v.double() for k, v in sd.items()}
    b, u = rnd(W), rnd(W)
    b, u = b - b.mean(), u - u.mean()
    u -= (u @ b) / (b @ b) * b
    sd["embed"] = sd["embed"] + b / cfg["embedding"]["scale"]
    sd["embed"][token] = 3.0 * u / cfg["embedding"]["scale"]
    for i, l in enumerate(cfg["layers"]):
        mix, p = l["mixer"], f"l{i}.mix."
        sd[f"l{i}.norm1"] = torch.ones(W, dtype=torch.float64)
        if l["type"] == "latent_attention":
            H, d, r = mix["heads"], mix["dim"], mix["rot_dim"]
            c = rnd(d)
            c *= 1.2 * strength / c.norm() / mix["scale"] ** 0.5
            sd[p + "dq"][0], sd[p + "dkv"][0] = 8.0 * b / (b @ b) ** 0.5, 8.0 * u / (u @ u) ** 0.5
            sd[p + "uq"] *= 0.3
            sd[p + "uq"].view(H, d + r, -1)[:, :d, 0] = c
            sd[p + "uk"] *= 0.3
            sd[p + "uk"].view(H, d, -1)[:, :, 0] = c
            continue
        if l["type"] == "parallel":
            mix, p = mix["left"], p + "left."
        c = rnd(mix["dim"])
        c *= 3.0 * strength / c.norm() / mix["scale"] ** 0.5
        sd[p + "q"] = 0.3 * sd[p + "q"] + torch.outer(c.repeat(mix["heads"]), b) / (b @ b) * 1.5
        sd[p + "k"] = 0.3 * sd[p + "k"] + torch.outer(c.repeat(mix["kv_heads"]), u) / (u @ u)
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}


EDGES = {
    # one mixer each, the windows' far ends and the first blocks behind them inside the prompt
    "attention": lambda size, pool: config([(attn(dim=64, scale=0.1, size=size, pool=pool), None)]),
    "latent_attention": lambda size, pool: config([(latent(size=size, kv_rank=64), None)]),
    "parallel": lambda size, pool: config([(both(size=size, dim=64, scale=0.4, right=0.05), None)]),
}
STRENGTH = {"attention": 1.9, "latent_attention": 1.0, "parallel": 1.0}      # a block's mean holds only a part of the key
