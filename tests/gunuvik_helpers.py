"""Small Gunuvik configurations, checkpoints of random weights, and comparison helpers for the tests."""
import json
import os

import torch
from safetensors.torch import save_file

from tests.oracle import gunuvik_oracle as O


def attn(heads=4, kv_heads=2, dim=40, vdim=24, window=19, keep=3, far=45, scale=0.21, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, bias_max=far)
    if window is not None or keep:
        m["mask"] = dict(size=window, keep_first=keep)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def memory(heads=3, dim=24, vdim=56, cap=9.0):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def layer(mixer, ff=88):
    return dict(type="mlstm" if "gate_cap" in mixer else "attention", mixer=mixer,
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def config(layers, vocab=203, width=136, eps=3e-5, scale=5.0, rel_rows=14):
    return dict(architecture="Gunuvik", vocab=vocab, width=width, embedding=dict(scale=scale), norm=dict(eps=eps),
                layers=layers, _rel_rows=rel_rows)


CONFIGS = {
    # grouped heads, unequal q/k and v sizes, a layer that reads another's keys under a window of its own
    "mixed": lambda: config([layer(attn()), layer(memory(), None), layer(attn(window=11, keep=0, far=30, kv_from=0)),
                             layer(attn(window=33, keep=5)), layer(memory(heads=2, dim=40, vdim=16, cap=4.0), 72)]),
    # recurrent layer first, attention without a window, attention without a feed-forward, sizes of 1 and odd sizes
    "odd": lambda: config([layer(memory(heads=1, dim=13, vdim=19)), layer(attn(heads=3, kv_heads=1, dim=18, vdim=33, window=None, keep=0), None),
                           layer(attn(heads=5, kv_heads=5, dim=7, vdim=9, window=1, keep=1, far=9), 45)],
                          vocab=151, width=77, rel_rows=6),
    # head sizes of whole 64-column tiles, window of one page and of several, sharing from the layer before last
    "tiles": lambda: config([layer(attn(heads=2, kv_heads=1, dim=64, vdim=128, window=16, keep=16, far=200)),
                             layer(attn(heads=4, kv_heads=2, dim=128, vdim=64, window=129, keep=1, far=64, scale=0.09)),
                             layer(attn(heads=4, kv_heads=2, dim=128, vdim=64, window=80, keep=40, far=100, scale=0.09, kv_from=1), None),
                             layer(memory(heads=2, dim=128, vdim=256, cap=15.0), 64)], vocab=320, width=192, rel_rows=20),
}


def write_checkpoint(path, cfg, sd):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump({k: v for k, v in cfg.items() if not k.startswith("_")}, fh)
    save_file({k: v.contiguous() for k, v in sd.items()}, os.path.join(path, "model.safetensors"))


def make(tmp_path, name_or_cfg, seed=0):
    """``(cfg, weights, checkpoint dir)`` of random weights."""
    cfg = CONFIGS[name_or_cfg]() if isinstance(name_or_cfg, str) else name_or_cfg
    sd = O.random_model(cfg, seed)
    d = os.path.join(str(tmp_path), f"ckpt{seed}")
    write_checkpoint(d, cfg, sd)
    return cfg, sd, d


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def row_errors(got, want):
    """Error of every row of logits: mean removed, root mean square, over the root mean square of the expected ones."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


TOL = {torch.float32: 2e-5, torch.bfloat16: 6e-2}


def close(got, want, dtype):
    """Every row within the rounding of ``dtype``.  A few tokens of a random model are ill-conditioned in 16 bits (the
    normaliser of a recurrent layer nearly cancels), so there one row in ten may be up to three times over."""
    e = row_errors(got, want)
    if dtype == torch.float32:
        return bool((e <= TOL[dtype]).all())
    return bool((e <= 3 * TOL[dtype]).all()) and int((e > TOL[dtype]).sum()) <= max(1, len(e) // 10)
