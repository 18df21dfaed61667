"""Plain, slow statement of the Gunuvik decoder: one function per mechanism, one sequence at a time, no cache.

Everything is written from the equations of the design in torch CPU tensors (double precision unless the caller passes
another dtype) and shares no code with the package.  ``cfg`` is the parsed ``config.json`` (a plain dict), ``sd`` a dict
of tensors under their on-disk names.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def distance_bucket(n: int, rows: int, far: int) -> int:
    """Row of the distance table for a key ``n`` positions back: exact below ``rows // 2``, then logarithmic up to
    ``far``.  The floor of the logarithm is taken in integers: the largest ``k`` with
    ``(far / half) ** k <= (n / half) ** (rows - half)``."""
    half = rows // 2
    if n < half:
        return n
    m = rows - half
    k = 0
    while k < m and far ** (k + 1) * half ** (m - k - 1) <= n ** m:
        k += 1
    return min(rows - 1, half + k)


def window_mask(T: int, size, keep_first: int):
    """``[T, T]`` bool: query i (row) sees key j (column)."""
    i = torch.arange(T).unsqueeze(1)
    j = torch.arange(T).unsqueeze(0)
    near = (i - j) < size if size is not None else torch.ones(T, T, dtype=torch.bool)
    return (j <= i) & (near | (j < keep_first))


def distance_bias(T: int, rel, far: int):
    """``[heads, T, T]`` learned bias of query i, key j <= i (zero above the diagonal)."""
    rows, heads = rel.shape
    by_distance = torch.stack([rel[distance_bucket(n, rows, far)] for n in range(T)])       # [T, heads]
    d = (torch.arange(T).unsqueeze(1) - torch.arange(T).unsqueeze(0)).clamp(min=0)
    return by_distance[d].permute(2, 0, 1)


def sink_softmax(scores, visible, sink):
    """Weights of ``scores [heads, T, T]`` where the denominator also contains ``exp(sink_h)``."""
    s = scores.masked_fill(~visible, -math.inf)
    top = torch.maximum(s.amax(-1, keepdim=True), sink.view(-1, 1, 1))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.view(-1, 1, 1) - top))


def attention_kv(h, mix, p, sd, eps):
    G, dk, dv = mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    k = (h @ sd[p + "k"].T + sd[p + "k.b"]).view(T, G, dk)
    v = (h @ sd[p + "v"].T + sd[p + "v.b"]).view(T, G, dv)
    return rms_norm(k, eps, sd[p + "k.norm"]), v


def attention(h, mix, p, sd, eps, kv):
    """Attention mixer of one layer; ``kv`` = normed keys ``[T, G, dk]`` and values of the layer that owns them."""
    H, G, dk = mix["heads"], mix["kv_heads"], mix["dim"]
    T = h.shape[0]
    k, v = kv
    q = rms_norm((h @ sd[p + "q"].T + sd[p + "q.b"]).view(T, H, dk), eps, sd[p + "q.norm"])
    owner = torch.arange(H) // (H // G)
    scores = torch.einsum("ihd,jhd->hij", q, k[:, owner]) * mix["scale"] + distance_bias(T, sd[p + "rel"], mix["bias_max"])
    mask = mix.get("mask") or {}
    w = sink_softmax(scores, window_mask(T, mask.get("size"), mask.get("keep_first", 0)), sd[p + "sink"])
    o = torch.einsum("hij,jhd->ihd", w, v[:, owner])
    o = o * torch.sigmoid(h @ sd[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, -1) @ sd[p + "o"].T


def mlstm_cell(q, k, v, log_i, log_f):
    """Token-by-token matrix memory of one head: ``q, k [T, dk]``, ``v [T, dv]``, gates ``[T]``; returns ``[T, dv]``."""
    T, dk = q.shape
    S = torch.zeros(dk, v.shape[1], dtype=q.dtype)
    n = torch.zeros(dk, dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(log_f[t] + m, log_i[t])
        keep, add = torch.exp(log_f[t] + m - m_new), torch.exp(log_i[t] - m_new)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = m_new
        out.append((S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def mlstm(h, mix, p, sd, eps):
    H, dk, dv, cap = mix["heads"], mix["dim"], mix["vdim"], mix["gate_cap"]
    T = h.shape[0]
    q = (h @ sd[p + "q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ sd[p + "k"].T).view(T, H, dk)
    v = (h @ sd[p + "v"].T).view(T, H, dv)
    log_i = cap * torch.tanh((h @ sd[p + "i"].T + sd[p + "i.b"]) / cap)
    log_f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ sd[p + "f"].T + sd[p + "f.b"]) / cap))
    o = torch.stack([mlstm_cell(q[:, a], k[:, a], v[:, a], log_i[:, a], log_f[:, a]) for a in range(H)], 1)
    o = rms_norm(o, eps).reshape(T, H * dv) * sd[p + "norm"] * torch.sigmoid(h @ sd[p + "g"].T)
    return o @ sd[p + "o"].T


def feed_forward(h, p, sd):
    return (silu(h @ sd[p + "gate"].T) * (h @ sd[p + "up"].T)) @ sd[p + "down"].T


def forward(cfg, sd, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the residual stream after every layer."""
    sd = {k: v.to(dtype) for k, v in sd.items()}
    eps = cfg["norm"]["eps"]
    x = sd["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    kv_of = {}
    for li, layer in enumerate(cfg["layers"]):
        p, mix = f"l{li}.", layer["mixer"]
        h = rms_norm(x, eps, sd[p + "norm1"])
        if layer["type"] == "attention":
            if "kv_from" in mix:
                kv = kv_of[mix["kv_from"]]
            else:
                kv = kv_of[li] = attention_kv(h, mix, p + "mix.", sd, eps)
            y = attention(h, mix, p + "mix.", sd, eps, kv)
        elif layer["type"] == "mlstm":
            y = mlstm(h, mix, p + "mix.", sd, eps)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(y, eps, sd[p + "norm1b"]) * sd[p + "ls1"]
        if layer["mlp"] is not None:
            y = feed_forward(rms_norm(x, eps, sd[p + "norm2"]), p + "mlp.", sd)
            x = x + rms_norm(y, eps, sd[p + "norm2b"]) * sd[p + "ls2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, eps, sd["final.norm"]) @ sd["head"].T


def random_model(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights under the on-disk names and shapes for ``cfg``.  Norm weights, biases, gates and layer scales are
    spread around non-trivial values so that leaving one of them out shows."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i: rnd(o, i) / math.sqrt(i)
    near1 = lambda *s: 1.0 + 0.2 * rnd(*s)
    sd = {"embed": rnd(V, W) * 0.1, "final.norm": near1(W), "head": lin(V, W)}
    for li, layer in enumerate(cfg["layers"]):
        p, mix = f"l{li}.", layer["mixer"]
        H, dk, dv = mix["heads"], mix["dim"], mix["vdim"]
        sd[p + "norm1"], sd[p + "norm1b"], sd[p + "ls1"] = near1(W), near1(W), 0.5 * near1(W)
        m = p + "mix."
        if layer["type"] == "attention":
            G = mix["kv_heads"]
            sd[m + "q"], sd[m + "q.b"], sd[m + "q.norm"] = lin(H * dk, W), 0.3 * rnd(H * dk), near1(dk)
            if "kv_from" not in mix:
                sd[m + "k"], sd[m + "k.b"], sd[m + "k.norm"] = lin(G * dk, W), 0.3 * rnd(G * dk), near1(dk)
                sd[m + "v"], sd[m + "v.b"] = lin(G * dv, W), 0.3 * rnd(G * dv)
            sd[m + "rel"] = 0.7 * rnd(cfg.get("_rel_rows", 16), H)
            sd[m + "sink"] = 0.5 * rnd(H) + 1.0
            sd[m + "g"], sd[m + "o"] = lin(H, W), lin(W, H * dv)
        else:
            sd[m + "q"], sd[m + "k"], sd[m + "v"] = lin(H * dk, W), lin(H * dk, W), lin(H * dv, W)
            sd[m + "q"] = 0.7 * sd[m + "q"] + 0.7 * sd[m + "k"]      # q . k of a token is positive: the normaliser rarely cancels
            sd[m + "g"], sd[m + "o"], sd[m + "norm"] = lin(H * dv, W), lin(W, H * dv), near1(H * dv)
            sd[m + "i"], sd[m + "i.b"] = 2 * lin(H, W), rnd(H)
            sd[m + "f"], sd[m + "f.b"] = 2 * lin(H, W), 3.0 + rnd(H)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            sd[p + "norm2"], sd[p + "norm2b"], sd[p + "ls2"] = near1(W), near1(W), 0.5 * near1(W)
            sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"] = lin(F, W), lin(F, W), lin(W, F)
    return {k: v.to(dtype) for k, v in sd.items()}
