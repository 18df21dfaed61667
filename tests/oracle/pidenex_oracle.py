"""Plain, slow statement of the Pidenex decoder: one function per mechanism, one sequence at a time, no cache.

Everything is written from the equations of the design in torch CPU tensors (double precision unless the caller passes
another dtype) and shares no code with the package.  ``cfg`` is the parsed ``config.json`` (a plain dict), ``sd`` a dict
of tensors under their on-disk names.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------
# norms, activation
# ------------------------------------------------------------------------------------
def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def softplus(t):
    return torch.logaddexp(t, torch.zeros_like(t))


def xielu(z, pq):
    up, low = softplus(pq[0]), 0.5 + softplus(pq[1])
    return torch.where(z > 0, up * z * z, low * (torch.exp(z.clamp(max=0.0)) - 1.0 - z)) + 0.5 * z


def dense(h, p, sd):
    return xielu(h @ sd[p + "up"].T, sd[p + "act"]) @ sd[p + "down"].T


# ------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------
def rotate(x, positions, dims, base):
    """Rotate the first ``dims`` entries of the last axis of ``x [T, heads, d]`` in pairs ``(2 i, 2 i + 1)``."""
    out = x.clone()
    for i in range(dims // 2):
        ang = [p * base ** (-2.0 * i / dims) for p in positions]
        c = torch.tensor([[math.cos(a)] for a in ang], dtype=torch.float64).to(x.dtype)
        s = torch.tensor([[math.sin(a)] for a in ang], dtype=torch.float64).to(x.dtype)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_mask(T, size):
    """``[T, T]`` bool: query (row) sees key (column); ``size`` None: every earlier key."""
    d = torch.arange(T).view(-1, 1) - torch.arange(T)
    return (d >= 0) & (d < (T if size is None else size))


def block_mask(T, size, pool):
    """``[T, T // pool]`` bool: query sees the mean of a block, which lies wholly in front of its window."""
    last = torch.arange(T // pool) * pool + pool - 1
    return last <= torch.arange(T).view(-1, 1) - size


def block_means(k, pool):
    """Means of the whole blocks of ``pool`` rows of ``k [T, G, d]``."""
    n = k.shape[0] // pool
    return k[:n * pool].view(n, pool, *k.shape[1:]).mean(1)


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def attention_core(q, k, v, scale, size=None, pool=None, slope=None):
    """Softmax attention of ``q [T, H, dk]`` over ``k [T, G, dk]``, ``v [T, G, dv]`` in a window, with block means beside it;
    ``slope [H]``: what a head's scores lose per token of distance."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    keys, vals, see = k, v, window_mask(T, size)
    dist = (torch.arange(T).view(-1, 1) - torch.arange(T)).to(q.dtype)
    if pool is not None:
        keys, vals = torch.cat([k, block_means(k, pool)]), torch.cat([v, block_means(v, pool)])
        see = torch.cat([see, block_mask(T, size, pool)], 1)
        dist = torch.nn.functional.pad(dist, (0, T // pool))
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for a in range(H):
        b = a // (H // G)
        s = q[:, a] @ keys[:, b].T * scale
        if slope is not None:
            s = s - slope[a] * dist
        out[:, a] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ vals[:, b]
    return out


def _mask(mix):
    m = mix.get("mask") or {}
    return m.get("size"), m.get("pool")


def attention(h, mix, p, sd):
    """Attention whose values are its keys, over a window and pooled blocks, no positions."""
    T, H, G, d = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"]
    q, k = (h @ sd[p + "q"].T).view(T, H, d), (h @ sd[p + "k"].T).view(T, G, d)
    size, pool = _mask(mix)
    return attention_core(q, k, k, mix["scale"], size, pool).reshape(T, -1) @ sd[p + "o"].T


def biased_attention(h, mix, p, sd, eps):
    """Attention with norms over the whole projections, raw keys as values, a distance bias and an output gate."""
    T, H, G, d = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"]
    q, raw = h @ sd[p + "q"].T, h @ sd[p + "k"].T
    k = rms_norm(raw, sd[p + "k.norm"], eps).view(T, G, d)
    q = rms_norm(q, sd[p + "q.norm"], eps).view(T, H, d)
    o = attention_core(q, k, raw.view(T, G, d), mix["scale"], _mask(mix)[0], None, slopes(H))
    return (o.reshape(T, -1) * torch.sigmoid(h @ sd[p + "g"].T)) @ sd[p + "o"].T


def latent_attention(h, mix, p, sd, eps):
    T, H, d, r, dv, R = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    turn = lambda x: rotate(x, range(T), mix["rot"]["dims"], mix["rot"]["base"])
    cq = rms_norm(h @ sd[p + "dq"].T, sd[p + "dq.norm"], eps)
    q = (cq @ sd[p + "uq"].T).view(T, H, d + r)
    low = h @ sd[p + "dkv"].T
    c = rms_norm(low[:, :R], sd[p + "dkv.norm"], eps)
    k = torch.cat([(c @ sd[p + "uk"].T).view(T, H, d), turn(low[:, R:].reshape(T, 1, r)).expand(T, H, r)], -1)
    q = torch.cat([q[..., :d], turn(q[..., d:])], -1)
    o = attention_core(q, k, (c @ sd[p + "uv"].T).view(T, H, dv), mix["scale"], _mask(mix)[0])
    return o.reshape(T, -1) @ sd[p + "o"].T


# ------------------------------------------------------------------------------------
# gated recurrence
# ------------------------------------------------------------------------------------
def min_gru_core(z_pre, u, state=None):
    """``S <- (1 - z) S + z * candidate`` token by token over ``[T, D]``; returns the states and the last one."""
    S = torch.zeros(u.shape[1], dtype=u.dtype) if state is None else state
    z, cand = torch.sigmoid(z_pre), torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = []
    for t in range(u.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out.append(S)
    return torch.stack(out), S


def min_gru(h, p, sd):
    S, _ = min_gru_core(h @ sd[p + "z"].T + sd[p + "z.b"], h @ sd[p + "x"].T + sd[p + "x.b"])
    g = h @ sd[p + "g"].T
    return (S * g * torch.sigmoid(g)) @ sd[p + "o"].T


def parallel(h, mix, p, sd, eps):
    return mix["left_scale"] * biased_attention(h, mix["left"], p + "left.", sd, eps) + \
        mix["right_scale"] * min_gru(h, p + "right.", sd)


# ------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------
def layer_order(cfg):
    """``(layer, pass)`` of every layer run; ``pass`` is set on the first layer of a pass of the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    body = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


def forward(cfg, sd, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the residual after every layer run."""
    sd = {k: v.to(dtype) for k, v in sd.items()}
    eps = cfg["norm"]["eps"]
    first = sd["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = first
    for li, t in layer_order(cfg):
        layer, p = cfg["layers"][li], f"l{li}."
        if t is not None:
            x = x + (first if t > 0 else 0.0) + sd["loop.step"][t]
        mix, mlp = layer["mixer"], layer["mlp"]
        h = layer_norm(x, sd[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention(h, mix, p + "mix.", sd)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, mix, p + "mix.", sd, eps)
        elif layer["type"] == "parallel":
            y = parallel(h, mix, p + "mix.", sd, eps)
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(y, sd[p + "norm1b"], eps)
        if mlp is not None:
            x = x + layer_norm(dense(layer_norm(x, sd[p + "norm2"], eps), p + "mlp.", sd), sd[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, sd["final.norm"], eps) @ sd["head"].T


def random_model(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights under the on-disk names and shapes for ``cfg``, spread so that leaving a mechanism out shows."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, f=1.0: f * rnd(o, i) / math.sqrt(i)
    near1 = lambda *s: 1.0 + 0.2 * rnd(*s)
    sd = {"embed": rnd(V, W) / cfg["embedding"]["scale"], "final.norm": near1(W), "head": lin(V, W)}
    if cfg.get("loop"):
        sd["loop.step"] = 0.5 * rnd(cfg["loop"]["times"], W)

    def attn(m, mix):
        H, G, d = mix["heads"], mix["kv_heads"], mix["dim"]
        sd[m + "q"], sd[m + "k"] = lin(H * d, W, 1.5), lin(G * d, W, 1.5)
        sd[m + "o"] = lin(W, H * d)

    for li, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{li}.", layer["mixer"], layer["mlp"]
        for n in ("norm1", "norm1b") if mlp is None else ("norm1", "norm1b", "norm2", "norm2b"):
            sd[p + n] = near1(W)
        m = p + "mix."
        if layer["type"] == "attention":
            attn(m, mix)
        elif layer["type"] == "latent_attention":
            H, d, r, dv, Q, R = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["q_rank"], mix["kv_rank"]
            sd[m + "dq"], sd[m + "dq.norm"], sd[m + "uq"] = lin(Q, W), near1(Q), lin(H * (d + r), Q, 1.5)
            sd[m + "dkv"], sd[m + "dkv.norm"] = lin(R + r, W, 1.5), near1(R)
            sd[m + "uk"], sd[m + "uv"], sd[m + "o"] = lin(H * d, R, 1.5), lin(H * dv, R), lin(W, H * dv)
        else:
            l, D = mix["left"], mix["right"]["width"]
            attn(m + "left.", l)
            sd[m + "left.q.norm"], sd[m + "left.k.norm"] = 1.5 * near1(l["heads"] * l["dim"]), near1(l["kv_heads"] * l["dim"])
            sd[m + "left.g"] = lin(l["heads"] * l["dim"], W)
            r = m + "right."
            for n in ("z", "x"):
                sd[r + n], sd[r + n + ".b"] = lin(D, W), 0.5 * rnd(D)
            sd[r + "z.b"] -= 1.5                          # states that remember some tokens
            sd[r + "g"], sd[r + "o"] = lin(D, W), lin(W, D)
        if mlp is not None:
            F = mlp["ff"]
            sd[p + "mlp.up"], sd[p + "mlp.down"] = lin(F, W, 1.5), lin(W, F)
            sd[p + "mlp.act"] = torch.tensor([0.4, -0.3], dtype=torch.float64) + 0.2 * rnd(2)
    return {k: v.to(dtype) for k, v in sd.items()}
