"""Plain, slow statement of the Niralix decoder: one function per mechanism, one sequence at a time, no cache.

Everything is written from the equations of the design in torch CPU tensors (double precision unless the caller passes
another dtype) and shares no code with the package.  ``cfg`` is the parsed ``config.json`` (a plain dict), ``sd`` a dict
of tensors under their on-disk names.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ------------------------------------------------------------------------------------
# rotation
# ------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """``(frequencies [dims / 2], factor of sine and cosine)``, with the YaRN blend when ``rot`` has a scaling."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    turn = lambda t: dims * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turn(s["fast"])), 0), min(math.ceil(turn(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot, interleaved):
    """Rotate the first ``rot.dims`` entries of the last axis of ``x [T, heads, d]``."""
    f, m = rotary_frequencies(rot)
    out, half = x.clone(), rot["dims"] // 2
    for t, p in enumerate(positions):
        for i in range(half):
            a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
            c, s = m * math.cos(p * f[i]), m * math.sin(p * f[i])
            u, v = x[t, :, a], x[t, :, b]
            out[t, :, a], out[t, :, b] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------
def attention_core(q, k, v, scale, sink=None):
    """Causal softmax attention: ``q [T, H, dk]`` over ``k [T, G, dk]``, ``v [T, G, dv]``; ``sink [H]`` joins the denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for a in range(H):
        b = a // (H // G)
        s = q[:, a] @ k[:, b].T * scale
        s = s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[a].to(s.dtype).expand(T, 1)], 1)
        w = torch.softmax(s, -1)[:, :T]
        out[:, a] = w @ v[:, b]
    return out


def attention(h, mix, p, sd, v_first):
    """Attention mixer; ``v_first``: values of the first layer that mixes values (None in that layer and in layers that do
    not mix).  Returns the output and this layer's values."""
    T, H, G, dk, dv = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    lin = lambda n: h @ sd[p + n].T + sd[p + n + ".b"]
    q, k, v = lin("q").view(T, H, dk), lin("k").view(T, G, dk), lin("v").view(T, G, dv)
    q, k = rotate(q, range(T), mix["rot"], False), rotate(k, range(T), mix["rot"], False)
    own = v
    if v_first is not None:
        v = (1 - sd[p + "vmix"]) * v + sd[p + "vmix"] * v_first
    o = attention_core(q, k, v, mix["scale"])
    return o.reshape(T, -1) @ sd[p + "o"].T + sd[p + "o.b"], own


def latent_attention(h, mix, p, sd, eps):
    T, H, d, r, dv, R = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    cq = rms_norm(h @ sd[p + "dq"].T, sd[p + "dq.norm"], eps)
    q = (cq @ sd[p + "uq"].T).view(T, H, d + r)
    low = h @ sd[p + "dkv"].T
    c = rms_norm(low[:, :R], sd[p + "dkv.norm"], eps)
    kr = rotate(low[:, R:].view(T, 1, r), range(T), mix["rot"], True)
    k = torch.cat([(c @ sd[p + "uk"].T).view(T, H, d), kr.expand(T, H, r)], -1)
    q = torch.cat([q[..., :d], rotate(q[..., d:], range(T), mix["rot"], True)], -1)
    o = attention_core(q, k, (c @ sd[p + "uv"].T).view(T, H, dv), mix["scale"], sd[p + "sink"])
    return (o.reshape(T, -1) * torch.sigmoid(h @ sd[p + "g"].T)) @ sd[p + "o"].T


# ------------------------------------------------------------------------------------
# gated linear attention
# ------------------------------------------------------------------------------------
def gla_decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def gla_core(q, k, v, alpha, state=None):
    """``q, k, alpha [T, H, dk]``, ``v [T, H, dv]``, token by token; returns the outputs and the last state."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(T):
        S = alpha[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out.append((q[t].unsqueeze(-1) * S).sum(1))
    return torch.stack(out), S


def gla(h, mix, p, sd, eps):
    T, H, dk, dv = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    lin = lambda n: h @ sd[p + n].T
    q, k, v = lin("q").view(T, H, dk) * dk ** -0.5, lin("k").view(T, H, dk), lin("v").view(T, H, dv)
    z = (lin("a1") @ sd[p + "a2"].T + sd[p + "a2.b"]).view(T, H, dk)
    o, _ = gla_core(q, k, v, gla_decay(z, mix["tau"]))
    o = rms_norm(o, sd[p + "norm"], eps).reshape(T, -1)
    g = lin("g")
    return (o * g * torch.sigmoid(g)) @ sd[p + "o"].T


# ------------------------------------------------------------------------------------
# feed-forward
# ------------------------------------------------------------------------------------
def gated_unit(x, p, sd):
    g = x @ sd[p + "gate"].T
    return (g * torch.sigmoid(g) * (x @ sd[p + "up"].T)) @ sd[p + "down"].T


def route(h, router, top: int):
    """``(weights, experts)`` of every token: the ``top`` largest softmax scores over all experts, as they are."""
    s = torch.softmax(h @ router.T, -1)
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return s.gather(1, order), order


def mixture(h, mlp, p, sd):
    w, which = route(h, sd[p + "router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(w.shape[1]):
            out[t] += w[t, j] * gated_unit(h[t], f"{p}e{int(which[t, j])}.", sd)
    return out


# ------------------------------------------------------------------------------------
# residual streams
# ------------------------------------------------------------------------------------
def streams_in(xs, w_in):
    return sum(w_in[s] * xs[s] for s in range(len(xs)))


def streams_out(xs, y, mix, out):
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out[t] * y for t in range(n)]


def forward(cfg, sd, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the sum of the streams after every layer."""
    sd = {k: v.to(dtype) for k, v in sd.items()}
    eps = cfg["norm"]["eps"]
    xs = [sd["embed"][torch.as_tensor(tokens, dtype=torch.long)]] * cfg["streams"]
    v_first = None
    for li, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{li}.", layer["mixer"], layer["mlp"]
        h = rms_norm(streams_in(xs, sd[p + "hc1.in"]), 1 + sd[p + "norm1"], eps)
        if layer["type"] == "attention":
            mixes = bool(mix.get("v_mix"))
            y, own = attention(h, mix, p + "mix.", sd, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, mix, p + "mix.", sd, eps)
        elif layer["type"] == "gla":
            y = gla(h, mix, p + "mix.", sd, eps)
        else:
            raise ValueError(layer["type"])
        xs = streams_out(xs, y, sd[p + "hc1.mix"], sd[p + "hc1.out"])
        if mlp is not None:
            h = rms_norm(streams_in(xs, sd[p + "hc2.in"]), 1 + sd[p + "norm2"], eps)
            y = gated_unit(h, p + "mlp.", sd) if mlp["kind"] == "dense" else mixture(h, mlp, p + "mlp.", sd)
            xs = streams_out(xs, y, sd[p + "hc2.mix"], sd[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(sum(xs))
    return rms_norm(sum(xs), 1 + sd["final.norm"], eps) @ sd["embed"].T * cfg["logit_scale"]
