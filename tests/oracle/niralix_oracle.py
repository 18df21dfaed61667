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
    pairs = [(2 * i, 2 * i + 1) if interleaved else (i, i + half) for i in range(half)]
    for i, (a, b) in enumerate(pairs):
        c = torch.tensor([[m * math.cos(p * f[i])] for p in positions], dtype=torch.float64).to(x.dtype)
        s = torch.tensor([[m * math.sin(p * f[i])] for p in positions], dtype=torch.float64).to(x.dtype)
        u, v = x[:, :, a], x[:, :, b]
        out[:, :, a], out[:, :, b] = u * c - v * s, v * c + u * s
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


def random_model(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights under the on-disk names and shapes for ``cfg``, spread so that leaving a mechanism out shows.  Every gla
    layer has ``cfg["_rank"]`` decay features, and decay biases around ``mixer["_bias"]`` (2 when absent).

    Routing has no close calls: the first ``experts`` coordinates of an embedding are flags, ``top`` of them high, that no
    sublayer writes to and that the streams only scale; a router row reads one flag (which one differs by layer) and a little
    of everything else.  The mixtures of a model must therefore agree on ``experts`` and ``top``."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    lin = lambda o, i, f=1.0: f * rnd(o, i) / math.sqrt(i)
    near1 = lambda *s: 1.0 + 0.2 * rnd(*s)
    moe = [l["mlp"] for l in cfg["layers"] if l["mlp"] is not None and l["mlp"]["kind"] == "moe"]
    E, top = (moe[0]["router"]["experts"], moe[0]["router"]["top"]) if moe else (0, 0)
    if any((m["router"]["experts"], m["router"]["top"]) != (E, top) for m in moe):
        raise ValueError("mixtures of different router sizes")

    def back(cols, f=1.0):                       # a projection back to the residual streams
        w = lin(W, cols, f)
        w[:E] = 0.0
        return w

    def norm(n):                                 # stored around zero
        w = 0.2 * rnd(n)
        w[:E] = 0.0
        return w

    embed = rnd(V, W)
    for t in range(V):
        embed[t, :E] = -4.0
        embed[t, torch.randperm(E, generator=g)[:top]] = 4.0
    sd = {"embed": embed, "final.norm": norm(W)}
    for li, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{li}.", layer["mixer"], layer["mlp"]
        for q in (1,) if mlp is None else (1, 2):
            sd[p + f"norm{q}"] = norm(W)
            sd[p + f"hc{q}.in"] = (0.8 + 0.5 * torch.rand(S, generator=g, dtype=torch.float64)) / S
            sd[p + f"hc{q}.out"] = near1(S)
            sd[p + f"hc{q}.mix"] = 0.8 * torch.eye(S, dtype=torch.float64) + 0.2 * torch.rand(S, S, generator=g, dtype=torch.float64)
        m = p + "mix."
        H, dv = mix["heads"], mix["vdim"]
        if layer["type"] == "attention":
            G, dk = mix["kv_heads"], mix["dim"]
            for n, o, i, f in (("q", H * dk, W, 1.5), ("k", G * dk, W, 1.5), ("v", G * dv, W, 1.0)):
                sd[m + n], sd[m + n + ".b"] = lin(o, i, f), 0.5 * rnd(o)
            sd[m + "o"], sd[m + "o.b"] = back(H * dv, 2.0), 0.3 * rnd(W)
            sd[m + "o.b"][:E] = 0.0
            if mix.get("v_mix"):
                sd[m + "vmix"] = torch.tensor(0.3, dtype=torch.float64) + 0.2 * rnd(1)[0].abs()
        elif layer["type"] == "latent_attention":
            d, r, Q, R = mix["dim"], mix["rot_dim"], mix["q_rank"], mix["kv_rank"]
            sd[m + "dq"], sd[m + "dq.norm"], sd[m + "uq"] = lin(Q, W), near1(Q), lin(H * (d + r), Q, 1.5)
            sd[m + "dkv"], sd[m + "dkv.norm"] = lin(R + r, W, 1.5), near1(R)
            sd[m + "uk"], sd[m + "uv"] = lin(H * d, R, 1.5), lin(H * dv, R)
            sd[m + "sink"], sd[m + "g"], sd[m + "o"] = 1.0 + rnd(H), lin(H * dv, W), back(H * dv, 3.0)
        else:
            dk, r = mix["dim"], cfg["_rank"]
            for n, o in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
                sd[m + n] = lin(o, W)
            sd[m + "o"], sd[m + "norm"] = back(H * dv, 1.5), near1(dv)
            sd[m + "a1"], sd[m + "a2"], sd[m + "a2.b"] = lin(r, W), lin(H * dk, r, 1.5), mix.get("_bias", 2.0) + rnd(H * dk)
        if mlp is None:
            continue
        m = p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            sd[m + "gate"], sd[m + "up"], sd[m + "down"] = lin(F, W, 1.5), lin(F, W, 1.5), back(F)
            continue
        for i in range(E):
            F, e = mlp["expert"]["ff"], f"{m}e{i}."
            sd[e + "gate"], sd[e + "up"], sd[e + "down"] = lin(F, W, 1.5), lin(F, W, 1.5), back(F, 2.0)
        router = lin(E, W, 0.2)
        router[:, :E] = 0.5 * torch.eye(E, dtype=torch.float64)[torch.randperm(E, generator=g)]
        sd[m + "router"] = router
    return {k: v.to(dtype) for k, v in sd.items()}


def router_margin(cfg, sd, tokens):
    """Smallest distance in router logits between a chosen and a passed-over expert, over all tokens and mixtures."""
    low = [math.inf]
    keep = globals()["route"]

    def watch(h, router, top):
        z = (h @ router.T).sort(-1, descending=True).values
        if z.shape[1] > top:
            low[0] = min(low[0], float((z[:, top - 1] - z[:, top]).min()))
        return keep(h, router, top)
    globals()["route"] = watch
    try:
        forward(cfg, sd, tokens)
    finally:
        globals()["route"] = keep
    return low[0]
