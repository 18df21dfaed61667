"""Plain, slow statement of the Ditilix decoder: one function per mechanism, one sequence at a time, no cache.

Everything is written from the equations of the design in torch CPU tensors (double precision unless the caller passes
another dtype) and shares no code with the package.  ``cfg`` is the parsed ``config.json`` (a plain dict), ``sd`` a dict
of tensors under their on-disk names.
"""
from __future__ import annotations

import math

import torch


def group_rms_norm(x, groups: int, eps, w):
    """Each of ``groups`` equal consecutive parts of the last axis over its own root mean square, then the weight."""
    parts = []
    for p in x.chunk(groups, dim=-1):
        parts.append(p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps))
    return torch.cat(parts, -1) * w


def sinusoid(positions, width: int):
    """``[n, width]``: sine of ``p * 10000 ** (-2 i / width)`` at entry ``2 i``, the cosine of the same behind it."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for r, p in enumerate(positions):
        for c in range(width):
            a = p * 10000.0 ** (-2.0 * (c // 2) / width)
            out[r, c] = math.sin(a) if c % 2 == 0 else math.cos(a)
    return out


def query_temperature(positions, coef: float, every):
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in positions], dtype=torch.float64)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def keys_values(h, mix, p, sd):
    T, G = h.shape[0], mix["kv_heads"]
    return (h @ sd[p + "k"].T).view(T, G, mix["dim"]), (h @ sd[p + "v"].T).view(T, G, mix["vdim"])


def attention_core(q, k, v, scale, cap):
    """Causal softmax attention: ``q [T, H, dk]`` over ``k [T, G, dk]``, ``v [T, G, dv]``; returns ``[T, H, dv]``."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for a in range(H):
        b = a // (H // G)
        s = q[:, a] @ k[:, b].T * scale
        if cap is not None:
            s = soft_cap(s, cap)
        s = s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf)
        out[:, a] = torch.softmax(s, -1) @ v[:, b]
    return out


def attention(h, mix, p, sd, kv):
    """Attention mixer of one layer; ``kv``: keys and values of the layer that owns them."""
    T, H = h.shape[0], mix["heads"]
    q = (h @ sd[p + "q"].T).view(T, H, mix["dim"])
    if mix.get("q_temp"):
        q = q * query_temperature(range(T), mix["q_temp"]["coef"], mix["q_temp"]["every"]).to(q.dtype).view(T, 1, 1)
    return attention_core(q, *kv, mix["scale"], mix.get("softcap")).reshape(T, -1) @ sd[p + "o"].T


def poly_norm(z, act, eps):
    n = lambda t: t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)
    a, b, c, e = act
    return a * n(z) + b * n(z * z) + c * n(z * z * z) + e


def dense(h, p, sd, eps):
    return poly_norm(h @ sd[p + "up"].T, sd[p + "act"], eps) @ sd[p + "down"].T


def clamped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(x, p, sd, limit):
    return clamped_glu(x @ sd[p + "gate"].T, x @ sd[p + "up"].T, limit) @ sd[p + "down"].T


def route(h, router, top: int):
    """``(weights, experts)`` of every token: the ``top`` largest sigmoid scores."""
    s = torch.sigmoid(h @ router.T)
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return s.gather(1, order), order


def mixture(h, mlp, p, sd):
    w, which = route(h, sd[p + "router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(w.shape[1]):
            out[t] += expert(w[t, j] * h[t], f"{p}e{int(which[t, j])}.", sd, mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ sd[p + "shared.sg"].T) * expert(h, p + "shared.", sd, mlp["shared"]["limit"])
    return out


def forward(cfg, sd, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the residual stream after every layer."""
    sd = {k: v.to(dtype) for k, v in sd.items()}
    eps, groups, width = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["width"]
    x = sd["embed"][torch.as_tensor(tokens, dtype=torch.long)] + sinusoid(range(len(tokens)), width).to(dtype)
    kv_of = {}
    for li, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{li}.", layer["mixer"], layer["mlp"]
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        h = group_rms_norm(x, groups, eps, sd[p + "norm1"])
        if mix.get("kv_from") is not None:
            kv = kv_of[mix["kv_from"]]
        else:
            kv = kv_of[li] = keys_values(h, mix, p + "mix.", sd)
        y = attention(h, mix, p + "mix.", sd, kv)
        if mlp is not None:
            y = y + (dense(h, p + "mlp.", sd, eps) if mlp["kind"] == "dense" else mixture(h, mlp, p + "mlp.", sd))
        x = x + cfg["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return group_rms_norm(x, groups, eps, sd["final.norm"]) @ sd["head"].T * cfg["logit_scale"]


def random_model(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights under the on-disk names and shapes for ``cfg``, spread so that leaving a mechanism out shows.

    Routing has no close calls: the first ``experts`` coordinates of an embedding are flags, ``top`` of them high, that no
    layer writes to; a router row reads one flag (which one differs by layer) and a little of everything else.  The mixtures
    of a model must therefore agree on ``experts`` and ``top``."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, f=1.0: f * rnd(o, i) / math.sqrt(i)
    near1 = lambda *s: 1.0 + 0.2 * rnd(*s)
    moe = [l["mlp"] for l in cfg["layers"] if l["mlp"] is not None and l["mlp"]["kind"] == "moe"]
    E, top = (moe[0]["router"]["experts"], moe[0]["router"]["top"]) if moe else (0, 0)
    if any((m["router"]["experts"], m["router"]["top"]) != (E, top) for m in moe):
        raise ValueError("mixtures of different router sizes")

    def back(cols, f=1.0):                       # a projection back to the residual stream
        w = lin(W, cols, f)
        w[:E] = 0.0
        return w

    embed = rnd(V, W)
    for t in range(V):
        embed[t, :E] = -4.0
        embed[t, torch.randperm(E, generator=g)[:top]] = 4.0
    sd = {"embed": embed, "final.norm": near1(W), "head": lin(V, W)}
    for li, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{li}.", layer["mixer"], layer["mlp"]
        H, G, dk, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
        sd[p + "norm1"] = near1(W)
        m = p + "mix."
        sd[m + "q"], sd[m + "o"] = lin(H * dk, W, 1.5), back(H * dv, 2.0)
        if mix.get("kv_from") is None:
            sd[m + "k"], sd[m + "v"] = lin(G * dk, W, 1.5), lin(G * dv, W)
        if mlp is None:
            continue
        m = p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            sd[m + "up"], sd[m + "down"] = lin(F, W), back(F)
            sd[m + "act"] = torch.tensor([0.6, -0.5, 0.4, 0.1], dtype=torch.float64) * near1(4)
            continue
        ex = [(f"{m}e{i}.", mlp["expert"]["ff"]) for i in range(E)]
        if mlp.get("shared"):
            ex.append((m + "shared.", mlp["shared"]["ff"]))
            sd[m + "shared.sg"] = lin(1, W)
        for e, F in ex:
            sd[e + "gate"], sd[e + "up"], sd[e + "down"] = lin(F, W, 1.5), lin(F, W, 1.5), back(F)
        sd[p + "norm1"][:E] = 1.0
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
