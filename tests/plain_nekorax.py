"""A plain, slow implementation of the Nekorax decoder: float64, whole sequences, one function per mechanism.

It shares nothing with the library: it takes the dictionary that config.json holds and a dictionary of tensors by
name, and runs one sequence from its first token.  Notation: x the residual [T, W], h a sublayer's input, p positions.

    norm         n(x) = tanh(alpha x) * w + b, element by element
    layer        x <- x + n1b(mixer(n1(x)));  x <- x + n2b(ff(n2(x)))
    attention    q, k, v through a short convolution; q, k rotated; the values rotated by their positions and the
                 heads' outputs turned back by the query's; softmax with a 1 in the denominator; elementwise gate
    latent       queries through a low rank, one cached latent and one rotated key part per position, a window
    ff           experts chosen from the best groups by softmax scores plus a correction; identity experts
    loop         a range of layers several times in a row, each pass entered by x <- W_in [x; x0] + step[t]
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def dynamic_tanh(x, W, name):
    """One scalar alpha, a weight and an offset per element; no statistics of x."""
    return torch.tanh(W[name + ".alpha"].to(F) * x) * W[name].to(F) + W[name + ".b"].to(F)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def lin(W, name, x):
    return x @ W[name].to(F).T


# ---- positions ---------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """(frequencies [dims / 2], amplitude).  With `scaling`, pairs that turn slowly over the original length are
    slowed down by `factor`, fast ones kept, a linear ramp over the pair index between them."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def turn(x, pos, f, amplitude=1.0, layout="halves", sign=1.0):
    """x [T, n, D]: the first 2 len(f) elements of every vector turn in pairs by sign * pos * f; pairs (i, i + len(f))
    for "halves", (2i, 2i + 1) for "interleaved"."""
    n = len(f)
    a = sign * pos.to(F)[:, None] * f[None, :]
    c, s = (torch.cos(a) * amplitude)[:, None, :], (torch.sin(a) * amplitude)[:, None, :]
    first, second = (slice(0, n), slice(n, 2 * n)) if layout == "halves" else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


# ---- attention ---------------------------------------------------------------------------------------------------
def visible(T, size=None):
    """[T, T] booleans: query i sees key j; `size`: itself and the size - 1 tokens before it."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    ok = back >= 0
    return ok if size is None else ok & (back < int(size))


def weighted_values(q, k, v, scale, ok, sink_of_one):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G).  With
    `sink_of_one` the denominator has one more term exp(0) that brings no value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~ok, float("-inf"))
        m = s.max(-1, keepdim=True).values
        if sink_of_one:
            m = torch.clamp(m, min=0.0)
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True)
        if sink_of_one:
            den = den + torch.exp(-m)
        out[:, h] = (e / den) @ v[:, g]
    return out


def short_conv(u, w):
    """u [T, C], w [C, taps] (last column: the current token); zeros before the first token."""
    T, C = u.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=F), u])
    return sum(pad[j:j + T] * w[:, j].to(F) for j in range(taps))


def attention_mixer(h, W, p, m):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q, k, v = (lin(W, p + n, h) for n in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(u, W[p + n + ".conv"]) for u, n in ((q, "q"), (k, "k"), (v, "v")))
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    f, _ = frequencies(int(m["rot"]["dims"]), m["rot"]["base"])
    q, k = turn(q, pos, f), turn(k, pos, f)
    fv, _ = frequencies(dv, m["rot"]["base"])
    v = turn(v, pos, fv)
    o = weighted_values(q, k, v, float(m["scale"]), visible(T), True)
    o = turn(o, pos, fv, sign=-1.0).reshape(T, H * dv)
    o = o * torch.sigmoid(lin(W, p + "g", h))
    return lin(W, p + "o", o)


def latent_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T)
    f, amp = frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    cq = rms(lin(W, p + "dq", h), eps) * W[p + "dq.norm"].to(F)
    q = lin(W, p + "uq", cq).view(T, H, d + r)
    down = lin(W, p + "dkv", h)
    c = rms(down[:, :rank], eps) * W[p + "dkv.norm"].to(F)
    k_rot = turn(down[:, rank:].view(T, 1, r), pos, f, amp, "interleaved")
    q_rot = turn(q[..., d:], pos, f, amp, "interleaved")
    q = torch.cat([q[..., :d], q_rot], -1)
    k = torch.cat([lin(W, p + "uk", c).view(T, H, d), k_rot.expand(T, H, r)], -1)
    v = lin(W, p + "uv", c).view(T, H, dv)
    o = weighted_values(q, k, v, float(m["scale"]), visible(T, m["mask"]["size"] if m.get("mask") else None), False)
    return lin(W, p + "o", o.reshape(T, H * dv))


# ---- feed-forward ------------------------------------------------------------------------------------------------
def expert(h, W, p, limit):
    g = torch.clamp(lin(W, p + "gate", h), max=limit)
    u = torch.clamp(lin(W, p + "up", h), -limit, limit)
    return lin(W, p + "down", g * torch.sigmoid(1.702 * g) * (u + 1.0))


def route(z, correction, r):
    """z [E + identity] router logits of one token -> (chosen, their weights)."""
    n = z.numel()
    s = torch.softmax(z, -1)
    c = s + correction
    groups = r.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        per = n // count
        best = torch.topk(c.view(count, per).max(-1).values, keep).indices.tolist()
        c = torch.stack([c[e] if e // per in best else torch.tensor(-math.inf, dtype=F) for e in range(n)])
    idx = torch.topk(c, int(r["top"])).indices
    return idx, s[idx]


def routed_ff(h, W, p, mlp, forced=None, own=None):
    """`forced` ([T, top] expert numbers): these are used instead of the router's own choice, with the weights their
    scores give; `own` (a list) receives the router's own choices either way."""
    T, r, limit = h.shape[0], mlp["router"], float(mlp["expert"]["limit"])
    z = lin(W, p + "router", h)
    n_real = int(r["experts"])
    weight = torch.zeros(T, n_real + int(r.get("identity") or 0), dtype=F)
    for t in range(T):
        idx, w = route(z[t], W[p + "correction"].to(F), r)
        if own is not None:
            own.append(sorted(idx.tolist()))
        if forced is not None:
            idx = torch.as_tensor(forced[t], dtype=torch.long)
            w = torch.softmax(z[t], -1)[idx]
        weight[t, idx] = w
    out = weight[:, n_real:].sum(-1, keepdim=True) * h            # the identity experts
    for e in range(n_real):
        rows = torch.nonzero(weight[:, e]).flatten()
        if rows.numel():
            out[rows] += weight[rows, e, None] * expert(h[rows], W, f"{p}e{e}.", limit)
    return out


# ---- the model ---------------------------------------------------------------------------------------------------
def run_order(cfg):
    """[(layer, number of the pass it enters or None), ...]"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, W, tokens, layers_out=None, forced=None, own_choices=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` (a list) receives x after every layer run.
    `forced` {layer run: [T, top]} replaces the routers' choices there, `own_choices` (a dictionary) receives every
    routed layer run's own choices."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x0 = x.clone()
    for n, (i, entering) in enumerate(run_order(cfg)):
        L, p = cfg["layers"][i], f"l{i}."
        if entering is not None:
            x = lin(W, "loop.in", torch.cat([x, x0], -1)) + W["loop.step"][entering].to(F)
        h = dynamic_tanh(x, W, p + "norm1")
        if L["type"] == "attention":
            y = attention_mixer(h, W, p + "mix.", L["mixer"])
        else:
            y = latent_mixer(h, W, p + "mix.", L["mixer"], eps)
        x = x + dynamic_tanh(y, W, p + "norm1b")
        if L.get("mlp"):
            h = dynamic_tanh(x, W, p + "norm2")
            own = None if own_choices is None else own_choices.setdefault(n, [])
            y = routed_ff(h, W, p + "mlp.", L["mlp"], None if forced is None else forced.get(n), own)
            x = x + dynamic_tanh(y, W, p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = lin(W, "head", dynamic_tanh(x, W, "final.norm"))
    cap = cfg.get("logit_softcap")
    return logits if not cap else float(cap) * torch.tanh(logits / float(cap))
