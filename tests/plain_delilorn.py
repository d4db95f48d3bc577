"""A plain, slow implementation of the Delilorn decoder: float64, whole sequences, one function per mechanism.

It shares nothing with the library: it takes the dictionary that config.json holds and a dictionary of tensors by
name, and runs one sequence from its first token.  Notation: x the residual [T, W], h a sublayer's input, p positions.

    norm         n(x) = x / rms(x) * (1 + w)
    layer        x <- x + n1b(mixer(n1(x)));  x <- x + n2b(ff(n2(x)))
    lightning    a matrix state per head that shrinks by a constant factor a token and gains k v^T; silu on q, k and v
    latent       queries through a low rank; one cached latent and one rotated key part per position, its own or those of
                 an earlier layer; a learned sink per head; an elementwise gate
    attention    grouped heads, a rotation of part of a head, a sliding window beside the sequence's first tokens
    ff           ungated experts with a squared relu, weighted by the softmax scores of the chosen ones as they are
    logits       from the embedding table
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_about_one(x, w, eps):
    """The weight is a distance from one."""
    return rms(x, eps) * (1.0 + w.to(F))


def lin(W, name, x):
    return x @ W[name].to(F).T


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ---- positions ---------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """One frequency per pair.  With `scaling`, waves longer than original / low are slowed down by `factor`, waves
    shorter than original / high stay, and between the two the frequency is a blend by the number of waves that fit."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            wave = 2.0 * math.pi / f
            n, lo, hi = float(scaling["original"]) / wave, float(scaling["low"]), float(scaling["high"])
            slow = f / float(scaling["factor"])
            if n < lo:
                f = slow
            elif n <= hi:
                s = (n - lo) / (hi - lo)
                f = (1.0 - s) * slow + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def turn(x, pos, f):
    """x [T, n, D]: the first 2 len(f) elements of every vector turn in pairs (i, i + len(f)) by pos * f_i."""
    n = len(f)
    a = pos.to(F)[:, None, None] * f
    c, s = torch.cos(a), torch.sin(a)
    u, v, rest = x[..., :n], x[..., n:2 * n], x[..., 2 * n:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


# ---- softmax attention -------------------------------------------------------------------------------------------
def visible(T, size=None, keep_first=0):
    """[T, T] booleans: query i sees key j.  `size`: itself and the size - 1 tokens before it, and besides these the
    sequence's first `keep_first` tokens, never a later token."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if size is None else ok & ((i - j < int(size)) | (j < int(keep_first)))


def weighted_values(q, k, v, scale, ok, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G).  `sink` [H]:
    the denominators have one more term exp(sink_h)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~ok, float("-inf"))
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = torch.maximum(m, sink[h].to(F))
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h].to(F) - m)
        out[:, h] = (e / den) @ v[:, g]
    return out


def attention_mixer(h, W, p, m):
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G, dv = int(m["kv_heads"]), int(m["vdim"])
    q, k, v = lin(W, p + "q", h).view(T, H, d), lin(W, p + "k", h).view(T, G, d), lin(W, p + "v", h).view(T, G, dv)
    if m.get("rot"):
        f = frequencies(int(m["rot"]["dims"]), m["rot"]["base"], m["rot"].get("scaling"))
        pos = torch.arange(T)
        q, k = turn(q, pos, f), turn(k, pos, f)
    mask = m.get("mask")
    ok = visible(T, mask["size"], mask.get("keep_first", 0)) if mask else visible(T)
    return lin(W, p + "o", weighted_values(q, k, v, float(m["scale"]), ok).reshape(T, H * dv))


def latent_of(h, W, p, m, eps):
    """What a layer with its own latent keeps per position: the normed latent and the rotated key part."""
    rank, r = int(m["kv_rank"]), int(m["rot_dim"])
    down = lin(W, p + "dkv", h)
    c = rms(down[:, :rank], eps) * W[p + "dkv.norm"].to(F)
    f = frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    return c, turn(down[:, None, rank:], torch.arange(h.shape[0]), f)


def latent_mixer(h, W, p, m, eps, kept):
    """`kept`: (c [T, rank], r [T, 1, rot_dim]) of this layer or of the layer it reads."""
    T = h.shape[0]
    H, d, r, dv = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim"))
    c, k_rot = kept
    f = frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    q = lin(W, p + "uq", rms(lin(W, p + "dq", h), eps) * W[p + "dq.norm"].to(F)).view(T, H, d + r)
    q = torch.cat([q[..., :d], turn(q[..., d:], torch.arange(T), f)], -1)
    k = torch.cat([lin(W, p + "uk", c).view(T, H, d), k_rot.expand(T, H, r)], -1)
    v = lin(W, p + "uv", c).view(T, H, dv)
    o = weighted_values(q, k, v, float(m["scale"]), visible(T), W[p + "sink"]).reshape(T, H * dv)
    return lin(W, p + "o", o * torch.sigmoid(lin(W, p + "g", h)))


# ---- the recurrence ----------------------------------------------------------------------------------------------
def decayed_sum(q, k, v, decay, S=None):
    """q, k [T, H, d], v [T, H, dv], decay [H]: per head S <- decay S + k v^T, o = S^T q.  Returns (o, the last S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if S is None else S.to(F).clone()
    a = torch.as_tensor(decay, dtype=F)[:, None, None]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = a * S + k[t, :, :, None] * v[t, :, None, :]
        out[t] = (q[t, :, :, None] * S).sum(1)
    return out, S


def lightning_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = silu(lin(W, p + "q", h)).view(T, H, d), silu(lin(W, p + "k", h)).view(T, H, d)
    v = silu(lin(W, p + "v", h)).view(T, H, dv)
    o = decayed_sum(q, k, v, m["decay"])[0].reshape(T, H * dv)
    o = rms(o, eps) * W[p + "norm"].to(F) * torch.sigmoid(lin(W, p + "g", h))
    return lin(W, p + "o", o)


# ---- feed-forward ------------------------------------------------------------------------------------------------
def expert(h, W, p):
    return lin(W, p + "down", torch.clamp(lin(W, p + "up", h), min=0.0) ** 2)


def routed_ff(h, W, p, mlp, forced=None, own=None):
    """`forced` ([T, top] expert numbers): these are used instead of the router's own choice, with the weights their
    scores give; `own` (a list) receives the router's own choices either way."""
    T, n, top = h.shape[0], int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    s = torch.softmax(lin(W, p + "router", h), -1)
    weight = torch.zeros(T, n, dtype=F)
    for t in range(T):
        idx = torch.topk(s[t], top).indices
        if own is not None:
            own.append(sorted(idx.tolist()))
        if forced is not None:
            idx = torch.as_tensor(forced[t], dtype=torch.long)
        weight[t, idx] = s[t, idx]
    out = torch.zeros_like(h)
    for e in range(n):
        rows = torch.nonzero(weight[:, e]).flatten()
        if rows.numel():
            out[rows] += weight[rows, e, None] * expert(h[rows], W, f"{p}e{e}.")
    return out


# ---- the model ---------------------------------------------------------------------------------------------------
def forward(cfg, W, tokens, layers_out=None, forced=None, own_choices=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` (a list) receives x after every layer.
    `forced` {layer: [T, top]} replaces the routers' choices there, `own_choices` (a dictionary) receives every routed
    layer's own choices."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm_about_one(x, W[p + "norm1"], eps)
        if L["type"] == "attention":
            y = attention_mixer(h, W, p + "mix.", m)
        elif L["type"] == "lightning":
            y = lightning_mixer(h, W, p + "mix.", m, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                src = i
                kept[i] = latent_of(h, W, p + "mix.", m, eps)
            y = latent_mixer(h, W, p + "mix.", m, eps, kept[src])
        x = x + norm_about_one(y, W[p + "norm1b"], eps)
        if L.get("mlp"):
            h = norm_about_one(x, W[p + "norm2"], eps)
            own = None if own_choices is None else own_choices.setdefault(i, [])
            y = routed_ff(h, W, p + "mlp.", L["mlp"], None if forced is None else forced.get(i), own)
            x = x + norm_about_one(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(W, "embed", norm_about_one(x, W["final.norm"], eps))
