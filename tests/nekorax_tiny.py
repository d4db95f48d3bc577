"""Small Nekorax configurations and weights for the tests.

The weights are drawn here, not by the library's random mode, with spreads chosen so that faults show: attention scores
a few units wide (a single key can carry a row), norm alphas, weights and offsets away from one and zero, gates on both
sides of a half, expert inputs beyond their clamps, router rows that separate the experts and corrections of both signs
that change the choice, pass vectors that differ.
"""
from __future__ import annotations

import json
import os
import random
import tempfile

import torch


def attention(heads, kv_heads, dim, vdim, rot_dims, conv=None, base=10000.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
         "scale": (2.5 / dim ** 0.5) if scale is None else scale}
    if conv is not None:
        m["conv"] = conv
    return m


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot_dim}, "scale": (1.5 / (dim + rot_dim) ** 0.5) if scale is None else scale}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    return m


def moe(experts, top, ff, identity=None, groups=None, limit=1.5):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}


def layer(mixer, mlp):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def model(layers, width, vocab, eps=1e-5, logit_softcap=None, scale=None, loop=None):
    cfg = {"architecture": "Nekorax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if logit_softcap is not None:
        cfg["logit_softcap"] = logit_softcap
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: sizes that are no multiples of 8 (the float32-pipe products, the separate preparation kernels); the latent layer
# first; three query heads per key head, values larger and smaller than keys, a rotation of part of a head, a window that
# ends inside a page, the scaled frequency rule; groups with identity experts in a group of their own and among others;
# three passes over two layers; a layer without a feed-forward.
MIXED_A = model([
    layer(latent(3, 6, 4, 10, 9, 11, window=19, base=300.0, scaling=(4.0, 64, 8.0, 1.0)), moe(5, 3, 20, identity=1, groups=(3, 2))),
    layer(attention(6, 2, 10, 14, 6, conv=3, base=300.0), moe(6, 2, 12, identity=3, groups=(3, 2), limit=0.8)),
    layer(latent(2, 10, 6, 4, 14, 7, window=70, base=50.0, scaling=(8.0, 32, 4.0, 0.5)), None),
    layer(attention(2, 1, 12, 6, 12, conv=5), moe(4, 2, 28)),
], width=52, vocab=97, logit_softcap=6.0, scale=0.7, loop=(1, 3, 3))

# B: multiples of 8 and 16, so that the bfloat16 path runs the tensor-core products, the fused preparation and the
# tensor-core attention kernels (heads of 64, and one layer whose keys and values differ in size); latents of several
# sizes under windows shorter and longer than a page; the first layer is looped; sixteen experts, a quarter of them the identity.
MIXED_B = model([
    layer(attention(4, 2, 64, 64, 32, conv=4, base=2.5e5), moe(12, 4, 96, identity=4, groups=(4, 2))),
    layer(latent(4, 32, 16, 48, 48, 96, window=50, base=5000.0, scaling=(4.0, 128, 16.0, 1.0)), moe(8, 3, 32, identity=2)),
    layer(attention(2, 1, 32, 64, 16, conv=2, scale=0.4), moe(6, 2, 64, groups=(2, 1))),
    layer(latent(20, 16, 32, 16, 64, 160, window=100), None),
], width=192, vocab=384, eps=1e-6, logit_softcap=12.0, scale=1.7, loop=(0, 2, 2))

# C: what the other two make different or present: one head, no convolution, one tap, a whole-head rotation, a window of
# one and none, no scaling, no groups, no identity experts, one expert a token, all experts a token, no loop, no cap on the
# logits, no embedding scale.
MIXED_C = model([
    layer(attention(1, 1, 8, 8, 8), moe(3, 1, 16)),
    layer(latent(1, 4, 2, 6, 5, 6, window=1), moe(2, 3, 8, identity=1)),
    layer(attention(3, 3, 16, 16, 2, conv=1), None),
    layer(latent(5, 8, 8, 8, 12, 24), moe(1, 1, 8)),
    layer(attention(2, 2, 8, 24, 4, conv=8, base=20.0), moe(4, 2, 16, identity=4, groups=(8, 2))),
], width=40, vocab=64)


def draw_config(seed: int) -> dict:
    """A configuration whose every size, option and constant is drawn from the seed."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 5)):
        if rng.random() < 0.5:
            G, D = rng.choice([1, 2, 3]), rng.choice([4, 8, 16, 32, 64, 128])
            m = attention(G * rng.choice([1, 2, 4]), G, D, rng.choice([D, D, 8, 24, 2 * D]), rng.choice([D, max(2, D // 4 * 2)]),
                          conv=rng.choice([None, 1, 2, 4, 6]), base=rng.choice([100.0, 1e4, 1e6]))
        else:
            r = rng.choice([2, 8, 16, 32])
            m = latent(rng.choice([1, 2, 6, 8]), rng.choice([4, 16, 32]), r, rng.choice([6, 16, 40]), rng.choice([10, 32]),
                       rng.choice([12, 16, 48, 64, 144]), window=rng.choice([None, 1, 7, 33, 64, 100]), base=rng.choice([50.0, 1e4]),
                       scaling=rng.choice([None, (rng.choice([2.0, 8.0]), rng.choice([16, 256]), rng.choice([8.0, 32.0]),
                                                  rng.choice([0.5, 1.0]))]))
        mlp = None
        if rng.random() < 0.8:
            groups = rng.choice([None, (1, 1), (2, 1), (2, 2), (4, 2)])
            per = rng.choice([1, 2, 4])
            total = groups[0] * per if groups else rng.choice([1, 3, 6])
            room = groups[1] * per if groups else total
            ident = rng.randint(0, total - 1)
            mlp = moe(total - ident, rng.randint(1, room), rng.choice([8, 32, 64]), identity=rng.choice([ident, ident or None]),
                      groups=groups, limit=rng.choice([0.7, 2.0]))
        layers.append(layer(m, mlp))
    n = len(layers)
    start = rng.randint(0, n - 1)
    loop = rng.choice([None, (start, rng.randint(start + 1, n), rng.choice([1, 2, 3]))])
    return model(layers, width=rng.choice([24, 40, 64, 128, 264]), vocab=rng.choice([50, 131, 449]), eps=rng.choice([1e-5, 1e-3]),
                 logit_softcap=rng.choice([None, 8.0, 30.0]), scale=rng.choice([None, 0.6, 2.0]), loop=loop)


def draw_weights(cfg: dict, seed: int) -> dict:
    """{name: bfloat16 tensor} for a configuration."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def rn(shape, std, mean=0.0):
        shape = (shape,) if isinstance(shape, int) else shape
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    width, vocab = cfg["width"], cfg["vocab"]

    def norm(name, alpha, w):
        W[name], W[name + ".b"] = rn(width, 0.15, w), rn(width, 0.2)
        W[name + ".alpha"] = torch.tensor(alpha * (1.0 + 0.2 * torch.rand((), generator=g).item())).to(torch.bfloat16)

    W["embed"] = rn((vocab, width), 1.0)
    W["head"] = rn((vocab, width), 1.5 * width ** -0.5)
    norm("final.norm", 0.4, 1.0)
    if cfg.get("loop"):
        W["loop.in"] = rn((width, 2 * width), (2 * width) ** -0.5)
        W["loop.step"] = rn((cfg["loop"]["times"], width), 0.5)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1", 0.6, 1.0)
        norm(p + "norm1b", 0.8, 0.8)
        q = p + "mix."
        if L["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                W[q + n] = rn((rows, width), 1.5 * width ** -0.5)
                if m.get("conv"):
                    W[q + n + ".conv"] = rn((rows, m["conv"]), 0.5, 0.3)
            W[q + "g"] = rn((H * Dv, width), 2.5 * width ** -0.5)
            W[q + "o"] = rn((width, H * Dv), 2.0 * (H * Dv) ** -0.5)
        else:
            H, D, R, Dv, qr, kr = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            W[q + "dq"], W[q + "dq.norm"] = rn((qr, width), 1.5 * width ** -0.5), rn(qr, 0.3, 1.0)
            W[q + "uq"] = rn((H * (D + R), qr), 1.5 * qr ** -0.5)
            W[q + "dkv"], W[q + "dkv.norm"] = rn((kr + R, width), 1.5 * width ** -0.5), rn(kr, 0.3, 1.0)
            W[q + "uk"], W[q + "uv"] = rn((H * D, kr), 1.5 * kr ** -0.5), rn((H * Dv, kr), 1.5 * kr ** -0.5)
            W[q + "o"] = rn((width, H * Dv), 2.0 * (H * Dv) ** -0.5)
        mlp = L.get("mlp")
        if mlp:
            norm(p + "norm2", 0.6, 1.0)
            norm(p + "norm2b", 0.8, 0.8)
            f, E, ff = p + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
            total = E + (mlp["router"].get("identity") or 0)
            W[f + "router"] = rn((total, width), 2.0 * width ** -0.5)
            W[f + "correction"] = rn(total, 0.15, -0.1)
            for e in range(E):
                W[f + f"e{e}.gate"] = rn((ff, width), 1.8 * width ** -0.5)
                W[f + f"e{e}.up"] = rn((ff, width), 1.8 * width ** -0.5)
                W[f + f"e{e}.down"] = rn((width, ff), 1.5 * ff ** -0.5)
    return W


def write_model(cfg: dict, W: dict, root=None) -> str:
    from cpi_b200.weights.safetensors_io import write_safetensors
    d = tempfile.mkdtemp(prefix="nekorax_tiny_", dir=root)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.contiguous() for k, v in W.items()})
    return d


def tokens(n: int, vocab: int, seed: int) -> list:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
