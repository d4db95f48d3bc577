"""Small Delilorn configurations and weights for the tests.

The weights are drawn here, not by the library's random mode, with spreads chosen so that faults show: attention scores
a few units wide (a single key can carry a row), sinks that take a share, norm weights on both sides of zero, gates on
both sides of a half, decays from almost nothing to almost one, router rows that separate the experts.
"""
from __future__ import annotations

import json
import os
import random
import tempfile

import torch


def lightning(heads, dim, vdim, decay=None):
    decay = [0.5 + 0.49 * (i + 1) / heads for i in range(heads)] if decay is None else list(decay)
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, kv_from=None, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot_dim}, "scale": (1.5 / (dim + rot_dim) ** 0.5) if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def attention(heads, kv_heads, dim, vdim, rot_dims, window=None, keep=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": (2.0 / dim ** 0.5) if scale is None else scale}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    return m


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp):
    kind = "lightning" if "decay" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(layers, width, vocab, eps=1e-5):
    return {"architecture": "Delilorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# A: sizes that are no multiples of 8 (the float32-pipe products, the separate preparation kernels, the shared-memory norm);
# two layers that read the first one's latent with other head counts, sizes and query ranks, the second after other kinds of
# layers; values larger and smaller than keys; three query heads per key head; a window that ends inside a page and kept
# tokens that reach past the first page; the scaled frequency rule; a layer without a feed-forward.
MIXED_A = model([
    layer(latent(3, 6, 4, 10, 9, 11, base=300.0), moe(5, 3, 20)),
    layer(latent(2, 10, 4, 6, 14, 11, kv_from=0, base=300.0), moe(4, 1, 12)),
    layer(lightning(3, 10, 14, decay=(0.05, 0.8, 0.995)), moe(6, 2, 28)),
    layer(attention(6, 2, 10, 14, 6, window=19, keep=3, base=300.0, scaling=(4.0, 1.0, 4.0, 64)), moe(3, 3, 9)),
    layer(latent(5, 2, 4, 4, 6, 11, kv_from=0, base=300.0, scale=0.5), None),
    layer(attention(2, 1, 12, 6, 12, window=40, keep=70), moe(4, 2, 20)),
], width=54, vocab=97)

# B: multiples of 8 and 16, so that the bfloat16 path runs the tensor-core products, the fused preparation, the tensor-core
# attention kernels (heads of 64 and of 128) and the latent kernel; two latents, each read again; twenty heads over one
# latent; twelve experts, four of them chosen.
MIXED_B = model([
    layer(attention(4, 2, 64, 64, 32, window=50, keep=4, base=2.5e5, scaling=(8.0, 0.5, 4.0, 128)), moe(12, 4, 96)),
    layer(latent(4, 32, 16, 48, 48, 96, base=5000.0), moe(8, 3, 32)),
    layer(lightning(8, 32, 16), moe(6, 2, 64)),
    layer(latent(20, 16, 16, 16, 64, 96, kv_from=1, base=5000.0), None),
    layer(latent(2, 16, 32, 64, 32, 160), moe(5, 1, 48)),
    layer(latent(6, 24, 32, 32, 40, 160, kv_from=4), moe(4, 2, 32)),
    layer(attention(2, 1, 128, 128, 128, window=100, keep=65, scale=0.2), moe(4, 4, 40)),
    layer(lightning(2, 64, 128, decay=(0.3, 0.9995)), None),
], width=256, vocab=384, eps=2e-5)

# C: what the other two make different or present: one head of each kind, one value per head, no rotation, no window, a window
# of one with no kept tokens, a window with one kept token, decays of zero and one, one expert, all experts a token.
MIXED_C = model([
    layer(lightning(1, 1, 1, decay=(1.0,)), moe(1, 1, 8)),
    layer(attention(1, 1, 8, 8, 0), moe(3, 1, 16)),
    layer(latent(1, 4, 2, 6, 5, 6), moe(2, 2, 8)),
    layer(attention(3, 3, 16, 16, 2, window=1), None),
    layer(lightning(2, 24, 8, decay=(0.0, 0.97)), moe(4, 2, 16)),
    layer(attention(2, 2, 8, 24, 4, window=2, keep=1, base=20.0), None),
    layer(latent(2, 2, 2, 2, 3, 6, kv_from=2), moe(2, 1, 4)),
], width=40, vocab=64)


def draw_config(seed: int) -> dict:
    """A configuration whose every size, option and constant is drawn from the seed."""
    rng = random.Random(seed)
    layers, own = [], []
    for i in range(rng.randint(1, 6)):
        kind = rng.choice(["lightning", "latent", "latent", "attention"])
        if kind == "lightning":
            H = rng.choice([1, 2, 3, 8])
            m = lightning(H, rng.choice([4, 10, 16, 48, 64]), rng.choice([6, 16, 20, 64]),
                          decay=[rng.choice([0.0, 0.3, 0.9, 0.99, 0.999, 1.0]) for _ in range(H)])
        elif kind == "latent":
            src = rng.choice([None] + own)
            if src is None:
                r, rank, base = rng.choice([2, 8, 16, 32]), rng.choice([12, 16, 48, 64, 144]), rng.choice([50.0, 1e4])
                own.append(i)
            else:
                o = layers[src]["mixer"]
                r, rank, base = o["rot_dim"], o["kv_rank"], o["rot"]["base"]
            m = latent(rng.choice([1, 2, 6, 8]), rng.choice([4, 16, 32]), r, rng.choice([6, 16, 40]), rng.choice([10, 32]), rank,
                       kv_from=src, base=base)
        else:
            G, D = rng.choice([1, 2, 3]), rng.choice([4, 8, 16, 32, 64, 128])
            m = attention(G * rng.choice([1, 2, 4]), G, D, rng.choice([D, D, 8, 24, 2 * D]), rng.choice([0, D, D, max(2, D // 4 * 2)]),
                          window=rng.choice([None, 1, 7, 33, 64, 100]), keep=rng.choice([None, 0, 1, 5, 64, 80]),
                          base=rng.choice([100.0, 1e4, 1e6]),
                          scaling=rng.choice([None, (rng.choice([2.0, 8.0]), rng.choice([0.5, 1.0]), rng.choice([2.0, 4.0]),
                                                     rng.choice([16, 256]))]))
        mlp = None
        if rng.random() < 0.8:
            E = rng.choice([1, 3, 8, 20])
            mlp = moe(E, rng.randint(1, min(E, 6)), rng.choice([8, 20, 32, 64]))
        layers.append(layer(m, mlp))
    return model(layers, width=rng.choice([24, 40, 64, 128, 264]), vocab=rng.choice([50, 131, 449]), eps=rng.choice([1e-5, 1e-3]))


def draw_weights(cfg: dict, seed: int) -> dict:
    """{name: bfloat16 tensor} for a configuration."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def rn(shape, std, mean=0.0):
        shape = (shape,) if isinstance(shape, int) else shape
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    width, vocab = cfg["width"], cfg["vocab"]
    W["embed"] = rn((vocab, width), 1.0)
    W["final.norm"] = rn(width, 0.3)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        W[p + "norm1"], W[p + "norm1b"] = rn(width, 0.3), rn(width, 0.25, -0.5)
        q, H, D, Dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        if L["type"] == "lightning":
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * Dv)):
                W[q + n] = rn((rows, width), 1.5 * width ** -0.5)
            W[q + "g"], W[q + "norm"] = rn((H * Dv, width), 2.5 * width ** -0.5), rn(H * Dv, 0.3, 1.0)
        elif L["type"] == "attention":
            for n, rows in (("q", H * D), ("k", m["kv_heads"] * D), ("v", m["kv_heads"] * Dv)):
                W[q + n] = rn((rows, width), 1.5 * width ** -0.5)
        else:
            R, qr, kr = (m[n] for n in ("rot_dim", "q_rank", "kv_rank"))
            W[q + "dq"], W[q + "dq.norm"] = rn((qr, width), 1.5 * width ** -0.5), rn(qr, 0.3, 1.0)
            W[q + "uq"] = rn((H * (D + R), qr), 1.5 * qr ** -0.5)
            if m.get("kv_from") is None:
                W[q + "dkv"], W[q + "dkv.norm"] = rn((kr + R, width), 1.5 * width ** -0.5), rn(kr, 0.3, 1.0)
            W[q + "uk"], W[q + "uv"] = rn((H * D, kr), 1.5 * kr ** -0.5), rn((H * Dv, kr), 1.5 * kr ** -0.5)
            W[q + "sink"], W[q + "g"] = rn(H, 1.0, 1.5), rn((H * Dv, width), 2.5 * width ** -0.5)
        W[q + "o"] = rn((width, H * Dv), 2.0 * (H * Dv) ** -0.5)
        mlp = L.get("mlp")
        if mlp:
            W[p + "norm2"], W[p + "norm2b"] = rn(width, 0.3), rn(width, 0.25, -0.5)
            f, E, ff = p + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
            W[f + "router"] = rn((E, width), 2.0 * width ** -0.5)
            for e in range(E):
                W[f + f"e{e}.up"], W[f + f"e{e}.down"] = rn((ff, width), 1.8 * width ** -0.5), rn((width, ff), 1.5 * ff ** -0.5)
    return W


def strong_sublayers(W: dict) -> None:
    """Weights under which a greedy continuation moves about: with the output matrix being the embedding table, a residual
    in which the token's own embedding dominates would predict that token again and again."""
    for name in W:
        if name.endswith((".norm1b", ".norm2b")):
            W[name] = W[name] + 4.0


def write_model(cfg: dict, W: dict, root=None) -> str:
    from cpi_b200.weights.safetensors_io import write_safetensors
    d = tempfile.mkdtemp(prefix="delilorn_tiny_", dir=root)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.contiguous() for k, v in W.items()})
    return d


def tokens(n: int, vocab: int, seed: int) -> list:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
