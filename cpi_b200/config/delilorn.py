"""Typed configuration of the Delilorn decoder, read from config.json keys.

A Delilorn layer norms a sublayer's input and its output (an RMS norm whose weight is stored around zero).  The mixer is
linear attention with a constant decay per head, attention over a cached latent (its own, or the one of an earlier layer)
with a learned sink and an elementwise gate, or grouped softmax attention over a sliding window beside the sequence's
first tokens.  The feed-forward is routed experts without a gate.  The embedding table is the output matrix too.  Every
size and every constant that can differ between models is a key of config.json:

    architecture  "Delilorn"     vocab, width      norm {eps}
    layers        [{type: "lightning" | "latent_attention" | "attention", mixer {...}, mlp {...} | null}, ...]

lightning:         heads, dim, vdim, decay [one factor per head]
latent_attention:  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims (= rot_dim), scaling | absent},
                   kv_from (the number of an earlier layer) | absent
attention:         heads, kv_heads, dim, vdim, scale, mask {size, keep_first | absent} | absent,
                   rot {base, dims, scaling {factor, low, high, original} | absent} | absent
mlp:               {kind: "moe", expert {ff}, router {experts, top}}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .common import ConfigError
from .nogapel import _rot
from .veredra import _need, _pos_int

MIXER_TYPES = ("lightning", "latent_attention", "attention")


@dataclass(frozen=True)
class DelilornLayer:
    type: str
    mixer: dict                    # the validated keys of the mixer, defaults filled in
    mlp: Optional[dict]            # the validated keys of the feed-forward, None: the layer has none


@dataclass(frozen=True)
class DelilornConfig:
    architecture: str
    vocab: int
    width: int
    layers: tuple
    eps: float
    initializer_range: float

    @staticmethod
    def from_json_dict(raw: dict) -> "DelilornConfig":
        vocab, width = _pos_int(raw, "vocab", "the model"), _pos_int(raw, "width", "the model")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type must be one of {', '.join(MIXER_TYPES)}")
            m = L.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}.mixer must be an object with the mixer's sizes")
            read = {"lightning": _lightning, "latent_attention": _latent, "attention": _attention}[L["type"]]
            layers.append(DelilornLayer(L["type"], read(m, where + ".mixer"), _mlp(L.get("mlp"), where + ".mlp")))
        for i, L in enumerate(layers):
            _check_source(layers, i, L)
        norm = raw.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        return DelilornConfig(
            architecture=str(raw.get("architecture") or (raw.get("architectures") or ["Delilorn"])[0]),
            vocab=vocab, width=width, layers=tuple(layers), eps=float(_need(norm, "eps", "norm")),
            initializer_range=float(raw.get("initializer_range", 0.02)))


def _check_source(layers: list, i: int, L: DelilornLayer) -> None:
    """A layer that reads another's latent reads that of an earlier layer of its kind which has one of its own."""
    j = L.mixer.get("kv_from")
    if j is None:
        return
    where = f"layers[{i}].mixer.kv_from = {j}"
    if j >= i or layers[j].type != "latent_attention" or layers[j].mixer["kv_from"] is not None:
        raise ConfigError(f"config.json: {where} must name an earlier latent_attention layer with a latent of its own")
    for key in ("kv_rank", "rot_dim", "rot"):
        if layers[j].mixer[key] != L.mixer[key]:
            raise ConfigError(f"config.json: {where}: the two layers' {key} must be equal")


def _lightning(m: dict, where: str) -> dict:
    out = {k: _pos_int(m, k, where) for k in ("heads", "dim")}
    out["vdim"] = _pos_int(m, "vdim", where, default=out["dim"])
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != out["heads"]:
        raise ConfigError(f"config.json: {where}.decay must be a list of {out['heads']} numbers, one per head")
    for a in decay:
        if isinstance(a, bool) or not isinstance(a, (int, float)) or not 0.0 <= a <= 1.0:
            raise ConfigError(f"config.json: {where}.decay: a factor is a number from 0 to 1, not {a!r}")
    out["decay"] = tuple(float(a) for a in decay)
    return out


def _latent(m: dict, where: str) -> dict:
    out = {k: _pos_int(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")}
    out["scale"] = float(_need(m, "scale", where))
    out["rot"] = _rot(m, where, out["rot_dim"])
    if out["rot"] is None or out["rot"]["dims"] != out["rot_dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must equal rot_dim = {out['rot_dim']}")
    j = m.get("kv_from")
    if j is not None and (isinstance(j, bool) or not isinstance(j, int) or j < 0):
        raise ConfigError(f"config.json: {where}.kv_from must be a layer number, not {j!r}")
    out["kv_from"] = j
    return out


def _attention(m: dict, where: str) -> dict:
    out = {"heads": _pos_int(m, "heads", where)}
    out["kv_heads"] = _pos_int(m, "kv_heads", where, default=out["heads"])
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}: {out['heads']} heads over {out['kv_heads']} kv_heads")
    out["dim"] = _pos_int(m, "dim", where)
    out["vdim"] = _pos_int(m, "vdim", where, default=out["dim"])
    out["scale"] = float(_need(m, "scale", where))
    out["rot"] = _rot(m, where, out["dim"])
    out["mask"] = None
    if m.get("mask"):
        w, keep = where + ".mask", m["mask"].get("keep_first") or 0
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ConfigError(f"config.json: {w}.keep_first must be a count, not {keep!r}")
        out["mask"] = {"size": _pos_int(m["mask"], "size", w), "keep_first": keep}
    return out


def _mlp(m, where: str) -> Optional[dict]:
    if m is None:
        return None
    if not isinstance(m, dict) or m.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}.kind must be 'moe' (or mlp null)")
    e, r = m.get("expert"), m.get("router")
    if not isinstance(e, dict) or not isinstance(r, dict):
        raise ConfigError(f"config.json: {where} needs the objects 'expert' and 'router'")
    out = {"ff": _pos_int(e, "ff", where + ".expert"), "experts": _pos_int(r, "experts", where + ".router"),
           "top": _pos_int(r, "top", where + ".router")}
    if out["top"] > out["experts"]:
        raise ConfigError(f"config.json: {where}.router.top = {out['top']} exceeds its {out['experts']} experts")
    return out
