"""Typed configuration of the Nekorax decoder, read from config.json keys.

A Nekorax layer norms a sublayer's input and its output (with a tanh per element instead of a root mean square).  The
mixer is softmax attention over short-convolved q, k and v whose values are rotated by their positions and whose outputs
are turned back, with a one in the softmax denominator and an elementwise gate; or attention over a cached latent with a
sliding window.  The feed-forward is routed experts, some of which may be the identity.  A range of layers may run several
times.  Every size and every constant that can differ between models is a key of config.json:

    architecture  "Nekorax"      vocab, width      norm {eps}      embedding {scale}      logit_softcap | absent
    loop          {start, stop, times} | absent
    layers        [{type: "attention" | "latent_attention", mixer {...}, mlp {...} | null}, ...]

attention:         heads, kv_heads, dim, vdim, scale, conv (taps) | absent, rot {base, dims}
latent_attention:  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask {size} | absent,
                   rot {base, dims (= rot_dim), scaling {factor, original, fast, slow} | absent}
mlp:               {kind: "moe", expert {ff, limit}, router {experts, top, identity | absent,
                   groups {count, keep} | absent}}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .common import ConfigError
from .kikerax import _heads, _rot
from .veredra import _need, _pos_int

MIXER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class NekoraxLayer:
    type: str
    mixer: dict                    # the validated keys of the mixer, defaults filled in
    mlp: Optional[dict]            # the validated keys of the feed-forward, None: the layer has none


@dataclass(frozen=True)
class NekoraxConfig:
    architecture: str
    vocab: int
    width: int
    layers: tuple
    loop: Optional[tuple]          # (start, stop, times) or None
    eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    initializer_range: float

    @staticmethod
    def from_json_dict(raw: dict) -> "NekoraxConfig":
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
            mixer = _attention(m, where + ".mixer") if L["type"] == "attention" else _latent(m, where + ".mixer")
            layers.append(NekoraxLayer(L["type"], mixer, _mlp(L.get("mlp"), where + ".mlp")))
        norm = raw.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        cap = raw.get("logit_softcap")
        if cap is not None and not float(_need(raw, "logit_softcap", "the model")) > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        emb = raw.get("embedding")
        if emb is not None and not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object with 'scale'")
        return NekoraxConfig(
            architecture=str(raw.get("architecture") or (raw.get("architectures") or ["Nekorax"])[0]),
            vocab=vocab, width=width, layers=tuple(layers), loop=_loop(raw.get("loop"), len(layers)),
            eps=float(_need(norm, "eps", "norm")),
            embedding_scale=1.0 if not emb else float(_need(emb, "scale", "embedding")),
            logit_softcap=None if cap is None else float(cap),
            initializer_range=float(raw.get("initializer_range", 0.02)))

    def run_order(self) -> list:
        """[(layer, number of the pass that starts with it, or None), ...]"""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        out = [(i, None) for i in range(start)]
        for t in range(times):
            out += [(i, t if i == start else None) for i in range(start, stop)]
        return out + [(i, None) for i in range(stop, n)]


def _loop(lp, n_layers: int) -> Optional[tuple]:
    if not lp:
        return None
    if not isinstance(lp, dict):
        raise ConfigError("config.json: 'loop' must be an object with 'start', 'stop' and 'times'")
    start = lp.get("start")
    if isinstance(start, bool) or not isinstance(start, int):
        raise ConfigError(f"config.json: loop.start must be a layer number, not {start!r}")
    stop, times = _pos_int(lp, "stop", "loop"), _pos_int(lp, "times", "loop")
    if not 0 <= start < stop <= n_layers:
        raise ConfigError(f"config.json: loop: layers {start} .. {stop} of {n_layers}")
    return start, stop, times


def _attention(m: dict, where: str) -> dict:
    out = _heads(m, where)
    out["conv"] = None if m.get("conv") is None else _pos_int(m, "conv", where)
    if m.get("mask"):
        raise ConfigError(f"config.json: {where}.mask: this mixer sees every earlier position")
    out["rot"] = _rot(m, where, out["dim"])
    if out["rot"] is None:
        raise ConfigError(f"config.json: {where}.rot is missing")
    if out["vdim"] % 2:
        raise ConfigError(f"config.json: {where}.vdim = {out['vdim']} must be even (the values are rotated)")
    return out


def _latent(m: dict, where: str) -> dict:
    out = {k: _pos_int(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")}
    out["scale"] = float(_need(m, "scale", where))
    out["rot"] = _rot(m, where, out["rot_dim"])
    if out["rot"] is None or out["rot"]["dims"] != out["rot_dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must equal rot_dim = {out['rot_dim']}")
    out["mask"] = None
    if m.get("mask"):
        out["mask"] = {"size": _pos_int(m["mask"], "size", where + ".mask")}
    return out


def _mlp(m, where: str) -> Optional[dict]:
    if m is None:
        return None
    if not isinstance(m, dict) or m.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}.kind must be 'moe' (or mlp null)")
    e, r = m.get("expert"), m.get("router")
    if not isinstance(e, dict) or not isinstance(r, dict):
        raise ConfigError(f"config.json: {where} needs the objects 'expert' and 'router'")
    ident = r.get("identity") or 0
    if isinstance(ident, bool) or not isinstance(ident, int) or ident < 0:
        raise ConfigError(f"config.json: {where}.router.identity must be a count, not {ident!r}")
    out = {"kind": "moe", "ff": _pos_int(e, "ff", where + ".expert"), "limit": float(_need(e, "limit", where + ".expert")),
           "experts": _pos_int(r, "experts", where + ".router"), "identity": int(ident),
           "top": _pos_int(r, "top", where + ".router"), "groups": 1, "keep": 1}
    if not out["limit"] > 0:
        raise ConfigError(f"config.json: {where}.expert.limit must be positive")
    total = out["experts"] + out["identity"]
    g = r.get("groups")
    if g:
        out["groups"] = _pos_int(g, "count", where + ".router.groups")
        out["keep"] = _pos_int(g, "keep", where + ".router.groups", default=out["groups"])
    if total % out["groups"] or out["keep"] > out["groups"]:
        raise ConfigError(f"config.json: {where}.router: {total} experts in {out['groups']} groups of which "
                          f"{out['keep']} are kept")
    if out["top"] > out["keep"] * (total // out["groups"]):
        raise ConfigError(f"config.json: {where}.router.top = {out['top']} exceeds the experts of the kept groups")
    return out
