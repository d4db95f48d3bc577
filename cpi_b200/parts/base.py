"""Interfaces of the parts a layer is put together from, and the registries that name them.

A part is built from a `PartSpec` (its kind and its own parameters) and a tensor-name prefix.  It
declares the tensors it needs, loads them (fusing or transposing as it likes), and runs on the tokens
of a step.  No part knows which model it is in: what it may use is its parameters, its weights, the
step's `StepBatch`, and -- for mixers -- the cache and state views the engine hands it.

Interfaces
----------
Norm          requirements(); load(src, dev); __call__(x, out_dtype, rows=None) -> tensor;
              enter(y, x, following, h_out)             # x += norm(y); h_out = following(x)
Position      (no weights) prepare(dev); encoding() -> RotaryEncoding | ScoreBias | None, consumed by its mixer
Mixer         requirements(); load(src, dev); kv_requirement(); state_requirements();
              forward(h, residual, batch, cache)        # residual += mixer(h)
FeedForward   requirements(); load(src, dev); forward(h, residual, batch)   # residual += ffn(h);
              a routed one may also have expert_sum(h, batch) -> ExpertSum | None: its output, not yet added up
Block         run(layer, residual, batch, cache)        # the arrangement of the above; a block that norms the sublayers'
              outputs as well as their inputs declares two more norms (LayerSpec.mixer_post_norm, feed_forward_post_norm)
Junction      requirements(); load(src, dev); run(x, x0, batch)   # between two layers: rewrites the residual x in
              place; x0 is the embedding output (kept by the model when a junction sets `needs_embedding_output`)

`h` is the normed input in the activation dtype [tokens, hidden]; `residual` is the float32 residual
stream [tokens, hidden], updated in place.  A mixer must give the same result for a position whether
the sequence's tokens come in one step or one at a time; what it needs to remember lives in `cache`.

A new kind is added with `register_mixer("name")(cls)` (likewise for the others) and is then chosen
by a `PartSpec` of that kind; nothing else in the library changes.  A part whose step depends on the step
only through device buffers sets `graph_safe = True`; decode steps of a model are captured into CUDA
graphs only if all its parts do.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

from ..config.spec import PartSpec


class Part:
    # Whether a decode step through this part may be captured into a CUDA graph and replayed: its launches
    # must then depend on the step only through device buffers (tokens, positions, slots, page tables),
    # never through host values such as `batch.slots`, data-dependent shapes or a synchronisation.  A part
    # says so itself; the default is no, and the engine replays graphs only if every part of the model does.
    graph_safe = False

    def __init__(self, spec: PartSpec, prefix: str = ""):
        self.spec, self.prefix = spec, prefix

    def requirements(self) -> list:
        return []

    def load(self, source, device) -> None:
        pass


class Norm(Part):
    def __call__(self, x, out_dtype, rows=None, out=None):
        raise NotImplementedError

    def enter(self, y, x, following=None, h_out=None):
        """x += norm(y) for a sublayer's output y (float32 rows or an ExpertSum), then h_out = following(x) if given."""
        raise NotImplementedError(f"{type(self).__name__} does not norm a sublayer's output")


@dataclass(frozen=True)
class ExpertSum:
    """The output of routed experts before it is added up: per token the sum, in the order of its choices, of the chosen
    experts' output rows y[row_of_slot] (already weighted), or of weight * h for a chosen expert number >= n_real (an
    expert whose output is its input).  Lives in workspace buffers until the same part runs again."""
    y: torch.Tensor                # float32 [rows, width]
    row_of_slot: torch.Tensor      # int32 [T, k]
    expert: torch.Tensor           # int32 [T, k]
    weight: torch.Tensor           # float32 [T, k]
    h: torch.Tensor                # [T, width], the experts' input
    n_real: int

    def lists(self):
        return self.y, self.row_of_slot, self.expert, self.weight, self.h, self.n_real

    def add_to(self, x, add=True):
        """x (+)= the sums."""
        from ..csrc import lib as K
        K.norm_step(x, experts=self.lists(), add=add)

    def rows(self, ws):
        out = ws.get("expert_sum", (self.h.shape[0], self.y.shape[-1]), torch.float32)
        self.add_to(out, add=False)
        return out


@dataclass(frozen=True)
class RotaryEncoding:
    """q and k are rotated pairwise: the pair d of a head at position p turns by the angle p * inv_freq[d]
    (float32 [head_dim / 2] on the device); `interleaved` pairs (2d, 2d + 1), otherwise (d, d + head_dim / 2);
    `amplitude` multiplies every sine and cosine (a frequency rule that also rescales the rotated part)."""
    inv_freq: torch.Tensor
    interleaved: bool = False
    amplitude: float = 1.0


@dataclass(frozen=True)
class ScoreBias:
    """Positions act on the attention scores: table[head, min(query position - key position, n - 1)] (float32
    [heads, n] on the device) is added to the scaled score of a query and a key; q and k stay as projected."""
    table: torch.Tensor


class Position(Part):
    """How positions enter a mixer.  `prepare` builds device tables; `encoding()` then says what the part is to
    its mixer: a `RotaryEncoding`, a `ScoreBias`, or None (positions do not enter).  A mixer takes the kinds
    its kernels know and refuses the others by name."""

    def prepare(self, device) -> None:
        pass

    def encoding(self):
        return None


class Mixer(Part):
    """Built with `owns_cache=False` when every run entry of its layer reads another entry's cache."""

    def kv_requirement(self):
        return None

    def state_requirements(self) -> list:
        return []

    def forward(self, h, residual, batch, cache) -> None:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, h, residual, batch) -> None:
        raise NotImplementedError


class Block(Part):
    def run(self, layer, residual, batch, cache) -> None:
        raise NotImplementedError


class Junction(Part):
    needs_embedding_output = False

    def run(self, x, x0, batch) -> None:
        raise NotImplementedError


class CacheView:
    """What a mixer sees of the cache during one step, for its run entry."""

    def __init__(self, manager, entry: int, owns: bool = True):
        self._m, self._entry = manager, entry
        self.owns = owns          # False: this run entry reads `entry`'s cache and must not write it

    def kv(self):
        """(k, v, page_table, page_size): k, v are [pages, kv heads, page_size, head_dim]."""
        return self._m.kv_view(self._entry)

    def stream(self, name: str):
        """(tensor [pages, heads, page_size, dim], page_table, page_size) of a stream that the mixer's
        `KVRequirement.streams` names (attention's are "k" and "v")."""
        return self._m.stream_view(self._entry, name)

    def state(self, name: str) -> torch.Tensor:
        """[slots, *shape] tensor of the named per-sequence state."""
        return self._m.state_view(self._entry, name)


_REGISTRIES: dict = {"norm": {}, "position": {}, "mixer": {}, "feed_forward": {}, "block": {}, "junction": {}}


def _register(family: str, kind: str) -> Callable:
    def deco(cls):
        _REGISTRIES[family][kind] = cls
        return cls
    return deco


def register_norm(kind): return _register("norm", kind)
def register_position(kind): return _register("position", kind)
def register_mixer(kind): return _register("mixer", kind)
def register_feed_forward(kind): return _register("feed_forward", kind)
def register_block(kind): return _register("block", kind)
def register_junction(kind): return _register("junction", kind)


def build_part(family: str, spec: PartSpec, prefix: str = "", **kw):
    reg = _REGISTRIES[family]
    if spec.kind not in reg:
        raise KeyError(f"no {family} of kind '{spec.kind}' is registered; registered: {sorted(reg)}")
    return reg[spec.kind](spec, prefix, **kw)


def registered(family: str) -> list:
    return sorted(_REGISTRIES[family])
