"""What the tests of a model family share: a folder with its plain implementation, a runner that feeds an engine step by
step and holds every logit against the plain ones, the index arrays of a step for kernels alone."""
from __future__ import annotations

import math

import torch

DEV = "cuda"


def err(got, want, rms=False):
    """Difference of logit rows, mean taken off, relative to the spread of the expected row: the largest element of the
    worst row (float32), or with `rms` (bfloat16) a row's root mean square: what nine rows in ten stay under, and a
    quarter of the worst row but the worst in fifty (a router's near-tie may fall the other way, which is no fault).  The
    float32 measure leaves out nothing."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    size = (d.pow(2).mean(-1).sqrt() if rms else d.abs().max(-1).values) / w.pow(2).mean(-1).sqrt().clamp_min(1e-6)
    if rms:
        n = size.numel()
        drop = max(1, math.ceil(0.02 * n)) if n >= 5 else 0
        kept = size.sort().values[:n - drop]
        return max(torch.quantile(size, 0.9).item(), kept.max().item() / 4)
    return size.max().item()


class Built:
    """A model folder of a family and its plain implementation; `tiny` and `plain` are the family's modules."""

    def __init__(self, tiny, plain, cfg, seed, tmp, change=None):
        self.P, self.cfg, self.W = plain, cfg, tiny.draw_weights(cfg, seed)
        if change is not None:
            change(self.W)
        self.dir = tiny.write_model(cfg, self.W, root=str(tmp))
        self._plain = {}

    def plain(self, toks):
        key = tuple(toks)
        if key not in self._plain:
            self._plain[key] = self.P.forward(self.cfg, self.W, list(toks))
        return self._plain[key]

    def engine(self, dtype, **kw):
        from cpi_b200.engine import Engine
        kw.setdefault("max_tokens", 4096)
        return Engine.from_model_dir(self.dir, dtype=dtype, **kw)


class Run:
    """Feeds requests to an engine step by step and keeps the logits by (request, position).  In bfloat16 it also records
    the experts every token chose: a router's near-tie may fall the other way than in double precision, and the cache
    carries that token on.  The plain implementation is then run with the engine's choices, and the choices themselves are
    compared apart: all but a few must be the plain router's own.  In float32 nothing is recorded or forced."""

    def __init__(self, engine, record=True):
        self.e, self.slots, self.logits = engine, {}, {}
        self.routing = {}          # rid -> {layer run: {position: [experts]}}
        # (while choices are recorded the engine replays no graphs: `record=False` for a test of those)
        self.cap = engine.capture_routing(True) if record and engine.dtype == torch.bfloat16 else None
        order = [r.layer for r in engine.spec.run_order]
        self.runs = {layer: [n for n, l in enumerate(order) if l == layer] for layer in set(order)}

    def step(self, items):
        from cpi_b200.engine import StepEntry
        entries, layout = [], []
        for rid, toks, want in items:
            if rid not in self.slots:
                self.slots[rid] = self.e.acquire_slot()
            start = self.e.length(self.slots[rid])
            entries.append(StepEntry(self.slots[rid], list(toks), list(want)))
            layout.append((rid, start, list(want), len(entries[-1].tokens)))
        for lst in (self.cap or {}).values():
            lst.clear()
        out = self.e.step(entries).float().cpu()
        self.e.check_device_errors()
        r = 0
        for rid, start, want, n in layout:
            for w in want:
                self.logits.setdefault(rid, {})[start + w] = out[r]
                r += 1
        for layer, lst in (self.cap or {}).items():       # per piece of the step, one tensor per run of the layer
            runs = self.runs[layer]
            for k, run in enumerate(runs):
                idx, t = torch.cat([x.cpu() for x in lst[k::len(runs)]]), 0
                for rid, start, want, n in layout:
                    for i in range(n):
                        self.routing.setdefault(rid, {}).setdefault(run, {})[start + i] = sorted(idx[t + i].tolist())
                    t += n

    def end(self, rid):
        self.e.release_slot(self.slots.pop(rid))

    def check(self, built, requests, tol):
        for rid, got in self.logits.items():
            toks = requests[rid]
            forced = {}
            for run, by_pos in self.routing.get(rid, {}).items():
                n = max(by_pos) + 1
                assert sorted(by_pos) == list(range(n)), f"the choices of {rid} in layer run {run} have gaps"
                forced[run] = [by_pos[p] for p in range(n)]
            if forced:
                n = min(len(v) for v in forced.values())
                own = {}
                ref = built.P.forward(built.cfg, built.W, list(toks[:n]), forced={l: v[:n] for l, v in forced.items()}, own_choices=own)
                other = sum(a != b for l in forced for a, b in zip(forced[l][:n], own[l]))
                assert other <= max(2, 0.05 * n * len(forced)), f"request {rid}: {other} choices of {n * len(forced)} differ"
            else:
                ref = built.plain(toks)
            pos = sorted(got)
            e = err(torch.stack([got[p] for p in pos]), ref[pos], rms=tol > 1e-3)
            assert e < tol, f"request {rid}: error {e:.3g} (tolerance {tol}) over positions {pos[0]}..{pos[-1]}"


def K():
    from cpi_b200.csrc import lib
    return lib


class FakeBatch:
    """The index arrays a kernel reads of a step: sequences of `n_new` tokens that start at `starts`, in query tiles of at
    most `tile` tokens."""

    def __init__(self, slots, starts, n_new, dev=DEV, tile=256):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        self.n_seqs, self.max_new, self.n_tokens = len(slots), max(n_new), sum(n_new)
        self.is_decode = self.max_new == 1
        self.seq_slot, self.seq_start, self.seq_new = i32(slots), i32(starts), i32(n_new)
        tok0, seq, pos, tiles, base = [], [], [], [], 0
        for s, (st, n) in enumerate(zip(starts, n_new)):
            tok0.append(base); seq += [s] * n; pos += range(st, st + n)
            tiles += [(base + o, min(tile, n - o)) for o in range(0, n, tile)]
            base += n
        self.seq_tok0, self.token_seq, self.token_pos = i32(tok0), i32(seq), i32(pos)
        self.n_q_tiles, self.tile_tok0, self.tile_rows = len(tiles), i32([t[0] for t in tiles]), i32([t[1] for t in tiles])


def rn(g, *shape, std=1.0, mean=0.0):
    return torch.randn(*shape, generator=g) * std + mean


def build(family, kind, params, weights, **kw):
    from cpi_b200.config.spec import PartSpec
    from cpi_b200.parts.base import build_part
    from cpi_b200.parts.workspace import Workspace
    from cpi_b200.weights.store import DictSource
    part = build_part(family, PartSpec(kind, params), "", workspace=Workspace(torch.device(DEV)), **kw)
    part.load(DictSource(weights), torch.device(DEV))
    return part
