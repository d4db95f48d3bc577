"""Delilorn through the engine against the plain implementation (`plain_delilorn.py`): every mechanism alone, whole
prompts, portions, token-by-token decoding, unequal batches, reused slots and pages, the edges of windows and of the kept
first tokens, far keys, the recurrence cut into runs, latents read by later layers, long decoding, other sizes, generation
through the entry point, and the replay tool."""
from __future__ import annotations

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import delilorn_tiny as V
import plain_delilorn as P
from family_run import DEV, Built as FamilyBuilt, FakeBatch, K, Run, build, err, rn

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-4, "bfloat16": 4e-2}
F64 = torch.float64


def Built(*args):
    return FamilyBuilt(V, P, *args)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("delilorn")
    return {"A": Built(V.MIXED_A, 11, tmp), "B": Built(V.MIXED_B, 12, tmp), "C": Built(V.MIXED_C, 13, tmp)}


# ---- mechanisms alone ------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,W,dt", [(5, 54, torch.float32), (70, 256, torch.bfloat16), (3, 37, torch.bfloat16), (4, 1028, torch.float32),
                                    (9, 2048, torch.bfloat16), (3, 4100, torch.bfloat16), (2, 8192, torch.float32), (2, 8200, torch.bfloat16),
                                    (2, 13001, torch.float32)])
def test_norms_with_weights_around_zero_on_both_sides(T, W, dt):
    """A sublayer's output enters the residual through its norm and the next sublayer's input leaves it, in one kernel (rows
    in registers of several sizes, and in shared memory); with a plain weight; without a norm behind; with a wide row
    stride; weights in both precisions."""
    g = torch.Generator().manual_seed(W)
    eps = 3e-2                                      # large enough to show where it stands
    for wdt in (torch.float32, torch.bfloat16):
        Wt = {n: rn(g, W, std=0.4).to(wdt) for n in "abc"}
        kind = {"a": 1.0, "b": 1.0, "c": 0.0}
        norm = {n: build("norm", "rmsnorm", {"size": W, "eps": eps, "weight": n, "weight_offset": o}, Wt) for n, o in kind.items()}
        plain = {n: (lambda v, n=n: P.rms(v, eps) * (kind[n] + Wt[n].double())) for n in kind}
        x, y = rn(g, T, W, std=0.5), rn(g, T, W, std=0.2)
        tol = 4e-6 if dt == torch.float32 else 1e-2
        assert (norm["a"](x.to(DEV), dt).cpu().double() - P.norm_about_one(x.double(), Wt["a"], eps)).abs().max() < tol * 4
        wide = torch.zeros(T, W + 12, device=DEV)
        wide[:, :W] = y.to(DEV)
        for post, pre, src in (("a", "b", y.to(DEV)), ("a", "c", wide[:, :W]), ("c", "a", y.to(DEV)), ("b", None, wide[:, :W])):
            buf, h = x.to(DEV).clone(), torch.empty(T, W, dtype=dt, device=DEV)
            norm[post].enter(src, buf, None if pre is None else norm[pre], h)
            want = x.double() + plain[post](y.double())
            assert (buf.cpu().double() - want).abs().max() < 4e-6 * want.abs().max()
            if pre is not None:
                assert (h.cpu().double() - plain[pre](want)).abs().max() < tol * plain[pre](want).abs().max()


@pytest.mark.parametrize("T,W,k", [(17, 54, 3), (9, 64, 1), (5, 1024, 8), (4, 1500, 6), (3, 2052, 5), (6, 33, 2)])
def test_the_experts_sum_enters_through_a_norm(T, W, k):
    """Rows of the chosen experts by their lists, the norm after, the residual sum and the norm before: one kernel."""
    g = torch.Generator().manual_seed(k)
    idx, wt, h = torch.zeros(T, k).int(), torch.rand(T, k, generator=g), rn(g, T, W).bfloat16()
    ye, ros = rn(g, T * k, W), torch.randperm(T * k, generator=g).view(T, k).int()
    total = ye.double()[ros.long()].sum(1)
    from cpi_b200.parts.base import ExpertSum
    es = ExpertSum(ye.to(DEV), ros.to(DEV), idx.to(DEV), wt.to(DEV), h.to(DEV), 4)
    Wt = {"a": rn(g, W, std=0.3), "b": rn(g, W, std=0.3)}
    n = {x: build("norm", "rmsnorm", {"size": W, "eps": 1e-5, "weight": x, "weight_offset": 1.0}, Wt) for x in "ab"}
    x, out = rn(g, T, W), torch.empty(T, W, device=DEV)
    buf = x.to(DEV).clone()
    n["a"].enter(es, buf, n["b"], out)
    want = x.double() + P.norm_about_one(total, Wt["a"], 1e-5)
    assert (buf.cpu().double() - want).abs().max() < 2e-5
    assert (out.cpu().double() - P.norm_about_one(want, Wt["b"], 1e-5)).abs().max() < 4e-5


@pytest.mark.parametrize("H,D,Dv,run", [(3, 10, 14, 0), (3, 10, 14, 7), (1, 1, 1, 16), (8, 32, 16, 33), (2, 64, 128, 64), (4, 128, 128, 50),
                                        (2, 200, 24, 20), (1, 300, 20, 100), (5, 48, 36, 0), (2, 16, 70, 3)])
def test_recurrence_with_constant_decays(H, D, Dv, run):
    """The kernel alone: decays of zero, small, near one and one; a sequence whole, in portions (down to one token), beside
    other sequences of other lengths, cut into runs that are scanned side by side (a last run that is short, sequences
    with fewer runs than others) and not cut; silu in the kernel and before it; entry states that are not zero."""
    g = torch.Generator().manual_seed(D + Dv)
    T, T2 = 150, 31
    decay = torch.tensor(([0.999, 0.0, 1.0, 0.31, 0.95, 0.5, 0.99, 0.9995])[:H])
    C = 2 * H * D + H * Dv
    rows, rows2 = rn(g, T, C + 4, std=1.5), rn(g, T2, C + 4)
    S0 = rn(g, 3, H, D, Dv)

    def plain(r, S):
        q, k, v = (P.silu(r[:, a:b].double()) for a, b in ((0, H * D), (H * D, 2 * H * D), (2 * H * D, C)))
        n = r.shape[0]
        return P.decayed_sum(q.view(n, H, D), k.view(n, H, D), v.view(n, H, Dv), decay, S)

    want, end = plain(rows, S0[2])
    want2, end2 = plain(rows2, S0[0])
    for cuts in ([T], [100, 1, 2, 40, 7], [64, 86]):
        for ready in (False, True):
            state, outs, at = S0.to(DEV).clone(), [], 0
            for i, n in enumerate(cuts):
                b = FakeBatch([0, 2], [0, at], [T2, n]) if i == 0 else FakeBatch([2], [at], [n])
                x = (torch.cat([rows2, rows[:n]]) if i == 0 else rows[at:at + n]).to(DEV)
                if ready:
                    K().silu_rows(x[:, :C])
                    assert torch.equal(x[:, C:].cpu(), (torch.cat([rows2, rows[:n]]) if i == 0 else rows[at:at + n])[:, C:])
                o = torch.empty(x.shape[0], H * Dv, device=DEV)
                scratch = torch.full((b.n_seqs * (-(-b.max_new // run) if run else 1), H * D * Dv), float("nan"), device=DEV)
                K().linear_scan(x[:, H * D:2 * H * D], x[:, :H * D], x[:, 2 * H * D:C], state, o, b, n_heads=H, heads_per_group=1,
                                n_rows=D, n_cols=Dv, decay=decay.to(DEV), silu=not ready, run_state=scratch, run_len=run)
                if i == 0:
                    assert (o[:T2].cpu().double().view(T2, H, Dv) - want2).abs().max() < 2e-5 * want2.abs().max()
                    o = o[T2:]
                outs.append(o)
                at += n
            got = torch.cat(outs).cpu().double().view(T, H, Dv)
            assert (got - want).abs().max() < 2e-5 * want.abs().max(), (cuts, ready)
            assert (state[2].cpu().double() - end).abs().max() < 2e-5 * end.abs().max()
            assert (state[0].cpu().double() - end2).abs().max() < 2e-5 * end2.abs().max()
            assert torch.equal(state[1].cpu(), S0[1])


@pytest.mark.parametrize("H,D,Dv", [(4, 128, 128), (8, 32, 16), (1, 8, 8), (3, 24, 40), (2, 16, 200), (40, 64, 128), (2, 120, 48), (6, 56, 72)])
def test_chunked_recurrence_on_the_tensor_cores(H, D, Dv):
    """The same recurrence from bfloat16 rows, in chunks: whole, in portions that end inside chunks (down to one token),
    beside sequences that are shorter than a chunk and that end on one, from entry states that are not zero.  The state and
    the outputs are as exact as float32 sums are."""
    g = torch.Generator().manual_seed(D * 3 + Dv)
    lens, T = (31, 64), 210
    decay = torch.tensor([(0.999, 0.0, 1.0, 0.31, 0.95, 0.5, 0.99, 0.9995)[h % 8] for h in range(H)])
    C = H * (2 * D + Dv)
    rows = rn(g, T, C + 8, std=1.2).bfloat16()
    other = [rn(g, n, C + 8, std=1.2).bfloat16() for n in lens]
    S0 = rn(g, 4, H, D, Dv)

    def plain(r, S):
        n, x = r.shape[0], r.double()
        return P.decayed_sum(x[:, :H * D].view(n, H, D), x[:, H * D:2 * H * D].view(n, H, D), x[:, 2 * H * D:C].view(n, H, Dv), decay, S)

    (want, end), beside = plain(rows, S0[2]), [plain(r, S0[s]) for r, s in zip(other, (3, 0))]
    assert K().lightning_chunks_supported(D, Dv) and not K().lightning_chunks_supported(D + 4, Dv)
    close = lambda a, b: ((a.cpu().double() - b).abs().max() < 1e-5 * b.abs().max())
    for cuts in ([T], [100, 1, 2, 70, 37], [64, 146]):
        state, outs, at = S0.to(DEV).clone(), [], 0
        for i, n in enumerate(cuts):
            b = FakeBatch([3, 2, 0], [0, at, 0], [lens[0], n, lens[1]]) if i == 0 else FakeBatch([2], [at], [n])
            x = (torch.cat([other[0], rows[:n], other[1]]) if i == 0 else rows[at:at + n]).to(DEV)[:, :C]
            o = torch.empty(x.shape[0], H * Dv, device=DEV)
            K().lightning_chunks(x, decay.to(DEV), state, o, b, n_heads=H, n_rows=D, n_cols=Dv)
            if i == 0:
                assert close(o[:lens[0]].view(-1, H, Dv), beside[0][0]) and close(o[-lens[1]:].view(-1, H, Dv), beside[1][0])
                o = o[lens[0]:-lens[1]]
            outs.append(o)
            at += n
        assert close(torch.cat(outs).view(T, H, Dv), want), cuts
        assert close(state[2], end) and close(state[3], beside[0][1]) and close(state[0], beside[1][1])
        assert torch.equal(state[1].cpu(), S0[1])


@pytest.mark.parametrize("W,H,D,Dv,dtype", [(54, 3, 10, 14, "float32"), (64, 8, 32, 16, "bfloat16"), (128, 2, 64, 128, "bfloat16"),
                                            (40, 1, 1, 1, "float32")])
def test_lightning_mixer_alone(W, H, D, Dv, dtype):
    """Projections, recurrence, the norm over all heads together, gate and output; with the chunked kernel (bfloat16), in
    runs, and token by token."""
    from cpi_b200.parts import recurrent as R
    g = torch.Generator().manual_seed(W + D)
    dt = getattr(torch, dtype)
    T = 300
    m = V.lightning(H, D, Dv)
    Wt = {n: rn(g, r, W, std=1.5 * W ** -0.5).bfloat16() for n, r in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv))}
    Wt["norm"], Wt["o"] = rn(g, H * Dv, std=0.3, mean=1.0).bfloat16(), rn(g, W, H * Dv, std=(H * Dv) ** -0.5).bfloat16()
    part = build("mixer", "lightning", {"hidden_size": W, "heads": H, "key_dim": D, "value_dim": Dv, "decay": m["decay"],
                                        "norm_eps": 1e-5, "tensor_names": {n: n for n in Wt}}, Wt)
    h = rn(g, T, W).to(dt)
    want = P.lightning_mixer(h.double(), Wt, "", m, 1e-5)

    class Cache:
        def __init__(self):
            self.s = torch.zeros(1, H, D, Dv, device=DEV)

        def state(self, name):
            return self.s

    tol = 2e-5 if dtype == "float32" else 2e-2
    assert part.run_length(1, T) > 0 and part.run_length(1, 1) == 0
    for how in ("chunks", "runs", "tokens"):
        cache, out, at = Cache(), [], 0
        R.use_chunked_kernel = how == "chunks"
        if how == "tokens":
            part.run_length = lambda n, t: 0
        try:
            for n in (260, 2, 1, 37):
                o = torch.empty(n, W, device=DEV)
                part.forward(h[at:at + n].to(DEV), o, FakeBatch([0], [at], [n]), cache, add=False)
                out.append(o)
                at += n
        finally:
            R.use_chunked_kernel = True
        d = (torch.cat(out).cpu().double() - want).abs().max()
        assert d < tol * want.abs().max(), how


@pytest.mark.parametrize("W,parts", [(54, 1), (1000, 1), (1024, 1), (1028, 1), (2052, 1), (4096, 1), (8192, 1), (8196, 1), (4096, 4), (3072, 2), (6, 3)])
def test_norm_and_gate_over_rows_of_several_widths(W, parts):
    """The norm that follows the recurrence, gate after it and before it, silu and sigmoid, one weight per element or shared
    by the parts: narrow rows and wide ones, which take a kernel of their own, gates that are a slice of wider rows."""
    g = torch.Generator().manual_seed(W)
    T, eps, n = 5, 1e-2, W // parts
    y, gate = rn(g, T, W, std=0.3), rn(g, T, W + 8, std=2.0)
    for wlen in {W, n}:
        w = rn(g, wlen, std=0.3, mean=1.0)
        full = w.double().repeat(W // wlen)
        for act, f in (("sigmoid", torch.sigmoid), ("silu", P.silu)):
            a = f(gate[:, 8:].double())
            for first in (False, True):
                v = y.double() * a if first else y.double()
                want = P.rms(v.view(T, parts, n), eps).reshape(T, W) * full * (1.0 if first else a)
                for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 6e-3)):
                    out = torch.empty(T, W, dtype=dt, device=DEV)
                    K().gated_norm(y.to(DEV), gate.to(DEV)[:, 8:], w.to(DEV), out, parts=parts, gate_first=first, eps=eps, gate_act=act)
                    assert (out.cpu().double() - want).abs().max() < tol * want.abs().max(), (act, first, dt)


@pytest.mark.parametrize("H,G,D,Dv,dims", [(4, 2, 64, 64, 32), (8, 4, 128, 128, 96), (6, 2, 10, 14, 6), (2, 1, 128, 128, 128), (3, 1, 24, 16, 8),
                                           (2, 2, 16, 40, 0), (5, 1, 8, 8, 8)])
def test_rotation_of_part_of_a_head_into_the_pages(H, G, D, Dv, dims):
    """Queries turned, keys turned and values as they are into the pages of their positions: the fused kernel without a
    convolution where its sizes allow it, and the separate one."""
    g = torch.Generator().manual_seed(D + H)
    T, page, start = 90, 64, 40
    C = (H + G) * D + G * Dv
    u = rn(g, T, C + 4, std=1.5)
    f = P.frequencies(dims, 5e5, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 256})
    pos = torch.arange(start, start + T)
    q, k, v = u[:, :H * D].double().view(T, H, D), u[:, H * D:(H + G) * D].double().view(T, G, D), u[:, (H + G) * D:C].view(T, G, Dv)
    q, k = P.turn(q, pos, f), P.turn(k, pos, f)
    table = torch.tensor([[0, 0, 0], [7, 2, 3]], dtype=torch.int32, device=DEV)
    fd = f.float().to(DEV) if dims else None
    supported = K().qkv_conv_rotate_supported(D, Dv, dims, False, 1)
    assert supported == (D % 8 == 0 and Dv % 8 == 0 and dims % 8 == 0)
    for fused in ([True, False] if supported else [False]):
        for cuts in ([T], [1] * 5 + [84, 1]):
            kc, vc, at = torch.zeros(8, G, page, D, device=DEV), torch.zeros(8, G, page, Dv, device=DEV), 0
            out = torch.empty(T, H * D, device=DEV)
            for n in cuts:
                b = FakeBatch([1], [start + at], [n], tile=48)
                kw = dict(n_heads=H, n_kv_heads=G, head_dim=D, value_dim=Dv, inv_freq=fd, rotary_dims=dims)
                rows, o = u[at:at + n].to(DEV)[:, :C], torch.empty(n, H * D, device=DEV)
                if fused:
                    K().qkv_conv_rotate(rows, o, kc, vc, table, page, b, **kw)
                else:
                    K().qkv_prepare(rows, o, kc, vc, table, page, b.token_seq, b.token_pos, b.seq_slot, **kw)
                out[at:at + n] = o
                at += n
            assert (out.cpu().double().view(T, H, D) - q).abs().max() < 1e-4
            for t in range(T):
                pg, at = int(table[1, (start + t) // page]), (start + t) % page
                assert (kc[pg, :, at].cpu().double() - k[t]).abs().max() < 1e-4 and torch.equal(vc[pg, :, at].cpu(), v[t])


@pytest.mark.parametrize("T,W,E,top,ff,dtype", [(5, 54, 5, 3, 20, "float32"), (300, 64, 16, 4, 96, "bfloat16"), (7, 64, 12, 4, 96, "bfloat16"),
                                                (1, 128, 8, 1, 64, "bfloat16"), (6, 33, 4, 4, 16, "float32"), (40, 30, 3, 2, 9, "bfloat16"),
                                                (600, 256, 6, 2, 256, "bfloat16"), (90, 40, 1, 1, 8, "float32"), (33, 72, 200, 6, 8, "bfloat16")])
def test_routed_part_without_gates(T, W, E, top, ff, dtype):
    """Added into rows and handed over as a sum: sorted rows or gathered ones, few tokens in one launch or many in several,
    the float32 pipe and the tensor-core products; experts that no token chose; weights that do not sum to one."""
    g = torch.Generator().manual_seed(T + W)
    dt = getattr(torch, dtype)
    Wt = {"router": rn(g, E, W, std=2.5 * W ** -0.5).bfloat16()}
    for e in range(E):
        Wt[f"e{e}.up"], Wt[f"e{e}.down"] = rn(g, ff, W, std=2.0 * W ** -0.5).bfloat16(), rn(g, W, ff, std=2.0 * ff ** -0.5).bfloat16()
    part = build("feed_forward", "moe_mlp", {
        "hidden_size": W, "num_experts": E, "top_k": top, "expert_size": ff, "activation": "relu_squared", "router_gate": "scored",
        "router_name": "router", "expert_layout": "per_expert", "router_rule": {"score": "softmax", "normalise": False},
        "expert_names": {n: "e{e}." + n for n in ("up", "down")}}, Wt)
    mlp = {"expert": {"ff": ff}, "router": {"experts": E, "top": top}}
    h, res, own = rn(g, T, W).to(dt), rn(g, T, W), []
    want = P.routed_ff(h.double(), Wt, "", mlp, own=own)
    part.capture = []
    buf = res.to(DEV).clone()
    part.forward(h.to(DEV), buf, None)
    assert [sorted(x) for x in part.capture[0].cpu().tolist()] == own
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert (buf.cpu().double() - res.double() - want).abs().max() < tol * want.abs().max()
    out = part.expert_sum(h.to(DEV), None).rows(part.ws)
    assert (out.cpu().double() - want).abs().max() < tol * want.abs().max()


# ---- the model -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts_and_token_by_token(models, name, dtype):
    """A prompt in one step with logits everywhere, and the same tokens one by one from the first: both are the plain
    implementation's, which knows no cache and no state."""
    b = models[name]
    toks = V.tokens(150, b.cfg["vocab"], 5)
    r = Run(b.engine(dtype))
    r.step([("whole", toks, range(len(toks)))])
    r.end("whole")
    for i, t in enumerate(toks[:90]):
        r.step([("single", [t], [0])])
    r.check(b, {"whole": toks, "single": toks}, TOL[dtype])


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions_of_several_sizes(models, name):
    """A prompt cut into portions of 2, 3, 64, 1, 17, ... tokens and one long enough for the recurrence's runs, with cuts
    inside pages and windows; in float32 the logits are also those of the single step, to rounding."""
    b = models[name]
    toks = V.tokens(340, b.cfg["vocab"], 6)
    for dtype in ("float32", "bfloat16"):
        e = b.engine(dtype)
        r = Run(e)
        at = 0
        for n in (2, 3, 64, 1, 17, 2, 70, 5, 36, 140):
            r.step([("p", toks[at:at + n], range(n))])
            at += n
        assert at == 340
        r.check(b, {"p": toks}, TOL[dtype])
        if dtype == "float32":
            one = Run(e)
            one.step([("w", toks, range(340))])
            d = err(torch.stack([r.logits["p"][i] for i in range(340)]), torch.stack([one.logits["w"][i] for i in range(340)]))
            assert d < 5e-5, d


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_batches_in_reused_slots(models, name, dtype):
    """Requests of 1 to 190 tokens start together, are decoded together, end at different steps; a second group then
    runs in the slots and pages the first gave back.  Every logit is the request's own: nothing of a slot's earlier state
    or pages shows."""
    b = models[name]
    vocab = b.cfg["vocab"]
    reqs = {f"r{i}": V.tokens(n, vocab, 60 + i) for i, n in enumerate((1, 75, 190, 9, 66, 140))}
    e = b.engine(dtype, max_seqs=3, max_tokens=640)
    r = Run(e)
    for group in (("r0", "r1", "r2"), ("r3", "r4", "r5")):
        head = {i: max(1, len(reqs[i]) - 20) for i in group}
        r.step([(i, reqs[i][:head[i]], [0, head[i] - 1]) for i in group])
        live, k = [i for i in group if head[i] < len(reqs[i])], 0
        for i in group:
            if i not in live:
                r.end(i)
        while live:
            r.step([(i, [reqs[i][head[i] + k]], [0]) for i in live])
            k += 1
            for i in [i for i in live if head[i] + k == len(reqs[i])]:
                r.end(i)
                live.remove(i)
        e.cache.check_consistency()
    assert e.cache.free_slots == 3 and all(g.pages_held() == 0 for g in e.cache.groups)
    r.check(b, reqs, TOL[dtype])


@pytest.mark.parametrize("name", ["A", "B"])
def test_steps_larger_than_the_engine_takes_run_as_pieces(models, name):
    b = models[name]
    vocab = b.cfg["vocab"]
    reqs = {"x": V.tokens(123, vocab, 80), "y": V.tokens(8, vocab, 81), "z": V.tokens(66, vocab, 82)}
    for dtype in ("float32", "bfloat16"):
        r = Run(b.engine(dtype, max_step_tokens=50, max_seqs=3, max_tokens=512))
        r.step([("x", reqs["x"][:120], range(0, 120, 7)), ("y", reqs["y"][:7], [0, 6]), ("z", reqs["z"][:64], [1, 49, 50, 63])])
        r.step([("x", reqs["x"][120:121], [0]), ("y", reqs["y"][7:8], [0]), ("z", reqs["z"][64:65], [0])])
        r.end("y")
        r.step([("x", reqs["x"][121:123], [0, 1]), ("z", reqs["z"][65:66], [0])])
        r.check(b, reqs, TOL[dtype])


def _stand_out(W, layer, tokens, m, source=None):
    """Makes the keys of `tokens` stand out for every query that may see them.  Every token's embedding gets the same
    large element 1 and a small element 0, those of `tokens` a large element 0.  Attention: the last element of every q
    head (outside the rotated part) reads element 1, that of every k head element 0.  Latent attention: the last element
    of the queries' latent reads element 1, that of the cached latent (of `source`, the layer that has it) element 0,
    and the last plain element of every head's query and key reads those."""
    W["embed"][:, 0], W["embed"][:, 1] = 0.05, 3.0
    for token in tokens:
        W["embed"][token, 0] = 6.0
    W["l0.norm1"][:2] = 0.0
    pre = f"l{layer}.mix."

    def row(name, r, col, value, pre=pre):
        W[pre + name][r] = 0.0
        W[pre + name][r, col] = value

    if "kv_rank" in m:
        row("dq", m["q_rank"] - 1, 1, 8.0)
        row("dkv", m["kv_rank"] - 1, 0, 8.0, f"l{layer if source is None else source}.mix.")
        for h in range(m["heads"]):
            row("uq", (h + 1) * (m["dim"] + m["rot_dim"]) - m["rot_dim"] - 1, m["q_rank"] - 1, 3.0)
            row("uk", (h + 1) * m["dim"] - 1, m["kv_rank"] - 1, 1.5)
        return
    for name, heads, col in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        for h in range(heads):
            row(name, (h + 1) * m["dim"] - 1, col, 4.0)


@pytest.mark.parametrize("D,Dv,dims", [(8, 6, 4), (64, 64, 32), (128, 128, 64)])
def test_edges_of_the_window_and_of_the_kept_tokens(tmp_path, D, Dv, dims):
    """One layer: the keys at positions 0, 2, 3, 5, 62 .. 65, 127 and 128 stand out.  A query gives such a key most of its
    weight while it is inside the window or among the kept first tokens, and none of it one token further; in a prompt
    and token by token, for windows and kept counts that put the edges on a page border, before it and after it; on the
    general and on the tensor-core kernels."""
    special = (7, 9, 11, 13, 15, 17, 19, 21, 23, 25)
    toks = [t if t not in special else 8 for t in V.tokens(220, 50, 9)]
    for p, t in zip((0, 2, 3, 5, 62, 63, 64, 65, 127, 128), special):
        toks[p] = t
    last = []
    variants = ((64, None), (64, 3), (64, 4), (63, 1), (65, 6), (1, 63), (20, 64), (20, 65), (90, 128), (None, None))
    for window, keep in variants:
        m = V.attention(2, 1, D, Dv, dims, window=window, keep=keep, scale=4.0 / D)
        b = Built(V.model([V.layer(m, None)], width=24, vocab=50), 31, tmp_path, lambda W: _stand_out(W, 0, special, m))
        for dtype in ("float32", "bfloat16"):
            e = b.engine(dtype)
            r = Run(e)
            r.step([("x", toks[:126], range(126))])
            for i in range(126, 220):
                r.step([("x", toks[i:i + 1], [0])])
            r.check(b, {"x": toks}, TOL[dtype])
        last.append(b.plain(toks))
    for i in range(1, len(last)):                           # the variants do differ where the edges moved
        for j in range(i):
            assert (last[i] - last[j]).abs().max() > 1e-2, (variants[i], variants[j])


@pytest.mark.parametrize("rank,rot,kind", [(11, 4, "own"), (48, 16, "own"), (11, 4, "read"), (48, 16, "read"), (64, 32, "read")])
def test_one_position_that_stands_out_in_a_latent(tmp_path, rank, rot, kind):
    """Latent attention in which a token that occurs once, at position 2, is large in the cached latent: every later query
    gives that position most of its weight, hundreds of positions and several pages later -- in the layer that wrote the
    latent, or in a later one that only reads it (behind a recurrent layer, with other head counts)."""
    own = V.latent(2, 6, rot, 8, 12, rank, scale=0.3)
    layers = [V.layer(own, V.moe(3, 2, 16))]
    if kind == "read":
        layers += [V.layer(V.lightning(2, 8, 8), None), V.layer(V.latent(3, 10, rot, 6, 9, rank, kv_from=0, scale=0.3), None)]
    m = layers[-1]["mixer"]

    def change(W):
        _stand_out(W, len(layers) - 1, (7,), m, 0)
        if kind == "read":                     # what the reading layer's queries look at stays in the residual
            for n in ("l0.norm1b", "l0.norm2b", "l1.norm1b"):
                W[n][:2] = -1.0
            W["l2.norm1"][:2] = 0.0
    b = Built(V.model(layers, width=32, vocab=40), 3, tmp_path, change)
    toks = [t if t != 7 else 8 for t in V.tokens(330, 40, 1)]
    toks[2] = 7
    other = list(toks)
    other[2] = 9
    assert (b.plain(other)[300:] - b.plain(toks)[300:]).abs().max() > 1e-2      # the far token does matter to late rows
    for dtype in ("float32", "bfloat16"):
        r = Run(b.engine(dtype, max_tokens=512, max_seqs=2))
        r.step([("x", toks[:290], [0, 1, 2, 3, 63, 64, 65, 128, 289])])
        for i in range(290, 330):
            r.step([("x", toks[i:i + 1], [0])])
        r.check(b, {"x": toks}, TOL[dtype])


def test_the_sink_takes_its_share(tmp_path):
    """Scores near zero and sinks from far below to far above them, on the general and the tensor-core kernel; a sink of a
    size that leaves next to nothing, and one that cannot be told from none."""
    for rank, rot in ((10, 4), (64, 32)):
        m = V.latent(4, 8, rot, 16, 12, rank, scale=0.02)
        outs = []
        for sink in ([-40.0] * 4, [0.0, 1.0, 3.0, 6.0]):
            b = Built(V.model([V.layer(m, None)], width=32, vocab=40), 5, tmp_path,
                      lambda W: W.update({"l0.mix.sink": torch.tensor(sink).bfloat16()}))
            toks = V.tokens(100, 40, 3)
            for dtype in ("float32", "bfloat16"):
                r = Run(b.engine(dtype, max_tokens=512, max_seqs=2))
                r.step([("x", toks[:80], range(80))])
                for i in range(80, 100):
                    r.step([("x", toks[i:i + 1], [0])])
                r.check(b, {"x": toks}, TOL[dtype])
            outs.append(b.plain(toks))
        assert (outs[0] - outs[1]).abs().max() > 0.1


@pytest.mark.parametrize("name", ["A", "B"])
def test_a_far_token_among_hundreds_and_long_decoding(models, name):
    """700 tokens: the latent layers read every position back to the first across many pages while the windowed layers give
    their pages back but for the kept ones, through 120 decoded tokens."""
    b = models[name]
    toks = V.tokens(700, b.cfg["vocab"], 17)
    for dtype in ("float32", "bfloat16"):
        e = b.engine(dtype, max_tokens=1024, max_seqs=2)
        r = Run(e)
        r.step([("far", toks[:580], [0, 1, 300, 579])])
        for i in range(580, 700):
            r.step([("far", toks[i:i + 1], [0])])
        r.check(b, {"far": toks}, TOL[dtype])
        windowed = [g for g in e.cache.groups if g.req.window_kind == "sliding"]
        assert windowed and all(g.pages_held() <= -(-g.req.window_size // 64) + 1 + -(-g.req.keep_first // 64) for g in windowed)


def test_fused_and_separate_kernels_agree(models):
    """The fused preparation, the tensor-core attention kernels and the chunked recurrence, and the separate and general
    ones, in bfloat16: both give the plain implementation's logits (with the choices of experts that each of them made)."""
    from cpi_b200.parts import attention as A, recurrent as R
    b = models["B"]
    toks = V.tokens(300, b.cfg["vocab"], 3)
    for on in (True, False):
        A.use_tensor_core_kernels = A.use_fused_preparation = R.use_chunked_kernel = on
        try:
            r = Run(b.engine("bfloat16", max_tokens=1024, max_seqs=2))
            r.step([("x", toks[:200], range(0, 200, 7))])
            r.step([("x", toks[200:260], range(60))])
            for i in range(260, 300):
                r.step([("x", toks[i:i + 1], [0])])
            r.check(b, {"x": toks}, TOL["bfloat16"])
        finally:
            A.use_tensor_core_kernels = A.use_fused_preparation = R.use_chunked_kernel = True


def test_other_constants_change_the_result_as_the_plain_implementation_says(tmp_path):
    base = V.model([V.layer(V.latent(2, 6, 8, 10, 9, 12, base=20.0), V.moe(4, 2, 10)),
                    V.layer(V.lightning(2, 6, 8, decay=(0.9, 0.4)), V.moe(6, 2, 12)),
                    V.layer(V.latent(3, 4, 8, 6, 7, 12, kv_from=0, base=20.0), None),
                    V.layer(V.attention(4, 2, 8, 12, 4, window=9, keep=2, base=100.0, scaling=(4.0, 1.0, 4.0, 64)), V.moe(3, 1, 16))],
                   width=36, vocab=70)
    lat, lin, read, att = ((lambda c, i=i: c["layers"][i]["mixer"]) for i in range(4))
    ff = lambda c: c["layers"][1]["mlp"]
    sc = lambda c: att(c)["rot"]["scaling"]

    def both(**kw):
        return lambda c: (lat(c)["rot"].update(kw), read(c)["rot"].update(kw))
    same_weights = {
        "eps": lambda c: c["norm"].update(eps=0.3), "decay": lambda c: lin(c).update(decay=[0.4, 0.9]),
        "no_decay": lambda c: lin(c).update(decay=[1.0, 1.0]), "all_decay": lambda c: lin(c).update(decay=[0.0, 0.0]),
        "lat_base": both(base=1000.0), "lat_scale": lambda c: lat(c).update(scale=0.1), "read_scale": lambda c: read(c).update(scale=0.1),
        "window": lambda c: att(c)["mask"].update(size=8), "keep": lambda c: att(c)["mask"].update(keep_first=3),
        "no_keep": lambda c: att(c)["mask"].pop("keep_first"), "no_window": lambda c: att(c).pop("mask"),
        "base": lambda c: att(c)["rot"].update(base=1000.0), "dims": lambda c: att(c)["rot"].update(dims=8),
        "no_rot": lambda c: att(c).pop("rot"), "scale": lambda c: att(c).update(scale=0.3),
        "no_scaling": lambda c: att(c)["rot"].pop("scaling"), "factor": lambda c: sc(c).update(factor=16.0),
        "original": lambda c: sc(c).update(original=16), "low": lambda c: sc(c).update(low=3.0), "high": lambda c: sc(c).update(high=60.0),
        "top": lambda c: ff(c)["router"].update(top=1), "all": lambda c: ff(c)["router"].update(top=6),
        "no_mlp": lambda c: c["layers"][0].update(mlp=None),
    }
    other_weights = {
        "kv_heads": lambda c: att(c).update(kv_heads=4), "vdim": lambda c: att(c).update(vdim=8), "experts": lambda c: ff(c)["router"].update(experts=9),
        "own_latent": lambda c: read(c).pop("kv_from"), "ranks": lambda c: (lat(c).update(kv_rank=16, q_rank=5), read(c).update(kv_rank=16)),
        "heads": lambda c: lin(c).update(heads=3, decay=[0.2, 0.5, 0.99]), "rest_first": lambda c: c.update(layers=[c["layers"][i] for i in (0, 2, 3, 1)]),
    }
    toks = V.tokens(40, 70, 2)
    W0 = V.draw_weights(base, 21)
    ref = P.forward(base, W0, toks)
    for key, change in {**same_weights, **other_weights}.items():
        cfg = copy.deepcopy(base)
        change(cfg)

        def keep(W):
            if key in same_weights:
                for n in W:
                    W[n] = W0[n]
        b = Built(cfg, 21, tmp_path, keep)
        r = Run(b.engine("float32"))
        r.step([("x", toks[:25], range(25))])
        for i in range(25, 40):
            r.step([("x", toks[i:i + 1], [0])])
        r.check(b, {"x": toks}, TOL["float32"])
        if key in same_weights:
            assert (b.plain(toks) - ref).abs().max() > 1e-3, key      # same weights, other constant


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12, 13, 14])
def test_configurations_drawn_from_a_seed(seed, tmp_path):
    """Every size, option and constant drawn from a seed: a prompt with logits everywhere, a second request in a
    portion and then both decoded together, in float32 to rounding and in bfloat16."""
    cfg = V.draw_config(seed)
    b = Built(cfg, 40 + seed, tmp_path)
    vocab = cfg["vocab"]
    ta, tb = V.tokens(170, vocab, seed), V.tokens(75, vocab, seed + 100)
    for dtype in ("float32", "bfloat16"):
        r = Run(b.engine(dtype, max_tokens=1024, max_seqs=2))
        r.step([("a", ta[:150], range(150)), ("b", tb[:3], range(3))])
        r.step([("b", tb[3:70], range(67))])
        for i in range(5):
            r.step([("a", ta[150 + i:151 + i], [0]), ("b", tb[70 + i:71 + i], [0])])
        r.end("b")
        for i in range(155, 170):
            r.step([("a", ta[i:i + 1], [0])])
        r.check(b, {"a": ta, "b": tb}, TOL[dtype])


def test_layers_recorded_one_by_one(models):
    """The residual after every layer is the plain implementation's."""
    b = models["A"]
    toks = V.tokens(30, b.cfg["vocab"], 4)
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 5e-2)):
        e = b.engine(dtype)
        e.model.layer_capture = []
        r = Run(e)
        r.step([("x", toks, [29])])
        want = []
        P.forward(b.cfg, b.W, toks, want, forced={n: [by[p] for p in range(30)] for n, by in r.routing.get("x", {}).items()})
        assert len(e.model.layer_capture) == len(want) == 6
        for got, w in zip(e.model.layer_capture, want):
            assert (got.cpu().double() - w).abs().max() < tol * w.abs().max()


def test_greedy_generation_through_the_entry_point(tmp_path):
    """`Model.generate` (scheduler, sampler, decode graphs) picks the plain implementation's tokens: unequal prompts,
    more requests than slots."""
    from cpi_b200.api import Model
    b = Built(V.MIXED_A, 11, tmp_path, V.strong_sublayers)
    vocab = b.cfg["vocab"]
    prompts = [V.tokens(n, vocab, 30 + n) for n in (5, 33, 1, 70, 12)]
    m = Model.load(b.dir, dtype="float32", max_batch=2, max_context=128)
    results = m.generate(prompts, max_new=12, temperature=0.0)
    for p, res in zip(prompts, results):
        seq = list(p)
        for tok in res.tokens:
            ref = b.plain(seq)[-1]
            best = int(ref.argmax())
            if tok != best:            # a near-tie may fall either way; anything else is a fault
                assert (ref[best] - ref[tok]).item() < 1e-3 * ref.abs().max().item(), (len(p), len(seq))
            seq.append(tok)
        assert len(res.tokens) == 12 and len(set(res.tokens)) > 5


def test_decode_steps_replayed_as_graphs_are_the_eager_ones(models):
    """Every part of the model says it is safe to capture; replayed decode steps give the eager steps' logits."""
    b = models["B"]
    toks = V.tokens(60, b.cfg["vocab"], 77)
    logits = []
    for graphs in (True, False):
        e = b.engine("bfloat16", max_seqs=2, max_tokens=256)
        assert e.use_graphs
        e.use_graphs = graphs
        r = Run(e, record=False)
        r.step([("g", toks[:40], [39])])
        for i in range(40, 60):
            r.step([("g", toks[i:i + 1], [0])])
        assert (e.graph_kernel_launches > 0) == graphs
        logits.append(r.logits["g"])
    for p in range(39, 60):
        assert torch.equal(logits[0][p], logits[1][p]), p


def test_random_weights_mode_and_command_line(models):
    """A folder drawn by the library's random mode loads and generates; bin/llama_infer knows the family by its
    config.json and its greedy tokens are the plain implementation's."""
    from cpi_b200.engine import Engine
    e = Engine.from_random(V.MIXED_B, seed=3, dtype="bfloat16", max_tokens=512)
    out = Run(e)
    out.step([("x", V.tokens(70, 384, 1), [69])])
    assert torch.isfinite(out.logits["x"][69]).all()
    b = models["C"]
    prompt = V.tokens(9, b.cfg["vocab"], 50)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "llama_infer"), b.dir, "--tokens",
                        ",".join(map(str, prompt)), "--max-new", "6", "--temp", "0", "--dtype", "float32",
                        "--benchmark-phases", "--max-context", "64"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    line = next(l for l in r.stdout.splitlines() if l.startswith("Output tokens:"))
    got = [int(x) for x in line.split(":")[1].split()]
    assert got[:9] == prompt and len(got) == 15
    seq = list(prompt)
    for tok in got[9:]:
        ref = b.plain(seq)[-1]
        best = int(ref.argmax())
        assert tok == best or (ref[best] - ref[tok]).item() < 1e-3 * ref.abs().max().item()
        seq.append(tok)
    assert "Delilorn" in r.stdout and "scan" in r.stdout


def test_replay_tool_runs_a_delilorn_folder(models, tmp_path):
    """bin/trace_run in a process of its own: a request whole, and two requests batched then decoded."""
    import numpy as np
    b = models["B"]
    vocab = b.cfg["vocab"]
    ta, tb = V.tokens(80, vocab, 40), V.tokens(21, vocab, 41)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta, "want": list(range(80))}], "end": ["a"]},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:20], "want": []},
                                     {"id": "a2", "tokens": ta[:70], "want": [69]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": tb[20:], "want": [0]},
                                     {"id": "a2", "tokens": ta[70:71], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a2", "tokens": ta[71:72], "want": [0]}], "end": ["a2"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", b.dir, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    rd = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, vocab).copy())
    got = torch.cat([rd(i) for i in range(4)])
    ra, rb = b.plain(ta), b.plain(tb)
    want = torch.cat([ra, torch.stack([ra[69], rb[20], ra[70], ra[71]])])
    assert got.shape == want.shape and err(got, want) < TOL["float32"]
