"""Nekorax through the engine against the plain implementation (`plain_nekorax.py`): every mechanism alone, whole
prompts, portions, token-by-token decoding, unequal batches, reused slots and pages, the edges of windows, far keys, the
first tokens of a sequence, long decoding, other sizes, generation through the entry point, and the replay tool."""
from __future__ import annotations

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import nekorax_tiny as V
import plain_nekorax as P
from family_run import DEV, Built as FamilyBuilt, FakeBatch, K, Run, build, err, rn

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-4, "bfloat16": 4e-2}
F64 = torch.float64


def Built(*args):
    return FamilyBuilt(V, P, *args)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("nekorax")
    return {"A": Built(V.MIXED_A, 11, tmp), "B": Built(V.MIXED_B, 12, tmp), "C": Built(V.MIXED_C, 13, tmp)}


# ---- mechanisms alone ------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,W,dt", [(5, 52, torch.float32), (70, 256, torch.bfloat16), (3, 37, torch.bfloat16), (9, 4104, torch.bfloat16)])
def test_tanh_norms_around_the_residual_sum(T, W, dt):
    """The norm alone (all rows, or listed ones), a sublayer's entry through its norm, and both in one launch."""
    g = torch.Generator().manual_seed(W)
    Wt = {}
    for n, alpha in (("a", 0.7), ("b", 1.9)):
        Wt[n], Wt[n + ".b"], Wt[n + ".alpha"] = rn(g, W, std=0.3, mean=1.0), rn(g, W, std=0.4), torch.tensor(alpha)
    norm = {n: build("norm", "dynamic_tanh", {"size": W, "weight": n, "alpha": n + ".alpha", "offset": n + ".b"}, Wt) for n in "ab"}
    x, y = rn(g, T, W, std=2.0), rn(g, T, W, std=2.0)
    tol = 2e-6 if dt == torch.float32 else 1e-2
    rows = [2, 0, 2]
    got = norm["a"](x.to(DEV), dt, rows=torch.tensor(rows, dtype=torch.int32, device=DEV)).cpu().double()
    assert (got - P.dynamic_tanh(x.double(), Wt, "a")[rows]).abs().max() < tol
    want = x.double() + P.dynamic_tanh(y.double(), Wt, "b")
    h = torch.empty(T, W, dtype=dt, device=DEV)
    for following in (norm["a"], None):
        buf = x.to(DEV).clone()
        norm["b"].enter(y.to(DEV), buf, following, h)
        assert (buf.cpu().double() - want).abs().max() < 2e-6 * want.abs().max()
    assert (h.cpu().double() - P.dynamic_tanh(want, Wt, "a")).abs().max() < tol * 2


@pytest.mark.parametrize("W,k,n_real", [(52, 3, 4), (64, 1, 2), (33, 6, 7)])
def test_sum_over_experts_and_identity_experts_enters_through_a_norm(W, k, n_real):
    """Rows of the chosen experts by their lists, weight * input for the chosen identity experts, in one launch with the
    norm after, the residual sum and the norm before the next sublayer; and with RMS norms, where they are separate."""
    g = torch.Generator().manual_seed(k)
    T = 17
    idx = torch.stack([torch.randperm(n_real + 3, generator=g)[:k] for _ in range(T)]).int()
    wt, h, ye = torch.rand(T, k, generator=g), rn(g, T, W).bfloat16(), rn(g, T * k, W)
    ros = torch.randperm(T * k, generator=g).view(T, k).int()
    total = torch.zeros(T, W, dtype=F64)
    for t in range(T):
        for j in range(k):
            total[t] += ye[ros[t, j]].double() if idx[t, j] < n_real else wt[t, j].double() * h[t].double()
    from cpi_b200.parts.base import ExpertSum
    es = ExpertSum(ye.to(DEV), ros.to(DEV), idx.to(DEV), wt.to(DEV), h.to(DEV), n_real)
    Wt = {"a": rn(g, W, mean=1.0), "a.b": rn(g, W), "a.alpha": torch.tensor(0.8), "r": rn(g, W, std=0.2, mean=1.0)}
    tanh = build("norm", "dynamic_tanh", {"size": W, "weight": "a", "alpha": "a.alpha", "offset": "a.b"}, Wt)
    rms = build("norm", "rmsnorm", {"size": W, "eps": 1e-5, "weight": "r"}, Wt)
    plain = {tanh: lambda v: P.dynamic_tanh(v, Wt, "a"), rms: lambda v: P.rms(v, 1e-5) * Wt["r"].double()}
    x = rn(g, T, W)
    for post in (tanh, rms):
        for pre in (tanh, rms):
            buf, out = x.to(DEV).clone(), torch.empty(T, W, device=DEV)
            post.enter(es, buf, pre, out)
            want = x.double() + plain[post](total)
            assert (buf.cpu().double() - want).abs().max() < 2e-5
            assert (out.cpu().double() - plain[pre](want)).abs().max() < 4e-5
    buf = x.to(DEV).clone()
    es.add_to(buf)
    assert (buf.cpu().double() - x.double() - total).abs().max() < 1e-5


def test_embedding_rows_are_scaled():
    g = torch.Generator().manual_seed(0)
    for W, dt in ((40, torch.bfloat16), (13, torch.float32)):
        table, toks = rn(g, 20, W).to(dt), torch.tensor([3, 0, 19, 3], dtype=torch.int32)
        out, flag = torch.empty(4, W, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
        K().embedding(toks.to(DEV), table.to(DEV), out, flag, 0.375)
        assert torch.equal(out.cpu(), table[toks.long()].float() * 0.375) and int(flag) == 0


@pytest.mark.parametrize("W,T,dt", [(52, 5, "float32"), (64, 40, "bfloat16"), (256, 600, "bfloat16")])
def test_a_pass_is_entered_through_its_matrix_and_its_vector(W, T, dt):
    g = torch.Generator().manual_seed(W)
    Wt = {"loop.in": rn(g, W, 2 * W, std=(2 * W) ** -0.5).bfloat16(), "loop.step": rn(g, 3, W).bfloat16()}
    x, x0 = rn(g, T, W), rn(g, T, W)

    class B:
        dtype = getattr(torch, dt)
    from cpi_b200.weights.store import DictSource
    src = DictSource(Wt)
    parts = [build("junction", "concat_linear", {"hidden_size": W, "weight": "loop.in", "step": "loop.step", "pass_index": t,
                                                 "passes": 3}, Wt) for t in range(3)]
    for p in parts:
        p.load(src, torch.device(DEV))
    assert parts[0].weight.data_ptr() == parts[2].weight.data_ptr()              # one copy of the matrix
    for t, p in enumerate(parts):
        buf = x.to(DEV).clone()
        p.run(buf, x0.to(DEV), B)
        want = torch.cat([x, x0], -1).double() @ Wt["loop.in"].double().T + Wt["loop.step"][t].double()
        assert (buf.cpu().double() - want).abs().max() < (1e-5 if dt == "float32" else 2e-2) * want.abs().max()


def _pages(T, page, n_pages, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randperm(n_pages, generator=g)[:-(-T // page)].tolist()


@pytest.mark.parametrize("H,G,D,Dv,dims,taps,inter", [(4, 2, 64, 64, 32, 4, False), (6, 2, 16, 8, 8, 3, False), (2, 1, 24, 40, 16, 8, True),
                                                      (1, 1, 8, 8, 8, 1, False), (2, 2, 128, 128, 64, 2, True), (3, 1, 10, 14, 6, 3, False),
                                                      (2, 1, 32, 64, 0, 5, False), (5, 1, 16, 16, 8, None, True), (1, 1, 256, 256, 256, 2, False)])
def test_preparation_with_convolution_and_values_that_turn(H, G, D, Dv, dims, taps, inter):
    """Rows [q | k | v | rest]: convolution, rotation of q and k, rotation of the values by their positions, into pages --
    the fused kernel where its sizes allow it, and the separate ones always: a sequence of 80 tokens whole, in portions
    shorter than the convolution, one by one at the end, beside another sequence, in a slot whose carried inputs another
    sequence left and that was zeroed on acquisition."""
    g = torch.Generator().manual_seed(H * 10 + D)
    T, T2, page, base = 80, 21, 64, 300.0
    C = (H + G) * D + G * Dv
    u, u2 = rn(g, T, C + 8, std=1.5), rn(g, T2, C + 8, std=1.5)
    w = None if taps is None else rn(g, C, taps, std=0.5, mean=0.3)
    fq = P.frequencies(dims, base)[0] if dims else None
    fv = P.frequencies(Dv, base)[0]
    layout = "interleaved" if inter else "halves"

    def plain(rows):
        r = rows[:, :C].double()
        r = r if w is None else P.short_conv(r, w)
        n, pos = r.shape[0], torch.arange(r.shape[0])
        q, k, v = r[:, :H * D].view(n, H, D), r[:, H * D:(H + G) * D].view(n, G, D), r[:, (H + G) * D:].view(n, G, Dv)
        if dims:
            q, k = P.turn(q, pos, fq, layout=layout), P.turn(k, pos, fq, layout=layout)
        return q, k, P.turn(v, pos, fv, layout=layout)

    want, want2 = plain(u), plain(u2)
    table = torch.tensor([[0, 0], [7, 0], [3, 1]], dtype=torch.int32, device=DEV)
    f32 = lambda t: None if t is None else t.float().to(DEV)
    supported = K().qkv_conv_rotate_supported(D, Dv, dims, True, taps or 1)
    assert supported == (D % 8 == 0 and Dv % 8 == 0 and dims % 8 == 0)
    for fused in ([True, False] if supported else [False]):
        for cuts in ([T], [2, 1, 3, 64, 1, 9], [1] * 5 + [70] + [1] * 5):
            kc, vc = torch.zeros(8, G, page, D, device=DEV), torch.zeros(8, G, page, Dv, device=DEV)
            carry = torch.randn(3, max((taps or 1) - 1, 0), C, device=DEV)
            carry[1:] = 0
            qs, at = [], 0
            for i, n in enumerate(cuts):
                first = i == 0
                b = FakeBatch([1, 2] if first else [2], [0, 0] if first else [at], [T2, n] if first else [n], tile=48)
                rows = (torch.cat([u2, u[:n]]) if first else u[at:at + n]).to(DEV)[:, :C]
                q = torch.empty(rows.shape[0], H * D, device=DEV)
                if fused:
                    K().qkv_conv_rotate(rows, q, kc, vc, table, page, b, n_heads=H, n_kv_heads=G, head_dim=D, value_dim=Dv,
                                        conv_weight=None if w is None else w.t().contiguous().to(DEV), carry=carry,
                                        inv_freq=f32(fq), rotary_dims=dims, v_inv_freq=f32(fv), interleaved=inter)
                else:
                    if w is not None:
                        out = torch.empty(rows.shape[0], C, device=DEV)
                        K().causal_conv(rows, w.to(DEV), None, carry, out, b, silu=False)
                        rows = out
                    K().qkv_prepare(rows, q, kc, vc, table, page, b.token_seq, b.token_pos, b.seq_slot, n_heads=H, n_kv_heads=G,
                                    head_dim=D, value_dim=Dv, inv_freq=f32(fq), rotary_dims=dims, interleaved=inter, v_inv_freq=f32(fv))
                if first:
                    assert (q[:T2].cpu().double().view(T2, H, D) - want2[0]).abs().max() < 1e-4
                    q = q[T2:]
                qs.append(q)
                at += n
            assert (torch.cat(qs).cpu().double().view(T, H, D) - want[0]).abs().max() < 1e-4, (fused, cuts[:3])
            for t in range(T):
                pg = int(table[2, t // page])
                assert (kc[pg, :, t % page].cpu().double() - want[1][t]).abs().max() < 1e-4
                assert (vc[pg, :, t % page].cpu().double() - want[2][t]).abs().max() < 1e-4
            if taps and taps > 1:
                assert torch.equal(carry[2].cpu(), u[T - taps + 1:, :C])
                assert torch.equal(carry[1].cpu(), u2[T2 - taps + 1:, :C])


@pytest.mark.parametrize("H,Dv,inter,dt", [(3, 14, False, torch.float32), (4, 64, False, torch.bfloat16), (2, 24, True, torch.float32),
                                           (8, 128, False, torch.bfloat16), (1, 2, True, torch.float32)])
def test_outputs_turned_back_and_gated(H, Dv, inter, dt):
    g = torch.Generator().manual_seed(Dv)
    for T in (5, 700):
        o, gate = rn(g, T, H * Dv).to(dt), rn(g, T, H * Dv + 8, std=2.0)
        pos = torch.randint(0, 3000, (T,), generator=g)
        f = P.frequencies(Dv, 500.0)[0]
        a32 = (pos.float()[:, None] * f.float()[None, :]).double()              # the angle as a 32-bit number
        turned = o.double().view(T, H, Dv).clone()
        c, s = torch.cos(a32)[:, None], torch.sin(a32)[:, None]
        i1, i2 = (slice(0, None, 2), slice(1, None, 2)) if inter else (slice(0, Dv // 2), slice(Dv // 2, Dv))
        x, y = turned[..., i1].clone(), turned[..., i2].clone()
        turned[..., i1], turned[..., i2] = x * c + y * s, y * c - x * s
        sg = torch.sigmoid(gate[:, 8:].double()).view(T, H, Dv)
        tol = 2e-6 if dt == torch.float32 else 1e-2
        kw = dict(n_heads=H, value_dim=Dv, interleaved=inter)
        posd, gd = pos.int().to(DEV), gate.to(DEV)[:, 8:]
        for freq, gt, want in ((f.float().to(DEV), gd, turned * sg), (f.float().to(DEV), None, turned), (None, gd, o.double().view(T, H, Dv) * sg)):
            buf = o.to(DEV).clone()
            K().head_turn(buf, buf, posd, inv_freq=freq, gate=gt, **kw)
            assert (buf.cpu().double().view(T, H, Dv) - want).abs().max() < tol * 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_constant_sink_is_a_one_in_the_denominator(dtype):
    """Through the attention kernels of both precisions and all their forms (prompt, single tokens, general): scores around
    zero, where the one matters most, and scores far above and far below it."""
    from cpi_b200.parts.attention import attend
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(2)
    T, H, G, D, page = 90, 4, 2, 64, 64
    for std in (0.1, 1.0, 4.0):
        q, k, v = rn(g, T, H, D, std=std).to(dt), rn(g, T, G, D).to(dt), rn(g, T, G, D).to(dt)
        kc, vc = torch.zeros(3, G, page, D, dtype=dt, device=DEV), torch.zeros(3, G, page, D, dtype=dt, device=DEV)
        table = torch.tensor([[2, 0]], dtype=torch.int32, device=DEV)
        for t in range(T):
            kc[int(table[0, t // page]), :, t % page] = k[t].to(DEV)
            vc[int(table[0, t // page]), :, t % page] = v[t].to(DEV)
        want = P.weighted_values(q.double(), k.double(), v.double(), 0.2, P.visible(T), True)
        without = P.weighted_values(q.double(), k.double(), v.double(), 0.2, P.visible(T), False)
        assert (want[0] - without[0]).abs().max() > 0.1
        for single in (False, True):
            out = torch.empty(T, H * D, dtype=dt, device=DEV)
            for rows in ([range(T)] if not single else [[t] for t in range(0, T, 13)]):
                b = FakeBatch([0], [rows[0]], [len(rows)])
                b.ctx_bucket = 256
                sl = slice(rows[0], rows[0] + len(rows))
                attend(q[sl].reshape(len(rows), H * D).to(DEV).contiguous(), out[sl], kc, vc, table, page, b, n_heads=H, n_kv_heads=G,
                       head_dim=D, value_dim=D, window_kind="full", window_size=0, scale=0.2, sink=torch.zeros(H, device=DEV))
            pick = list(range(T)) if not single else list(range(0, T, 13))
            d = (out.cpu().double().view(T, H, D) - want)[pick].abs().max() / want.abs().max()
            assert d < (1e-5 if dtype == "float32" else 1.5e-2), (std, single)


@pytest.mark.parametrize("H,row,rank,window", [(4, 112, 96, 50), (20, 192, 160, 1), (3, 80, 64, 32), (64, 96, 64, 33), (8, 96, 64, 31),
                                               (80, 48, 32, 64), (16, 576, 512, 100), (5, 160, 128, 0)])
def test_windowed_attention_over_the_cached_latent(H, row, rank, window):
    """The tensor-core kernel: prompts and portions in query tiles, single tokens with and without key splits, windows on,
    before and after the edges of key tiles and pages.  Pages that lie wholly before the window of a portion hold NaN:
    they may have been given back and must not be read."""
    g = torch.Generator().manual_seed(row + window)
    T, page, scale = 230, 64, 0.12
    q, c = rn(g, T, H, row).bfloat16(), rn(g, T, 1, row).bfloat16()
    c[:, :, :] = c * (1.0 + 3.0 * (torch.rand(T, 1, 1, generator=g) > 0.9)).bfloat16()       # some keys stand out
    ok = P.visible(T, window or None)
    kk, vv = c.double(), c[:, :, :rank].double()
    want = P.weighted_values(q.double(), kk, vv, scale, ok, False)
    pages = [5, 2, 7, 0]
    table = torch.tensor([pages], dtype=torch.int32, device=DEV)

    def cache(first_needed):
        kc = torch.full((8, 1, page, row), float("nan"), dtype=torch.bfloat16, device=DEV)
        for t in range(max(0, first_needed) // page * page, T):
            kc[pages[t // page], 0, t % page] = c[t, 0].to(DEV)
        for t in range(T, 4 * page):
            kc[pages[t // page], 0, t % page] = 0
        return kc

    def check(out, n, at):
        got = out.cpu().double().view(H, n, rank).transpose(0, 1)
        assert (got - want[at:at + n]).abs().max() < 2e-2 * want.abs().max(), at

    for start, n in ((0, T), (0, 3), (130, 100), (64, 2), (199, 31)):
        b = FakeBatch([0], [start], [n])
        out = torch.empty(H * n, rank, dtype=torch.bfloat16, device=DEV)
        K().latent_attention(q[start:start + n].reshape(n, H * row).to(DEV).contiguous(), out,
                             cache(start - window + 1 if window else 0), table, page, b.token_seq, b.token_pos, b.seq_slot,
                             n_heads=H, rank=rank, scale=scale, tile_tok0=b.tile_tok0, tile_rows=b.tile_rows, window=window)
        check(out, n, start)
    for at in (0, 1, 31, 32, 33, 63, 64, 65, 127, 128, 191, 192, 229):
        for splits in (1, 3):
            b = FakeBatch([0], [at], [1])
            out = torch.empty(H, rank, dtype=torch.bfloat16, device=DEV)
            K().latent_attention(q[at].reshape(1, H * row).to(DEV).contiguous(), out, cache(at - window + 1 if window else 0), table,
                                 page, b.token_seq, b.token_pos, b.seq_slot, n_heads=H, rank=rank, scale=scale, n_splits=splits,
                                 window=window)
            check(out, 1, at)


def test_latent_rows_and_queries_take_the_rotation_s_amplitude():
    g = torch.Generator().manual_seed(5)
    T, H, D, R, rank, page, eps, amp = 6, 3, 10, 6, 14, 64, 1e-5, 1.37
    f = P.frequencies(R, 300.0)[0]
    x, w = rn(g, T, rank + R, std=2.0), rn(g, rank, std=0.3, mean=1.0)
    b = FakeBatch([1], [62], [T])
    table = torch.tensor([[0, 0], [2, 3]], dtype=torch.int32, device=DEV)
    cache = torch.zeros(4, 1, page, rank + R, device=DEV)
    K().latent_kv_write(x.to(DEV), w.to(DEV), eps, f.float().to(DEV), True, cache, table, page, b.token_seq, b.token_pos,
                        b.seq_slot, rank=rank, rot=R, amplitude=amp)
    pos = torch.arange(62, 62 + T)
    want_r = P.turn(x[:, rank:].double().view(T, 1, R), pos, f, amp, "interleaved").view(T, R)
    for t in range(T):
        row = cache[int(table[1, (62 + t) // page]), 0, (62 + t) % page].cpu().double()
        assert (row[rank:] - want_r[t]).abs().max() < 3e-5
        assert (row[:rank] - P.rms(x[t, :rank].double(), eps) * w.double()).abs().max() < 2e-5
    q = rn(g, T, H * (D + R))
    plain, full = torch.empty(H * T, D, device=DEV), torch.zeros(T, H * (rank + R), device=DEV)
    offsets, rows = torch.empty(H + 1, dtype=torch.int32, device=DEV), torch.empty(H * T, dtype=torch.int32, device=DEV)
    K().latent_q_split(q.to(DEV), f.float().to(DEV), True, plain, full, offsets, rows, b.token_pos, n_heads=H, dim=D, rot=R,
                       rank=rank, amplitude=amp)
    want = P.turn(q.view(T, H, D + R)[..., D:].double(), pos, f, amp, "interleaved")
    assert (full.cpu().double().view(T, H, rank + R)[..., rank:] - want).abs().max() < 3e-5


@pytest.mark.parametrize("E,top,groups,keep,T", [(6, 2, 3, 2, 40), (16, 4, 4, 2, 300), (8, 3, 2, 1, 5), (5, 5, 1, 1, 9), (3, 1, 1, 1, 70),
                                                 (12, 2, 6, 1, 33), (64, 6, 8, 3, 20), (256, 8, 64, 5, 130), (40, 7, 40, 11, 64)])
def test_choice_of_experts_by_softmax_scores(E, top, groups, keep, T):
    """Scores softmax(z) over all experts; the choice on score + correction inside the kept groups (a group's score: its
    largest choice score); the weights are the scores, neither corrected nor normed.  Corrections are drawn so that they
    change the groups kept and the experts chosen, and so that choice scores are negative."""
    g = torch.Generator().manual_seed(E * 7 + top)
    z, corr = rn(g, T, E, std=2.0), rn(g, E, std=0.3, mean=-0.3)
    idx = torch.empty(T, top, dtype=torch.int32, device=DEV)
    gate = torch.empty(T, top, device=DEV)
    K().router_select(z.to(DEV), idx, gate, top_k=top, sigmoid_gate="scored",
                      rule={"score": "softmax", "choice_bias": corr.to(DEV), "groups": groups, "keep": keep, "group_score": "max",
                            "normalise": False})
    r = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    moved = 0
    for t in range(T):
        wi, ww = P.route(z[t].double(), corr.double(), r)
        assert sorted(idx[t].tolist()) == sorted(wi.tolist()), t
        order = {e: k for k, e in enumerate(idx[t].tolist())}
        got = torch.tensor([gate[t, order[e]].item() for e in wi.tolist()], dtype=F64)
        assert ((got - ww) / ww).abs().max() < 1e-5
        moved += sorted(torch.topk(z[t], top).indices.tolist()) != sorted(wi.tolist())
    if E > top:
        assert moved > 0


@pytest.mark.parametrize("T,W,E,ident,top,ff,groups,dtype", [
    (5, 52, 5, 1, 3, 20, (3, 2), "float32"), (300, 64, 12, 4, 4, 96, (4, 2), "bfloat16"), (7, 64, 12, 4, 4, 96, (4, 2), "bfloat16"),
    (90, 40, 2, 6, 2, 12, (4, 3), "bfloat16"), (6, 33, 4, 4, 2, 16, None, "float32"), (1, 128, 8, 0, 3, 64, (2, 1), "bfloat16"),
    (40, 30, 3, 2, 1, 12, None, "bfloat16"), (600, 256, 4, 4, 2, 256, None, "bfloat16")])
def test_routed_part_with_clamped_and_identity_experts(T, W, E, ident, top, ff, groups, dtype):
    """The part as the model runs it, added into rows and handed over as a sum: sorted rows or gathered ones, few tokens in
    one launch or many in several, the float32 pipe and the tensor-core products; experts beyond their clamps, tokens
    whose chosen experts are all the identity, experts that no token chose."""
    g = torch.Generator().manual_seed(T + W)
    dt = getattr(torch, dtype)
    limit = 0.9
    Wt = {"router": rn(g, E + ident, W, std=2.5 * W ** -0.5).bfloat16(), "correction": rn(g, E + ident, std=0.2).bfloat16()}
    for e in range(E):
        for n, shape in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
            Wt[f"e{e}.{n}"] = rn(g, *shape, std=2.0 * shape[1] ** -0.5).bfloat16()
    part = build("feed_forward", "moe_swiglu", {
        "hidden_size": W, "num_experts": E, "identity_experts": ident, "top_k": top, "expert_size": ff, "activation": "swish_clamped",
        "limit": limit, "router_gate": "scored", "router_name": "router", "expert_layout": "per_expert",
        "router_rule": {"score": "softmax", "choice_bias": "correction", "groups": (groups or (1, 1))[0], "keep": (groups or (1, 1))[1],
                        "group_score": "max", "normalise": False},
        "expert_names": {n: "e{e}." + n for n in ("gate", "up", "down")}}, Wt)
    mlp = {"expert": {"ff": ff, "limit": limit}, "router": {"experts": E, "identity": ident, "top": top}}
    if groups:
        mlp["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    h, res = rn(g, T, W).to(dt), rn(g, T, W)
    own = []
    want = P.routed_ff(h.double(), Wt, "", mlp, own=own)

    class B:
        pass
    part.capture = []
    buf = res.to(DEV).clone()
    part.forward(h.to(DEV), buf, B())
    assert [sorted(x) for x in part.capture[0].cpu().tolist()] == own
    if ident and T > 20 and top <= 2:
        assert any(min(c) >= E for c in own)               # a token whose chosen experts are all the identity
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert (buf.cpu().double() - res.double() - want).abs().max() < tol * want.abs().max()
    out = part.expert_sum(h.to(DEV), B()).rows(part.ws)
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
    """A prompt cut into portions of 2, 3, 64, 1, 17, ... tokens, with cuts inside pages and windows and portions shorter
    than the convolution; in float32 the logits are also those of the single step, to rounding."""
    b = models[name]
    toks = V.tokens(200, b.cfg["vocab"], 6)
    for dtype in ("float32", "bfloat16"):
        e = b.engine(dtype)
        r = Run(e)
        at = 0
        for n in (2, 3, 64, 1, 17, 2, 70, 5, 36):
            r.step([("p", toks[at:at + n], range(n))])
            at += n
        assert at == 200
        r.check(b, {"p": toks}, TOL[dtype])
        if dtype == "float32":
            one = Run(e)
            one.step([("w", toks, range(200))])
            d = err(torch.stack([r.logits["p"][i] for i in range(200)]), torch.stack([one.logits["w"][i] for i in range(200)]))
            assert d < 5e-5, d


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_batches_in_reused_slots(models, name, dtype):
    """Requests of 1 to 140 tokens start together, are decoded together, end at different steps; a second group then
    runs in the slots and pages the first gave back.  Every logit is the request's own: nothing of a slot's earlier
    convolution inputs or pages shows."""
    b = models[name]
    vocab = b.cfg["vocab"]
    reqs = {f"r{i}": V.tokens(n, vocab, 60 + i) for i, n in enumerate((1, 75, 130, 9, 66, 140))}
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


def _stand_out(W, pre, tokens, m):
    """Makes the keys of `tokens` stand out for every query that may see them.  Every token's embedding gets the same
    large element 1 and a small element 0, those of `tokens` a large element 0, and the norm before the mixer lets both
    through.  Attention: the last element of every q head (outside the rotated part) reads element 1, that of every k head
    element 0, past the convolution.  Latent attention: the last element of the queries' latent reads element 1, that of
    the cached latent element 0, and the last plain element of every head's query and key reads those."""
    W["embed"][:, 0], W["embed"][:, 1] = 0.05, 3.0
    for token in tokens:
        W["embed"][token, 0] = 6.0
    W["l0.norm1.alpha"] = torch.tensor(1.0).bfloat16()
    W["l0.norm1"][:2], W["l0.norm1.b"][:2] = 1.0, 0.0

    def row(name, r, col, value):
        W[pre + name][r] = 0.0
        W[pre + name][r, col] = value

    if "kv_rank" in m:
        row("dq", m["q_rank"] - 1, 1, 8.0)
        row("dkv", m["kv_rank"] - 1, 0, 8.0)
        for h in range(m["heads"]):
            row("uq", (h + 1) * (m["dim"] + m["rot_dim"]) - m["rot_dim"] - 1, m["q_rank"] - 1, 3.0)
            row("uk", (h + 1) * m["dim"] - 1, m["kv_rank"] - 1, 1.5)
        return
    for name, heads, col in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        for h in range(heads):
            row(name, (h + 1) * m["dim"] - 1, col, 4.0)
            if m.get("conv"):
                row(name + ".conv", (h + 1) * m["dim"] - 1, m["conv"] - 1, 1.0)


def test_window_edges_through_the_model(tmp_path):
    """One latent layer: the keys at positions 0, 62 .. 65, 127 and 128 stand out.  A query gives such a key most of its
    weight while it is inside the window and none of it one token later; in a prompt and token by token, for windows that
    put the edge on a page border, before it and after it, a window of one and none; with sizes for the general kernel and
    for the tensor-core one."""
    special = (7, 9, 11, 13, 15, 17, 19)
    toks = [t if t not in special else 8 for t in V.tokens(200, 50, 9)]
    for p, t in zip((0, 62, 63, 64, 65, 127, 128), special):
        toks[p] = t
    for rank, rot in ((11, 4), (48, 16)):
        last = []
        for window in (64, 63, 65, 1, 20, 128, None):
            m = V.latent(2, 6, rot, 8, 12, rank, window=window, scale=0.3)
            b = Built(V.model([V.layer(m, None)], width=24, vocab=50), 31, tmp_path, lambda W: _stand_out(W, "l0.mix.", special, m))
            for dtype in ("float32", "bfloat16"):
                r = Run(b.engine(dtype))
                r.step([("x", toks[:126], range(126))])
                for i in range(126, 200):
                    r.step([("x", toks[i:i + 1], [0])])
                r.check(b, {"x": toks}, TOL[dtype])
            last.append(b.plain(toks)[64:])
        for i in range(1, len(last)):                           # the variants do differ where the edge moved
            assert (last[i] - last[0]).abs().max() > 1e-2, i


@pytest.mark.parametrize("D,Dv,dims,conv", [(10, 6, 4, 3), (64, 64, 32, 4), (16, 8, 8, None)])
def test_one_position_that_stands_out(tmp_path, D, Dv, dims, conv):
    """Attention dominated by one direction in which a token that occurs once, at position 2, is large: every later query
    gives that position most of its weight, also hundreds of positions and several pages later, so its value arrives
    turned by the distance; leaving it out would change every logit after it."""
    m = V.attention(2, 1, D, Dv, dims, conv=conv, scale=0.6)
    cfg = V.model([V.layer(m, V.moe(4, 2, 16, identity=2))], width=32, vocab=40)
    b = Built(cfg, 3, tmp_path, lambda W: _stand_out(W, "l0.mix.", (7,), m))
    toks = [t if t != 7 else 8 for t in V.tokens(330, 40, 1)]
    toks[2] = 7
    with_far = b.plain(toks)
    other = list(toks)
    other[2] = 9
    assert (b.plain(other)[300:] - with_far[300:]).abs().max() > 1e-2      # the far token does matter to late rows
    for dtype in ("float32", "bfloat16"):
        r = Run(b.engine(dtype, max_tokens=512, max_seqs=2))
        r.step([("x", toks[:290], [0, 1, 2, 3, 63, 64, 65, 128, 289])])
        for i in range(290, 330):
            r.step([("x", toks[i:i + 1], [0])])
        r.check(b, {"x": toks}, TOL[dtype])


@pytest.mark.parametrize("name", ["A", "B"])
def test_a_far_token_among_hundreds_and_long_decoding(models, name):
    """700 tokens: the attention layers read every position back to the first across many pages while the latent layers
    give their pages back, through 120 decoded tokens."""
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
        assert windowed and all(g.pages_held() <= -(-g.req.window_size // 64) + 1 for g in windowed)


def test_fused_and_separate_kernels_agree(models):
    """The fused preparation and the tensor-core attention kernels, and the separate and general ones, in bfloat16: both
    give the plain implementation's logits (with the choices of experts that each of them made)."""
    from cpi_b200.parts import attention as A
    b = models["B"]
    toks = V.tokens(300, b.cfg["vocab"], 3)
    for on in (True, False):
        A.use_tensor_core_kernels = A.use_fused_preparation = on
        try:
            r = Run(b.engine("bfloat16", max_tokens=1024, max_seqs=2))
            r.step([("x", toks[:200], range(0, 200, 7))])
            r.step([("x", toks[200:260], range(60))])
            for i in range(260, 300):
                r.step([("x", toks[i:i + 1], [0])])
            r.check(b, {"x": toks}, TOL["bfloat16"])
        finally:
            A.use_tensor_core_kernels = A.use_fused_preparation = True


def test_other_constants_change_the_result_as_the_plain_implementation_says(tmp_path):
    base = V.model([V.layer(V.attention(4, 2, 8, 12, 4, conv=3, base=100.0), V.moe(6, 2, 12, identity=2, groups=(4, 1))),
                    V.layer(V.latent(2, 6, 8, 10, 9, 12, window=9, base=20.0, scaling=(4.0, 64, 4.0, 0.5)), V.moe(4, 2, 10, identity=1)),
                    V.layer(V.attention(2, 2, 16, 12, 16), None)],
                   width=32, vocab=70, logit_softcap=5.0, scale=0.8, loop=(0, 2, 2))
    att, lat = (lambda c: c["layers"][0]["mixer"]), (lambda c: c["layers"][1]["mixer"])
    ff = lambda c: c["layers"][0]["mlp"]
    same_weights = {
        "eps": lambda c: c["norm"].update(eps=0.3),
        "no_logit_cap": lambda c: c.pop("logit_softcap"), "logit_cap": lambda c: c.update(logit_softcap=2.0),
        "no_embedding_scale": lambda c: c.pop("embedding"), "embedding_scale": lambda c: c["embedding"].update(scale=2.0),
        "no_scaling": lambda c: lat(c)["rot"].pop("scaling"), "factor": lambda c: lat(c)["rot"]["scaling"].update(factor=8.0),
        "original": lambda c: lat(c)["rot"]["scaling"].update(original=16),
        "fast": lambda c: lat(c)["rot"]["scaling"].update(fast=0.6), "slow": lambda c: lat(c)["rot"]["scaling"].update(slow=3.0),
        "lat_base": lambda c: lat(c)["rot"].update(base=1000.0), "lat_scale": lambda c: lat(c).update(scale=0.1),
        "window": lambda c: lat(c)["mask"].update(size=8), "no_window": lambda c: lat(c).pop("mask"),
        "base": lambda c: att(c)["rot"].update(base=1000.0), "dims": lambda c: att(c)["rot"].update(dims=8),
        "scale": lambda c: att(c).update(scale=0.3),
        "top": lambda c: ff(c)["router"].update(top=1), "keep": lambda c: ff(c)["router"]["groups"].update(keep=3),
        "groups": lambda c: ff(c)["router"]["groups"].update(count=2, keep=1), "no_groups": lambda c: ff(c)["router"].pop("groups"),
        "limit": lambda c: ff(c)["expert"].update(limit=0.4), "no_mlp": lambda c: c["layers"][0].update(mlp=None),
        "other_loop": lambda c: c["loop"].update(start=1, stop=3),
    }
    other_weights = {
        "kv_heads": lambda c: att(c).update(kv_heads=4), "taps": lambda c: att(c).update(conv=2), "no_conv": lambda c: att(c).pop("conv"),
        "identity": lambda c: ff(c)["router"].update(experts=2, identity=6), "no_identity": lambda c: ff(c)["router"].update(experts=8, identity=0),
        "times": lambda c: c["loop"].update(times=3), "once": lambda c: c["loop"].update(times=1), "no_loop": lambda c: c.pop("loop"),
        "order": lambda c: c["layers"].reverse(),
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


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12])
def test_configurations_drawn_from_a_seed(seed, tmp_path):
    """Every size, option and constant drawn from a seed: a prompt with logits everywhere, a second request in a
    portion and then both decoded together, in float32 to rounding and in bfloat16."""
    cfg = V.draw_config(seed)
    b = Built(cfg, 40 + seed, tmp_path)
    vocab = cfg["vocab"]
    ta, tb = V.tokens(110, vocab, seed), V.tokens(75, vocab, seed + 100)
    for dtype in ("float32", "bfloat16"):
        r = Run(b.engine(dtype, max_tokens=1024, max_seqs=2))
        r.step([("a", ta[:90], range(90)), ("b", tb[:3], range(3))])
        r.step([("b", tb[3:70], range(67))])
        for i in range(5):
            r.step([("a", ta[90 + i:91 + i], [0]), ("b", tb[70 + i:71 + i], [0])])
        r.end("b")
        for i in range(95, 110):
            r.step([("a", ta[i:i + 1], [0])])
        r.check(b, {"a": ta, "b": tb}, TOL[dtype])


def test_layers_recorded_one_by_one(models):
    """The residual after every layer run is the plain implementation's."""
    b = models["A"]
    toks = V.tokens(30, b.cfg["vocab"], 4)
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 5e-2)):
        e = b.engine(dtype)
        e.model.layer_capture = []
        r = Run(e)
        r.step([("x", toks, [29])])
        want = []
        P.forward(b.cfg, b.W, toks, want, forced={n: [by[p] for p in range(30)] for n, by in r.routing.get("x", {}).items()})
        assert len(e.model.layer_capture) == len(want) == 8
        for got, w in zip(e.model.layer_capture, want):
            assert (got.cpu().double() - w).abs().max() < tol * w.abs().max()


def test_greedy_generation_through_the_entry_point(models):
    """`Model.generate` (scheduler, sampler, decode graphs) picks the plain implementation's tokens: unequal prompts,
    more requests than slots."""
    from cpi_b200.api import Model
    b = models["A"]
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
        assert len(res.tokens) == 12


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
    assert "Nekorax" in r.stdout and "attention" in r.stdout


def test_replay_tool_runs_a_nekorax_folder(models, tmp_path):
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
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / f"out_{dtype}"
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", b.dir, "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps),
                           capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        rd = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, vocab).copy())
        got = torch.cat([rd(i) for i in range(4)])
        if dtype == "float32":
            ra, rb = b.plain(ta), b.plain(tb)
            want = torch.cat([ra, torch.stack([ra[69], rb[20], ra[70], ra[71]])])
            assert got.shape == want.shape and err(got, want) < TOL[dtype]
        else:                       # the engine's own logits of the same steps (held against the plain ones elsewhere)
            r = Run(b.engine(dtype, max_tokens=512), record=False)
            for st in steps:
                r.step([(x["id"], x["tokens"], x["want"]) for x in st["entries"]])
                for rid in st["end"]:
                    r.end(rid)
            want = [r.logits["a"][p] for p in range(80)] + [r.logits["a2"][69], r.logits["b"][20], r.logits["a2"][70], r.logits["a2"][71]]
            assert err(got, torch.stack(want)) < 1e-5
