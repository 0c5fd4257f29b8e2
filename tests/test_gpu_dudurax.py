"""Dudurax on the GPU against the plain restatement of tests/dudurax_oracle.py: the new operators called directly, every
mixer and feed-forward alone, prompts against token-by-token decoding, portions down to two tokens, mixed batches, re-used
pages and slots (the previous token of the pair embedding included), keys just inside and just outside the window (at page
borders too), tokens far back that only the recurrent state remembers, strong decays, close group choices and negative
choice scores, identity experts, the first tokens of a sequence, long decoding, sizes where counts collapse to 1 or are not
multiples of 4, the tensor-core paths, greedy generation through the engine's scheduler, the command line and the trace
replay program."""
import copy
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

import dudurax_oracle as O

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL32, TOL16 = 2e-4, 5e-2
F = torch.float64


def make(cfg=None, seed=0, dtype="float32", edit=None, **kw):
    from proxy_inference_engine_b200.dudurax import DuduraxArgs, DuduraxModel, random_weights
    cfg = copy.deepcopy(cfg) if cfg else O.random_config(**kw)
    args = DuduraxArgs.from_dict(cfg)
    w = random_weights(args, seed=seed)
    if edit:
        edit(w)
    return cfg, w, DuduraxModel(args, w, "cuda", dtype)


def engine(model, max_tokens=1024, max_seqs=4, graph=True):
    from proxy_inference_engine_b200.engine import HybridEngine
    return HybridEngine(model, max_tokens, max_seqs, use_graph=graph)


def toks(n, vocab=90, seed=1, avoid=()):
    g = torch.Generator().manual_seed(seed)
    out = torch.randint(0, vocab, (n,), generator=g).tolist()
    return [t if t not in avoid else (t + 7) % 80 for t in out]


def rows_err(got, want):
    got, want = got.double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def err(got, want):
    return float(rows_err(got, want).max())


def whole(eng, ids, sid="s"):
    out = eng.forward([(sid, ids, list(range(len(ids))))])
    eng.finish(sid)
    return out


def in_portions(eng, ids, sizes, sid="s"):
    """Feeds ids in portions of the given sizes (the last size repeats), every row wanted."""
    outs, at, k = [], 0, 0
    while at < len(ids):
        n = min(sizes[min(k, len(sizes) - 1)], len(ids) - at)
        outs.append(eng.forward([(sid, ids[at:at + n], list(range(n)))]))
        at, k = at + n, k + 1
    eng.finish(sid)
    return torch.cat(outs)


# ---- the operators, called directly ------------------------------------------------------------------------------------------
def _lib():
    from proxy_inference_engine_b200 import _lib as lib
    return lib, lib.load_hybrid(build_if_missing=True)


def _ptr(t):
    return None if t is None else C.c_void_p(t.data_ptr())


def _st():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def _rand(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.rand(shape, generator=g, dtype=F) * 2 - 1) * scale


def _cu(t):
    return t.float().contiguous().cuda()


def _batch(seqs, tokens=None):
    """seqs: [(rows, context, slot)] -> (BatchDetails, descriptor, keepalive)."""
    from proxy_inference_engine_b200.ragged import BatchDetails
    b = BatchDetails.build([(i, tokens[i] if tokens else [0] * n, ctx, list(range((ctx + n + 63) // 64)), slot)
                            for i, (n, ctx, slot) in enumerate(seqs)])
    desc, keep = b.hybrid_descriptor()
    return b, desc, keep


@pytest.mark.parametrize("M,N,K", [(5, 40, 24), (70, 96, 64), (33, 17, 128)])
def test_linear_with_gelu(M, N, K):
    lib, L = _lib()
    x, w = _rand(M, K, seed=1, scale=3.0), _rand(N, K, seed=2, scale=0.7)
    for dt, code, tol in ((torch.float32, lib.DTYPE_F32, 1e-5), (torch.bfloat16, lib.DTYPE_BF16, 1e-5)):
        xd, wd = x.to(dt).cuda(), w.to(dt).cuda()
        want = O.gelu_tanh(xd.double().cpu() @ wd.double().cpu().T)
        out = torch.empty((M, N), dtype=torch.float32, device="cuda")
        lib.check_hybrid(L.pieh_linear_act(_ptr(out), lib.DTYPE_F32, N, _ptr(xd), code, K, _ptr(wd), code, None, M, N, K,
                                           lib.EPI_GELU, 0.0, 0.0, _st()), "linear_act")
        assert float((out.double().cpu() - want).abs().max()) < tol * float(want.abs().max())


@pytest.mark.parametrize("W", [100, 66, 13])
def test_sum_norm_of_a_plain_row_and_of_a_mixture_with_identity_rows(W):
    lib, L = _lib()
    T, top, eps, alpha = 7, 3, 1e-5, 1.6
    x, y, nw = _rand(T, W, seed=3, scale=2.0), _rand(T, W, seed=4, scale=3.0), 1 + _rand(W, seed=5, scale=0.3)
    parts, pw = _rand(20, W, seed=6, scale=2.0), _rand(T, top, seed=7)
    g = torch.Generator().manual_seed(8)
    pr = torch.randint(0, 20, (T, top), generator=g)
    pr[1, 0] = pr[2, 2] = pr[4, :] = -1                      # a negative row is the token's own x
    mixed = torch.stack([sum(pw[t, k] * (x[t] if pr[t, k] < 0 else parts[pr[t, k]]) for k in range(top)) for t in range(T)])
    nwd, yd, pd, prd, pwd = _cu(nw), _cu(y), _cu(parts), pr.int().cuda(), _cu(pw)
    mix = lib.HybMixSum(pd.data_ptr(), prd.data_ptr(), pwd.data_ptr(), top, None, None, 0)
    for f, use_mix in ((y, False), (mixed, True)):
        want = O.unit_rms(alpha * x + f, eps) * nw
        for act in (None, torch.float32, torch.bfloat16):
            xd = _cu(x)
            h = torch.zeros((T, W), dtype=act, device="cuda") if act else None
            lib.check_hybrid(L.pieh_sum_norm(_ptr(xd), _ptr(h), lib.DTYPE_BF16 if act == torch.bfloat16 else lib.DTYPE_F32,
                                             None if use_mix else _ptr(yd), C.byref(mix) if use_mix else None, _ptr(nwd), alpha,
                                             eps, T, W, _st()), "sum_norm")
            assert float((xd.double().cpu() - want).abs().max()) < 1e-5
            if act:
                assert torch.equal(h, xd.to(act))


def test_pair_embedding_keeps_the_last_token_of_every_slot():
    lib, L = _lib()
    W, vocab, bg = 20, 50, {"buckets": 37, "mul_prev": 100003, "mul_cur": 999983}       # products far beyond 32 bits
    w = {"embed": _rand(vocab, W, seed=9), "bigram": _rand(38, W, seed=10)}
    seqs = [toks(9, vocab, seed=11), toks(6, vocab, seed=12)]
    emb = {"scale": 2.5, "bigram": bg}
    want = [O.embedding(s, w, emb) for s in seqs]
    prev = torch.full((3,), 17, dtype=torch.int32, device="cuda")                       # slots that held other sequences
    table, pairs = _cu(w["embed"]), _cu(w["bigram"])
    for spans in ([(0, 1), (0, 4)], [(1, 4), (4, 5)], [(4, 9), (5, 6)]):
        part = [s[lo:hi] for s, (lo, hi) in zip(seqs, spans)]
        b, desc, keep = _batch([(hi - lo, lo, 2 - i) for i, (lo, hi) in enumerate(spans)], part)
        T = b.total_tokens_in_step
        x, h = torch.empty((T, W), device="cuda"), torch.empty((T, W), dtype=torch.bfloat16, device="cuda")
        lib.check_hybrid(L.pieh_embed_pairs(_ptr(x), _ptr(h), lib.DTYPE_BF16, _ptr(table), _ptr(pairs), lib.DTYPE_F32,
                                            _ptr(b.token_ids), 2.5, bg["mul_prev"], bg["mul_cur"], bg["buckets"], _ptr(prev), W,
                                            vocab, C.byref(desc), _st()), "embed_pairs")
        assert float((x.double().cpu() - torch.cat([t[lo:hi] for t, (lo, hi) in zip(want, spans)])).abs().max()) < 1e-5
        assert torch.equal(h, x.to(torch.bfloat16))
        assert prev.tolist()[2 - 0] == part[0][-1] and prev.tolist()[2 - 1] == part[1][-1] and prev.tolist()[0] == 17
        del keep


@pytest.mark.parametrize("T,C_,rank,tau", [(5, 12, 3, 1.0), (40, 130, 16, 16.0), (17, 256, 70, 0.5), (3, 7, 1, 4.0)])
def test_channel_decays(T, C_, rank, tau):
    lib, L = _lib()
    low, w2, b = _rand(T, rank + 2, seed=13, scale=6.0), _rand(rank, C_, seed=14, scale=3.0), _rand(C_, seed=15, scale=40.0)
    z = low[:, 2:] @ w2 + b                                              # logits on both sides of any overflow
    want = torch.exp(-torch.nn.functional.softplus(-z, threshold=1e9) / tau)
    out = torch.empty((T, C_), device="cuda")
    lowd, w2d, bd = _cu(low), _cu(w2), _cu(b)
    lib.check_hybrid(L.pieh_gla_decay(_ptr(out), _ptr(lowd), rank + 2, 2, rank, _ptr(w2d), _ptr(bd), 1.0 / tau, C_, T, _st()), "decay")
    assert float((out.double().cpu() - want).abs().max()) < 2e-5 * max(1.0, 1.0 / tau)
    assert torch.isfinite(out).all()


def _gla_inputs(lens, H, dk, dv, lo=-6.0):
    out = []
    for s, n in enumerate(lens):
        q, k, v = (_rand(n, H, d, seed=20 + 3 * s + j) for j, d in enumerate((dk, dk, dv)))
        decay = torch.exp(-torch.exp(_rand(n, H, dk, seed=40 + s, scale=3.0) + lo / 2))
        out.append((q, k, v, decay, O.gla_scan(q, k, v, decay)))
    return out


GLA_SIZES = [(2, 16, 16), (3, 12, 20), (1, 40, 6), (2, 64, 64), (1, 130, 9), (2, 32, 70), (1, 128, 24), (2, 5, 7), (1, 300, 66),
             (1, 256, 65), (1, 1, 1)]


@pytest.mark.parametrize("H,dk,dv", GLA_SIZES)
@pytest.mark.parametrize("seg", [0, 1, 2])
def test_gla_scan_with_states_in_slots(H, dk, dv, seg):
    """Two sequences of unequal length in one step, then both continue from their slots (slots that held another sequence's
    state before); seg > 0: long portions in segments that are scanned side by side."""
    lib, L = _lib()
    data = _gla_inputs([301, 70], H, dk, dv)
    state = torch.full((3, H, dk, dv), 7.0, dtype=torch.float32, device="cuda")       # dirty slots
    cuts = [[(0, 265), (265, 268), (268, 301)], [(0, 2), (2, 69), (69, 70)]]
    for part in range(3):
        spans = [cuts[s][part] for s in range(2)]
        _, desc, keep = _batch([(hi - lo, lo, 2 - s) for s, (lo, hi) in enumerate(spans)])
        q, k, v, decay, want = (torch.cat([data[s][j][lo:hi] for s, (lo, hi) in enumerate(spans)]) for j in range(5))
        T = q.shape[0]
        proj = _cu(torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1))
        dec = _cu(decay.reshape(T, -1))
        gl = lib.HybGla(H, dk, dv, 0, H * dk, 2 * H * dk, 0.7, _ptr(state))
        o = torch.empty((T, H, dv), dtype=torch.float32, device="cuda")
        scratch = None
        if seg:
            n = ((desc.n_tiles - 1) // seg + desc.n_seq) * H * dk * (dv + 1)
            scratch = torch.full((n,), float("nan"), device="cuda")
        lib.check_hybrid(L.pieh_gla_scan(_ptr(o), _ptr(proj), proj.stride(0), _ptr(dec), C.byref(gl), C.byref(desc), _ptr(scratch),
                                         seg, _st()), "gla_scan")
        want = 0.7 * want
        assert float((o.double().cpu() - want).abs().max()) < 2e-5 * max(1.0, float(want.abs().max())), part
        del keep
    assert bool((state[0] == 7.0).all())                                              # the slot nobody owns


@pytest.mark.parametrize("H,dk,dv", GLA_SIZES + [(2, 64, 300), (1, 32, 600)])
def test_gla_step_does_decays_update_norm_and_gate(H, dk, dv):
    lib, L = _lib()
    n, rank, eps, tau = 3, 5, 1e-5, 3.0
    wide = 2 * H * dk + 2 * H * dv + rank
    w2, b2, nw = _rand(rank, H * dk, seed=50), _rand(H * dk, seed=51, scale=3.0), 1 + _rand(dv, seed=52, scale=0.3)
    S = {0: torch.zeros((H, dk, dv), dtype=F), 1: _rand(H, dk, dv, seed=53), 2: _rand(H, dk, dv, seed=54)}
    state = torch.full((4, H, dk, dv), 9.0, dtype=torch.float32, device="cuda")
    state[1], state[3] = S[1].float(), S[2].float()
    slots, ctxs = [0, 1, 3], [0, 5, 64]                                               # the first starts from zero
    w2d, b2d, nwd = _cu(w2), _cu(b2), _cu(nw)
    for it in range(2):
        proj = _rand(n, wide, seed=60 + it, scale=1.5)
        _, desc, keep = _batch([(1, c + it, s) for c, s in zip(ctxs, slots)])
        want = torch.zeros((n, H, dv), dtype=F)
        z = proj[:, 2 * H * dk + 2 * H * dv:] @ w2 + b2
        a = (torch.sigmoid(z) ** (1 / tau)).view(n, H, dk)
        q, k = proj[:, :H * dk].view(n, H, dk), proj[:, H * dk:2 * H * dk].view(n, H, dk)
        v = proj[:, 2 * H * dk:2 * H * dk + H * dv].view(n, H, dv)
        g = proj[:, 2 * H * dk + H * dv:2 * H * dk + 2 * H * dv].view(n, H, dv)
        for i in range(n):
            S[i] = a[i][:, :, None] * S[i] + k[i][:, :, None] * v[i][:, None, :]
            o = torch.einsum("hnd,hn->hd", S[i], q[i]) * 0.5
            want[i] = O.unit_rms(o, eps) * nw * O.silu(g[i])
        pd = _cu(proj)
        gl = lib.HybGla(H, dk, dv, 0, H * dk, 2 * H * dk, 0.5, _ptr(state))
        out = torch.empty((n, H * dv), dtype=torch.float32, device="cuda")
        lib.check_hybrid(L.pieh_gla_step(_ptr(out), lib.DTYPE_F32, _ptr(pd), wide, 2 * H * dk + 2 * H * dv, rank, _ptr(w2d), _ptr(b2d),
                                         1 / tau, 2 * H * dk + H * dv, _ptr(nwd), eps, C.byref(gl), C.byref(desc), _st()), "gla_step")
        assert float((out.double().cpu().view(n, H, dv) - want).abs().max()) < 3e-5 * max(1.0, float(want.abs().max())), it
        for i, s in enumerate(slots):
            assert float((state[s].double().cpu() - S[i]).abs().max()) < 1e-5
        del keep
    assert bool((state[2] == 9.0).all())


@pytest.mark.parametrize("E,idn,groups,top,shift", [(6, 2, (4, 2), 3, 0.0), (6, 2, (4, 2), 4, -5.0), (13, 0, (1, 1), 5, -2.0),
                                                    (40, 5, (9, 3), 7, 0.0), (3, 3, (3, 1), 2, 0.5), (1, 1, (1, 1), 2, 0.0),
                                                    (5, 1, (6, 4), 4, -1.0)])
def test_routing_with_correction_groups_and_identity_experts(E, idn, groups, top, shift):
    """Choices, weights and the slot plan; shift makes every choice score negative (what is not eligible must still lose)."""
    lib, L = _lib()
    T, n = 33, E + idn
    z, corr = _rand(T, n, seed=70, scale=3.0), _rand(n, seed=71, scale=0.3) + shift
    r = {"top": top, "scale": 1.7, "groups": {"count": groups[0], "keep": groups[1]}}
    i32 = lambda m: torch.full((m,), -7, dtype=torch.int32, device="cuda")
    P = T * top
    row, exp, slot, wt = i32(P), i32(P), i32(P), torch.empty(P, device="cuda")
    t64, t128 = i32(1 + 3 * (P // 64 + E)), i32(1 + 3 * (P // 128 + E))
    counters = torch.zeros(2 * E + 2, dtype=torch.int32, device="cuda")
    zd, cd = _cu(z), _cu(corr)
    plan = lib.HybMoePlan(E, top, groups[0], groups[1], 1.7, *[t.data_ptr() for t in (row, exp, slot, wt, t64, t128, counters)],
                          0, 1, _ptr(cd), 1, idn)
    lib.check_hybrid(L.pieh_moe_route(_ptr(zd), n, C.byref(plan), T, _st()), "moe_route")
    row, exp, slot, wt = row.tolist(), exp.tolist(), slot.view(T, top).tolist(), wt.view(T, top).tolist()
    used = set()
    for t in range(T):
        pick, w_, gap = O.route(z[t], corr, r)
        assert gap > 1e-5
        for k in range(top):
            assert abs(wt[t][k] - w_[k]) < 1e-5
            if pick[k] >= E:
                assert slot[t][k] == -1
            else:
                s = slot[t][k]
                assert exp[s] == pick[k] and row[s] == t and s not in used
                used.add(s)
    assert used == set(range(len(used))) and all(e == -1 for e in exp[len(used):])
    assert exp[:len(used)] == sorted(exp[:len(used)]) and int(counters.abs().sum()) == 0


# ---- every mechanism alone, through the model ----------------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(pattern="g", ffs="-"), dict(pattern="h", ffs="-"), dict(pattern="a", ffs="-"), dict(pattern="a", ffs="-", kv_rank=12, a_vdim=20),
    dict(pattern="a", ffs="-", kv_rank=12, a_vdim=8), dict(pattern="a", ffs="-", kv_rank=20, a_vdim=24), dict(pattern="a", ffs="-", window=0),
    dict(pattern="g", ffs="d"), dict(pattern="g", ffs="m"), dict(pattern="a", ffs="m"), dict(pattern="gahga", ffs="dm-md")])
def test_each_mixer_and_feed_forward_alone(kw):
    cfg, w, model = make(**kw)
    ids = toks(80)
    trace, otrace = [], []
    got = engine(model, graph=False).forward([("s", ids, list(range(80)))], trace=trace)
    want = O.forward(cfg, w, ids, otrace)
    assert len(trace) == len(otrace) == len(cfg["layers"])
    for a, b in zip(trace, otrace):
        assert err(a, b) < TOL32
    assert err(got, want) < TOL32


def test_the_pieces_of_the_latent_projection_are_folded_only_where_that_is_not_wider():
    for kw, q_rows, folded_q, folded_o in ((dict(kv_rank=16, a_vdim=16), 24, True, True), (dict(kv_rank=17, a_vdim=16), 24, False, False),
                                           (dict(kv_rank=14, a_vdim=12), 22, True, False), (dict(kv_rank=18, a_vdim=20), 24, False, True)):
        _, _, model = make(pattern="a", ffs="-", a_dim=16, rot_dim=8, **kw)
        ly = model.layers[0]
        assert ly["q_rows"] == q_rows and (ly["ukT"] is None) == folded_q and (ly["uv"] is None) == folded_o


def test_bf16_tracks_the_restatement():
    """In bf16 a token whose routing margin is within rounding may take another expert than the restatement, and nudges
    the tokens after it (attention, recurrent state): rows up to the first close call must be within the tolerance, nine
    rows in ten of all, and none far off."""
    cfg, w, model = make(pattern="gah", ffs="dmd", dtype="bfloat16", seed=5)
    ids = toks(150)
    margins = []
    e = rows_err(in_portions(engine(model), ids, [70, 33, 1]), O.forward(cfg, w, ids, None, margins))
    clear = torch.cummin(torch.tensor(margins).view(-1, len(ids)).min(0).values, 0).values > 5e-3
    assert int(clear.sum()) >= 5 and float(e[clear].max()) < TOL16
    assert float(e.quantile(0.9)) < TOL16 and float(e.max()) < 6 * TOL16


@pytest.mark.parametrize("kw", [dict(), dict(kv_rank=12, a_vdim=20)])
def test_bf16_without_routing_is_within_tolerance_everywhere(kw):
    cfg, w, model = make(pattern="gahg", ffs="d-d", dtype="bfloat16", **kw)
    ids = toks(150)
    assert err(in_portions(engine(model), ids, [70, 33, 1]), O.forward(cfg, w, ids)) < TOL16


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kv_rank,rot_dim,a_dim,a_vdim", [(64, 32, 64, 40), (64, 64, 40, 72), (128, 32, 128, 128), (128, 64, 64, 64),
                                                          (64, 0, 64, 64), (128, 0, 128, 40)])
def test_tensor_core_paths(dtype, kv_rank, rot_dim, a_dim, a_vdim):
    """Sizes at which prompt portions take the tiled attention kernel over bf16 latents (every shape it is built for) and the
    tcgen05 products (K a multiple of 64, more than 32 rows), with a window that ends inside a page."""
    cfg = O.random_config(width=128, pattern="ag", ffs="d-", a_heads=2, a_dim=a_dim, a_vdim=a_vdim, kv_rank=kv_rank, rot_dim=rot_dim,
                          window=90, dim=64, vdim=64, ff=128)
    cfg, w, model = make(cfg, dtype=dtype)
    ids = toks(300)
    e = rows_err(in_portions(engine(model), ids, [170, 80, 1]), O.forward(cfg, w, ids))
    assert float(e.max()) < (TOL32 if dtype == "float32" else TOL16)
    assert model.L.pieh_pipeline_error() == 0


# ---- prompts, decoding, portions, batches ---------------------------------------------------------------------------------------
def test_prefill_against_token_by_token_decoding():
    cfg, w, model = make(pattern="gah", ffs="dmm")
    ids = toks(70)
    want = O.forward(cfg, w, ids)
    eng = engine(model)
    assert err(whole(eng, ids), want) < TOL32
    assert err(in_portions(eng, ids, [1]), want) < TOL32            # one token at a time from the first one (graph replay)
    assert err(in_portions(engine(model, graph=False), ids, [1]), want) < TOL32


@pytest.mark.parametrize("sizes", [[2], [3, 2, 5, 2, 64, 7, 2], [63, 2, 1], [64, 64, 2], [65, 1], [17, 16, 15, 2], [129, 2]])
def test_portions_of_several_sizes(sizes):
    cfg, w, model = make(pattern="gah", ffs="dmm")
    ids = toks(140, seed=3)
    assert err(in_portions(engine(model), ids, sizes), O.forward(cfg, w, ids)) < TOL32


def test_unequal_requests_in_one_batch_match_each_alone():
    cfg, w, model = make(pattern="agh", ffs="mdm")
    seqs = {"a": toks(90, seed=5), "b": toks(31, seed=6), "c": toks(7, seed=7), "d": toks(260, seed=8)}
    want = {k: O.forward(cfg, w, v) for k, v in seqs.items()}
    eng = engine(model, max_tokens=512)
    plan = {"a": [40, 1, 1, 30, 2, 16], "b": [1, 1, 2, 20, 7], "c": [2, 5], "d": [130, 64, 1, 1]}
    at = {k: 0 for k in seqs}
    got = {k: [] for k in seqs}
    step = 0
    while any(at[k] < len(seqs[k]) for k in seqs):
        entries = []
        for k in seqs:
            if at[k] >= len(seqs[k]) or (k == "c" and step < 2) or (k == "b" and step == 3):     # c comes later, b rests once
                continue
            n = min(plan[k][step % len(plan[k])], len(seqs[k]) - at[k])
            entries.append((k, seqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
        out = eng.forward(entries)
        r = 0
        for k, part, _ in entries:
            got[k].append(out[r:r + len(part)])
            r += len(part)
            if at[k] == len(seqs[k]):
                eng.finish(k)
        step += 1
    for k in seqs:
        assert err(torch.cat(got[k]), want[k]) < TOL32, k


def test_pages_and_slots_are_used_again():
    cfg, w, model = make(pattern="gah", ffs="dmm")
    eng = engine(model, max_tokens=128, max_seqs=1)                  # two pages, one slot: everything is re-used
    for seed, n, sizes in ((11, 120, [50, 1]), (12, 100, [3, 64, 1]), (13, 128, [128]), (14, 9, [1]), (15, 2, [2]), (16, 1, [1])):
        ids = toks(n, seed=seed)
        assert err(in_portions(eng, ids, sizes, sid=seed), O.forward(cfg, w, ids)) < TOL32, seed
    assert eng.cache.allocator.get_num_free_pages() == 2 and len(eng.cache.free_slots) == 1


def test_long_decoding():
    cfg, w, model = make(pattern="ga", ffs="dm", window=50)
    ids = toks(260, seed=9)
    assert err(in_portions(engine(model), ids, [20, 1]), O.forward(cfg, w, ids)) < TOL32


# ---- inputs made so that one token stands out -----------------------------------------------------------------------------------
def _point_a_key_at_a_query(w, cfg, q_tok, k_tok, gain):
    """Rewrites the embedding of k_tok so that its latent points where all heads' queries of q_tok look, drops the pair table and
    raises the queries: wherever both tokens are visible that key takes nearly all the weight, so one key more or less in the
    window shows."""
    w["bigram"] = torch.zeros_like(w["bigram"])
    m = cfg["layers"][0]["mixer"]
    H, d, dr, r = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    f = lambda n: w[n].double()
    q = (f("l0.mix.q") @ f("embed")[q_tok]).view(H, d + dr)[:, :d]
    look = torch.einsum("hdr,hd->r", f("l0.mix.uk").view(H, d, r), q) * f("l0.mix.dkv.norm")
    e = torch.linalg.pinv(f("l0.mix.dkv")[:r]) @ look
    w["embed"][k_tok] = (e / e.pow(2).mean().sqrt()).to(torch.bfloat16)          # the latent's norm takes the length out again
    w["l0.mix.q"] = (gain * f("l0.mix.q")).to(torch.bfloat16)


@pytest.mark.parametrize("window,probe", [(6, 20), (64, 64), (64, 100), (65, 130), (90, 200), (1, 9), (2, 65), (128, 191)])
def test_keys_just_inside_and_just_outside_the_window(window, probe):
    """One earlier token's key points at the probe's query, just inside the window or just outside it, so a window that is
    one token off changes the logits by far more than the tolerance."""
    cfg = O.random_config(pattern="a", ffs="-", window=window, rot_dim=4)
    cfg, w, model = make(cfg, edit=lambda w: _point_a_key_at_a_query(w, cfg, 89, 88, 3.0))
    for dist in (window - 1, window):
        ids = toks(probe + 6, seed=20 + dist, avoid=(88, 89))
        ids[probe - dist], ids[probe] = 88, 89
        want = O.forward(cfg, w, ids)
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = window + (1 if dist == window else -1)
        if other["layers"][0]["mixer"]["mask"]["size"] > 0:
            assert float(rows_err(O.forward(other, w, ids), want)[probe]) > 50 * TOL32   # the case does show the edge
        assert err(whole(engine(model), ids), want) < TOL32                              # inside a prompt
        assert err(in_portions(engine(model), ids, [probe - 3, 1]), want) < TOL32        # decoded alone
        assert err(in_portions(engine(model), ids, [probe - dist + 1, 2]), want) < TOL32  # portions that start at the edge


@pytest.mark.parametrize("kv_rank,rot_dim", [(64, 32), (128, 64)])
def test_window_edges_on_the_tiled_attention_kernel(kv_rank, rot_dim):
    """The same planted key in bf16 at latent sizes where prompt portions run on 64-row tiles over whole pages: the edge falls
    inside a tile and inside a page."""
    cfg = O.random_config(width=160, pattern="a", ffs="-", a_heads=2, a_dim=64, a_vdim=64, kv_rank=kv_rank, rot_dim=rot_dim, window=70)
    cfg, w, model = make(cfg, dtype="bfloat16", edit=lambda w: _point_a_key_at_a_query(w, cfg, 89, 88, 2.0))
    probe = 150
    for dist in (69, 70):
        ids = toks(probe + 40, seed=30 + dist, avoid=(88, 89))
        ids[probe - dist], ids[probe] = 88, 89
        want = O.forward(cfg, w, ids)
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = 70 + (1 if dist == 70 else -1)
        assert float(rows_err(O.forward(other, w, ids), want)[probe]) > 3 * TOL16
        assert float(rows_err(whole(engine(model), ids), want)[probe]) < TOL16
        assert float(rows_err(in_portions(engine(model), ids, [100, 90]), want)[probe]) < TOL16


@pytest.mark.parametrize("far,probe", [(0, 63), (0, 64), (63, 300), (64, 191), (128, 447)])
def test_a_key_far_away_without_a_window(far, probe):
    """One key at a page's border or at the very start takes the probe's weight among hundreds of keys."""
    cfg = O.random_config(pattern="a", ffs="-", window=0)
    cfg, w, model = make(cfg, edit=lambda w: _point_a_key_at_a_query(w, cfg, 89, 88, 3.0))
    ids = toks(probe + 3, seed=35 + far, avoid=(88, 89))
    ids[far], ids[probe] = 88, 89
    want = O.forward(cfg, w, ids)
    moved = list(ids)
    moved[far] = 3
    assert float(rows_err(O.forward(cfg, w, moved), want)[probe]) > 200 * TOL32
    assert err(whole(engine(model), ids), want) < TOL32
    assert err(in_portions(engine(model), ids, [far + 1, 50, 1] if far else [60, 1]), want) < TOL32


def _decay_bias(*values):
    """Decays without the low-rank part: channel c of every head gets the logit values[c mod n]."""
    def edit(w):
        for k in list(w):
            if k.endswith("mix.a2"):
                w[k] = torch.zeros_like(w[k])
            if k.endswith("mix.a2.b"):
                w[k] = torch.tensor(values).repeat(w[k].numel() // len(values) + 1)[:w[k].numel()].to(torch.bfloat16)
    return edit


@pytest.mark.parametrize("pattern,far,probe", [("g", 0, 63), ("g", 3, 300), ("h", 65, 447), ("gh", 2, 129)])
def test_tokens_far_back_live_on_in_the_state(pattern, far, probe):
    """With slow forgetting, a token hundreds of positions back still moves the logits through the recurrent state; the state
    has to survive portions, page borders, segments and decoding."""
    cfg, w, model = make(pattern=pattern, ffs="-", edit=_decay_bias(9.0))
    ids = toks(probe + 3, seed=40 + far)
    want = O.forward(cfg, w, ids)
    moved = list(ids)
    moved[far] = (ids[far] + 1) % 90
    assert float(rows_err(O.forward(cfg, w, moved), want)[probe]) > 10 * TOL32           # the far token carries weight
    eng = engine(model)
    assert err(whole(eng, ids), want) < TOL32
    assert err(in_portions(eng, ids, [probe - 1, 1]), want) < TOL32
    assert err(in_portions(eng, ids, [far + 1, 37]), want) < TOL32


@pytest.mark.parametrize("tau", [0.5, 1.0, 16.0])
def test_decays_from_nothing_to_everything_side_by_side(tau):
    """Channels that keep nothing beside channels that keep everything: products of decays leave the fp32 range downwards and
    nothing may overflow, in one pass and in segments."""
    cfg, w, model = make(pattern="gh", ffs="-", tau=tau, tau2=tau, edit=_decay_bias(-80.0, 12.0, -3.0, 0.0, 4.0))
    ids = toks(330, seed=45)
    want = O.forward(cfg, w, ids)
    assert err(whole(engine(model), ids), want) < TOL32
    assert err(in_portions(engine(model), ids, [200, 63, 1]), want) < TOL32


def test_the_pair_embedding_across_portions_and_at_the_start():
    def edit(w):
        w["bigram"] = (4 * w["bigram"].float()).to(torch.bfloat16)
    cfg, w, model = make(pattern="g", ffs="-", edit=edit)
    ids = toks(30, seed=46)
    want = O.forward(cfg, w, ids)
    lost = dict(w)
    lost["bigram"] = w["bigram"].clone()
    lost["bigram"][-1] = 0                                              # the row of a sequence's first token
    assert float(rows_err(O.forward(cfg, lost, ids), want)[0]) > 100 * TOL32
    swapped = copy.deepcopy(cfg)
    b = swapped["embedding"]["bigram"]
    b["mul_prev"], b["mul_cur"] = b["mul_cur"], b["mul_prev"]
    assert err(O.forward(swapped, w, ids), want) > 100 * TOL32
    eng = engine(model, max_tokens=64, max_seqs=1)                      # one slot: every run starts on the last one's token
    for sizes in ([1], [2], [3, 1, 2, 5], [30]):
        assert err(in_portions(eng, ids, sizes), want) < TOL32, sizes


def test_identity_experts_and_the_correction_count():
    cfg, w, model = make(pattern="g", ffs="m", experts=5, identity=3, groups=(4, 4), top=4)
    ids = toks(40, seed=47)
    want = O.forward(cfg, w, ids)
    none = dict(w)
    none["l0.mlp.correction"] = torch.zeros_like(w["l0.mlp.correction"])
    assert err(O.forward(cfg, none, ids), want) > 100 * TOL32
    assert err(in_portions(engine(model), ids, [23, 2, 1]), want) < TOL32
    # all choices are identity experts: no slot is handed out at all
    def only_identity(w):
        c = torch.full_like(w["l0.mlp.correction"], -3.0)
        c[-3:] = 3.0
        w["l0.mlp.correction"] = c
    cfg, w, model = make(pattern="g", ffs="m", experts=5, identity=3, groups=None, top=3, edit=only_identity)
    assert err(in_portions(engine(model), ids, [23, 2, 1]), O.forward(cfg, w, ids)) < TOL32


# ---- other sizes ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(heads=1, heads2=1, a_heads=1), dict(heads=5, dim=12), dict(top=1), dict(experts=3, identity=1, groups=(2, 2), top=4),
    dict(experts=1, identity=0, groups=None, top=1), dict(identity=0, groups=(3, 2)), dict(groups=None), dict(groups=(8, 5)),
    dict(groups=(2, 1)), dict(rot_dim=2), dict(rot_dim=0), dict(window=1), dict(window=1000), dict(window=0), dict(scale=1.0),
    dict(router_scale=1.0, alpha=1.0, embed_scale=1.0, tau=1.0, tau2=1.0, limit=0.2), dict(limit=5.0), dict(eps=1e-2),
    dict(buckets=0), dict(buckets=1), dict(mul_prev=1, mul_cur=1), dict(mul_prev=0, mul_cur=89),
    dict(width=72, dim=20, vdim=12, dim2=10, vdim2=18, a_dim=12, a_vdim=20, kv_rank=10, rot_dim=6, ff=28, expert_ff=10),
    dict(width=40, dim=4, vdim=4, dim2=8, vdim2=8, a_dim=8, a_vdim=8, kv_rank=8, rot_dim=8, ff=8, expert_ff=8),
    dict(width=66, heads=1, dim=34, vdim=50, heads2=1, dim2=7, vdim2=9, a_dim=10, a_vdim=34, kv_rank=21, rot_dim=10, ff=18, expert_ff=6),
    dict(dim=72, vdim=136, dim2=132, vdim2=68, heads=1, heads2=1, kv_rank=136, a_vdim=72), dict(kv_rank=300, a_heads=2),
    dict(dim=1, vdim=1, dim2=2, vdim2=3), dict(vocab=513, buckets=997)])
def test_other_sizes(kw):
    cfg, w, model = make(pattern="gahg", ffs="mdmm", seed=2, **kw)
    ids = toks(75, vocab=cfg["vocab"], seed=4)
    assert err(in_portions(engine(model), ids, [67, 2, 1]), O.forward(cfg, w, ids)) < TOL32


# ---- the engine's own entry points ------------------------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler():
    cfg, w, model = make(pattern="gah", ffs="dmm")
    prompts = [toks(33, seed=80), toks(5, seed=81), toks(70, seed=82), toks(1, seed=83)]
    eng = engine(model, max_tokens=256, max_seqs=2)                  # four prompts over two slots and four pages
    outs = eng.generate(prompts, max_new_tokens=12, step_tokens=48)
    assert not eng.cache.seqs and len(eng.cache.free_slots) == 2
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits = O.forward(cfg, w, p + o)
        for k, tok in enumerate(o):                                   # each new token is the restatement's choice, or ties it
            row = logits[len(p) + k - 1]
            assert float(row.max() - row[tok]) < 1e-2 * float(row.abs().max()), (k, tok)      # the sampler reads bf16 logits


def _save(tmp, cfg, w):
    from safetensors.torch import save_file
    tmp.mkdir(exist_ok=True)
    (tmp / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(tmp / "model.safetensors"))


def test_generate_command(tmp_path):
    cfg, w, model = make(pattern="ga", ffs="md")
    _save(tmp_path, cfg, w)
    prompts = [toks(9, seed=85), toks(40, seed=86)]
    cmd = [sys.executable, "-m", "proxy_inference_engine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
           "--max-new-tokens", "6"] + [x for p in prompts for x in ("--prompt-ids", ",".join(map(str, p)))]
    r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    assert [ln["prompt_ids"] for ln in lines] == prompts
    want = engine(model).generate(prompts, max_new_tokens=6)
    assert [ln["generated_ids"] for ln in lines] == want


def test_trace_replay_program(tmp_path):
    cfg, w, _ = make(pattern="gah", ffs="dmm")
    mdir, odir = tmp_path / "model", tmp_path / "out"
    _save(mdir, cfg, w)
    a, b = toks(70, seed=90), toks(20, seed=91)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:68], "want": []}, {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[19:], "want": [0]}, {"id": "a", "tokens": a[68:], "want": [1]}], "end": ["a", "b"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", "float32",
                        "--out", str(odir), "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    read = lambda n: torch.frombuffer(bytearray((odir / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert err(read(0), wa[[0, 65]]) < TOL32
    assert err(read(1), wb[[18]]) < TOL32
    assert err(read(2), torch.stack([wb[19], wa[69]])) < TOL32
