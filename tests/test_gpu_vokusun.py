"""Vokusun on the GPU against the plain restatement of tests/vokusun_oracle.py: the new operators called directly, every mixer
alone, looped stacks, prompts against token-by-token decoding, portions down to two tokens, mixed batches, re-used pages and
slots, keys just inside and just outside the window and the kept first tokens (at page borders too), keys far away, long
decoding, sizes where counts collapse to 1 or are not multiples of 4, the tensor-core paths, greedy generation through the
engine's scheduler, the command line and the trace replay program."""
import copy
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

import vokusun_oracle as O

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL32, TOL16 = 2e-4, 5e-2
F = torch.float64
BF = torch.bfloat16


def make(cfg=None, seed=0, dtype="float32", edit=None, **kw):
    from proxy_inference_engine_b200.vokusun import VokusunArgs, VokusunModel, random_weights
    cfg = copy.deepcopy(cfg) if cfg else O.random_config(**kw)
    args = VokusunArgs.from_dict(cfg)
    w = random_weights(args, seed=seed)
    if edit:
        edit(w)
    return cfg, w, VokusunModel(args, w, "cuda", dtype)


def engine(model, max_tokens=1024, max_seqs=4, graph=True):
    from proxy_inference_engine_b200.engine import HybridEngine
    return HybridEngine(model, max_tokens, max_seqs, use_graph=graph)


def toks(n, vocab=90, seed=1, avoid=()):
    g = torch.Generator().manual_seed(seed)
    out = torch.randint(0, vocab, (n,), generator=g).tolist()
    return [t if t not in avoid else (t + 5) % (vocab - 10) for t in out]


def rows_err(got, want):
    got, want = got.double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def err(got, want):
    return float(rows_err(got, want).max())


def in_portions(eng, ids, sizes, sid="s"):
    """Feeds ids in portions of the given sizes (the last size repeats), every row wanted."""
    outs, at, k = [], 0, 0
    while at < len(ids):
        n = min(sizes[min(k, len(sizes) - 1)], len(ids) - at)
        outs.append(eng.forward([(sid, ids[at:at + n], list(range(n)))]))
        at, k = at + n, k + 1
    eng.finish(sid)
    return torch.cat(outs)


def whole(eng, ids):
    return in_portions(eng, ids, [len(ids)])


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


def _batch(seqs, spare_pages=3):
    """seqs: [(rows, context)] -> (BatchDetails, descriptor, keepalive, page lists); pages are scattered over the pool."""
    from proxy_inference_engine_b200.ragged import BatchDetails
    need = [(n + ctx + 63) // 64 for n, ctx in seqs]
    ids = torch.randperm(sum(need) + spare_pages, generator=torch.Generator().manual_seed(5)).tolist()
    pages, at = [], 0
    for n in need:
        pages.append(ids[at:at + n])
        at += n
    b = BatchDetails.build([(i, [0] * n, ctx, pages[i], i) for i, (n, ctx) in enumerate(seqs)])
    desc, keep = b.hybrid_descriptor()
    return b, desc, keep, pages, len(ids)


@pytest.mark.parametrize("W", [64, 100, 66, 13, 2052, 5000, 8200])
@pytest.mark.parametrize("dt", [torch.float32, BF])
def test_layernorm_add_in_all_its_forms(W, dt):
    """Far-off means (the variance must not be formed from raw squares), strided y and saved rows, every optional part."""
    lib, L = _lib()
    T, eps, code = 5, 1e-5, lib.DTYPE_BF16 if dt == BF else lib.DTYPE_F32
    x, yy, zz = _rand(T, W, seed=1, scale=2.0) + 3, _rand(T, W + 8, seed=2) + 30, _rand(T, W + 4, seed=3, scale=2.0)
    vec, pw, pb, nw, nb = (_rand(W, seed=4 + k) + (1.0 if k in (1, 3) else 0.0) for k in range(5))
    y, z = yy[:, :W], zz[:, :W]
    dev = {k: _cu(v) for k, v in dict(yy=yy, zz=zz, vec=vec, pw=pw, pb=pb, nw=nw, nb=nb).items()}
    rows = torch.tensor([4, 1, 1], dtype=torch.int32, device="cuda")
    for use_y, post, adds, nxt, some in [(1, 1, 0, 1, 0), (1, 1, 0, 0, 0), (1, 0, 1, 1, 0), (0, 0, 0, 1, 0), (1, 1, 1, 1, 0),
                                         (1, 1, 0, 1, 1), (0, 0, 0, 1, 1), (1, 1, 0, None, 0), (1, 0, 0, None, 0)]:
        base = x if not use_y else (x + O.layer_norm(y, pw, pb, eps) if post else y)
        new = base + (z + vec if adds else 0)
        h_want = O.layer_norm(new, nw, nb, eps) if nxt else new
        xd, n = _cu(x), 3 if some else T
        h = torch.full((n, W), 7.0, dtype=dt, device="cuda") if nxt is not None else None
        g = lambda k, on: _ptr(dev[k]) if on else None
        lib.check_hybrid(L.pieh_layernorm_add(_ptr(xd), g("yy", use_y), W + 8, g("pw", post), g("pb", post), g("zz", adds), W + 4,
                                              g("vec", adds), _ptr(h), code, g("nw", nxt), g("nb", nxt), _ptr(rows) if some else None,
                                              eps, n, W, _st()), "layernorm_add")
        assert float((xd.double().cpu() - (x if some else new)).abs().max()) < 5e-5
        if h is not None:
            want = h_want[rows.long().cpu()] if some else h_want
            assert float((h.double().cpu() - want).abs().max()) < (5e-5 if dt == torch.float32 else 2e-2 * float(want.abs().max()))


@pytest.mark.parametrize("M,N,K", [(1, 40, 24), (5, 40, 24), (70, 96, 64), (33, 18, 128), (7, 22, 13), (200, 640, 192)])
def test_gelu_gated_pairs(M, N, K):
    lib, L = _lib()
    x, w = _rand(M, K, seed=1, scale=3.0), _rand(N, K, seed=2, scale=0.7)
    for dt, code in ((torch.float32, lib.DTYPE_F32), (BF, lib.DTYPE_BF16)):
        xd, wd = x.to(dt).cuda(), w.to(dt).cuda()
        p = xd.double().cpu() @ wd.double().cpu().T
        for act, want in ((lib.EPI_GELU, O.gelu_tanh(p[:, 0::2]) * (p[:, 1::2] + 0.5)),
                          (lib.EPI_NONE, p[:, 0::2] * torch.sigmoid(p[:, 0::2]) * (p[:, 1::2] + 0.5))):
            out = torch.empty((M, N // 2), dtype=torch.float32, device="cuda")
            lib.check_hybrid(L.pieh_linear_glu_act(_ptr(out), lib.DTYPE_F32, N // 2, _ptr(xd), code, K, _ptr(wd), code, M, N, K, act,
                                                   0.0, 0.5, _st()), "linear_glu_act")
            assert float((out.double().cpu() - want).abs().max()) < 1e-5 * float(want.abs().max())


@pytest.mark.parametrize("pairs", [0, 1])
@pytest.mark.parametrize("H,G,d,rot", [(4, 2, 16, 8), (3, 1, 10, 10), (2, 2, 70, 0), (8, 2, 64, 64)])
def test_per_head_norms_and_either_pairing(H, G, d, rot, pairs):
    lib, L = _lib()
    b, desc, keep, pages, n_pages = _batch([(5, 62), (3, 0)])
    T, eps = 8, 1e-4
    proj, qn, kn = _rand(T, (H + G) * d, seed=3, scale=2.0), 1 + _rand(d, seed=4, scale=0.5), 1 + _rand(d, seed=5, scale=0.5)
    pos = torch.tensor(list(range(62, 67)) + list(range(3)))
    q, k = proj[:, :H * d].view(T, H, d), proj[:, H * d:].view(T, G, d)
    half = rot // 2
    perm = list(range(d))                                                # half pairing = neighbour pairing of reordered features
    if not pairs:
        perm = [f for i in range(half) for f in (i, i + half)] + list(range(rot, d))
    back = [perm.index(i) for i in range(d)]
    turn = lambda v: O.rotate_pairs(v[:, :, perm], pos, rot, 300.0)[:, :, back] if rot else v
    wq, wk = turn(O.unit_rms(q, eps) * qn), turn(O.unit_rms(k, eps) * kn)
    cs = torch.stack([torch.stack([torch.cos(pos * 300.0 ** (-2.0 * i / rot)), torch.sin(pos * 300.0 ** (-2.0 * i / rot))], -1)
                      for i in range(half)], 1) if rot else None
    kp, vp = (torch.full((n_pages, 64, G, d), 9.0, device="cuda") for _ in range(2))
    pd, qnd, knd, csd = _cu(proj), _cu(qn), _cu(kn), _cu(cs) if rot else None
    at = lib.HybBiasAttn(H=H, G=G, d=d, dv=d, k_off=H * d, v_off=H * d, g_off=-1, q_norm=_ptr(qnd), k_norm=_ptr(knd), eps=eps, scale=1.0,
                         k_pages=_ptr(kp), v_pages=_ptr(vp), kv_dtype=lib.DTYPE_F32, rot_dims=rot, rot_cs=_ptr(csd), head_norm=1,
                         rot_pairs=pairs)
    out = torch.empty((T, H, d), device="cuda")
    lib.check_hybrid(L.pieh_bias_attn_prepare(_ptr(out), _ptr(pd), pd.stride(0), C.byref(at), C.byref(desc), _st()), "prepare")
    assert float((out.double().cpu() - wq).abs().max()) < 1e-5
    seq = [0] * 5 + [1] * 3
    for t in range(T):
        pg, o = pages[seq[t]][int(pos[t]) // 64], int(pos[t]) % 64
        assert float((kp[pg, o].double().cpu() - wk[t]).abs().max()) < 1e-5
        assert torch.equal(vp[pg, o].cpu(), k[t].float())                # the values: projected, neither normed nor turned
    assert int((kp != 9.0).any(-1).any(-1).sum()) == T
    del keep


def _visible(p, window, keep):
    return [j for j in range(p + 1) if not window or p - j < window or j < keep]


LATENT = [(4, 64, 0), (5, 64, 16), (16, 128, 64), (2, 128, 32), (17, 32, 32), (33, 16, 0), (5, 256, 64), (3, 48, 16), (20, 208, 16),
          (8, 64, 32), (16, 128, 0)]


@pytest.mark.parametrize("H,r,dr", LATENT)
@pytest.mark.parametrize("window,keep", [(0, 0), (20, 0), (7, 5), (64, 70)])
def test_decoding_over_a_shared_pool(H, r, dr, window, keep):
    """One row per sequence over bf16 pages: contexts at the borders of pages and slices, scores large enough that single keys
    stand out, a gate per head or per feature, a learned sink."""
    lib, L = _lib()
    D = r + dr
    ctxs = [0, 1, 15, 16, 63, 64, 130, 700]
    b, desc, keepalive, pages, n_pages = _batch([(1, c) for c in ctxs])
    T = len(ctxs)
    pool = torch.full((n_pages, 64, D), float("nan"), dtype=BF, device="cuda")             # what was never written must not count
    q = _rand(T, H * D, seed=7, scale=3.0)
    rows = [_rand(c + 1, D, seed=30 + i) for i, c in enumerate(ctxs)]
    for i, c in enumerate(ctxs):
        for pg in range(len(pages[i])):
            n = min(64, c + 1 - 64 * pg)
            pool[pages[i][pg], :n] = rows[i][64 * pg:64 * pg + n].to(BF).cuda()
    scale = 4.0 / D ** 0.5
    for gate_heads, sink in ((1, False), (0, True), (None, False)):
        gw = 0 if gate_heads is None else H if gate_heads else H * r
        gate, sinks = _rand(T, max(gw, 1), seed=8, scale=2.0), _rand(H, seed=9, scale=3.0)
        gd, qd, sd = _cu(gate), _cu(q), _cu(sinks)
        at = lib.HybBiasAttn(H=H, G=1, d=D, dv=r, g_off=0 if gw else -1, gate_heads=gate_heads or 0, scale=scale, window=window,
                             keep_first=keep if window else 0, k_pages=_ptr(pool), v_pages=_ptr(pool), kv_dtype=lib.DTYPE_BF16, v_ld=D,
                             sinks=_ptr(sd) if sink else None)
        out = torch.empty((T, H * r), dtype=BF, device="cuda")
        lib.check_hybrid(L.pieh_bias_attn_run(_ptr(out), lib.DTYPE_BF16, _ptr(qd), _ptr(gd), max(gw, 1), C.byref(at), C.byref(desc), _st()),
                         "attn_run")
        got = out.double().cpu().view(T, H, r)
        for i, c in enumerate(ctxs):
            js = torch.tensor(_visible(c, window, keep))
            kk = rows[i].to(BF).double()[js]
            s = q[i].float().to(BF).double().view(H, D) @ kk.T * scale
            if sink:
                s = torch.cat([s, sinks.float().double()[:, None]], 1)
            p = torch.softmax(s, -1)[:, :len(js)]
            want = p @ kk[:, :r]
            if gw:
                want = want * torch.sigmoid(gate[i].float().double().view(H, -1))
            assert float((got[i] - want).abs().max()) < 1.5e-2, (c, gate_heads, sink)
    del keepalive


def test_decoding_over_a_shared_pool_with_many_tokens():
    """Steps with more (token, head group) pairs than the GPU has room for clusters: 1, 2, 4 and 8 CTAs share a pair."""
    lib, L = _lib()
    H, r, dr, scale = 20, 64, 16, 0.3
    D = r + dr
    for T in (2, 12, 30, 60, 160):
        b, desc, keepalive, pages, n_pages = _batch([(1, 40 + 3 * i) for i in range(T)])
        pool = _rand(n_pages, 64, D, seed=11).to(BF).cuda()
        q = _rand(T, H * D, seed=12, scale=3.0)
        qd, out = _cu(q), torch.empty((T, H * r), dtype=BF, device="cuda")
        at = lib.HybBiasAttn(H=H, G=1, d=D, dv=r, g_off=-1, scale=scale, k_pages=_ptr(pool), v_pages=_ptr(pool), kv_dtype=lib.DTYPE_BF16, v_ld=D)
        lib.check_hybrid(L.pieh_bias_attn_run(_ptr(out), lib.DTYPE_BF16, _ptr(qd), None, 0, C.byref(at), C.byref(desc), _st()), "attn_run")
        for i in range(T):
            kk = pool[pages[i]].reshape(-1, D)[:41 + 3 * i].double().cpu()
            p = torch.softmax(q[i].float().to(BF).double().view(H, D) @ kk.T * scale, -1)
            assert float((out[i].double().cpu().view(H, r) - p @ kk[:, :r]).abs().max()) < 1.5e-2, (T, i)
        del keepalive


# ---- every mechanism alone, through the model ----------------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(pattern="l", ffs="-", loop=None), dict(pattern="l", ffs="-", loop=None, kv_rank=12, vdim=20), dict(pattern="a", ffs="-", loop=None),
    dict(pattern="l", ffs="-", loop=None, kv_rank=12, vdim=8), dict(pattern="l", ffs="-", loop=None, kv_rank=20, vdim=24),
    dict(pattern="a", ffs="-", loop=None, window=0), dict(pattern="a", ffs="-", loop=None, keep=0), dict(pattern="a", ffs="d", loop=None),
    dict(pattern="l", ffs="d", loop=None), dict(pattern="la", ffs="d"), dict(pattern="al", ffs="d-", loop=(0, 2, 3))])
def test_each_mixer_and_feed_forward_alone(kw):
    cfg, w, model = make(**kw)
    ids = toks(80)
    trace, otrace = [], []
    got = engine(model, graph=False).forward([("s", ids, list(range(80)))], trace=trace)
    want = O.forward(cfg, w, ids, otrace)
    assert len(trace) == len(otrace) == len(O.layer_runs(cfg))
    for a, b in zip(trace, otrace):
        assert err(a, b) < TOL32
    assert err(got, want) < TOL32
    assert err(whole(engine(model), ids), want) < TOL32                  # without the trace: norms and sums in one pass


@pytest.mark.parametrize("pattern,ffs,loop", [("la", "d", (0, 2, 2)), ("la", "-", (0, 1, 3)), ("lal", "d-d", (1, 3, 2)), ("lal", "d", (1, 2, 4)),
                                              ("la", "d", (0, 2, 1)), ("al", "d", (1, 2, 1)), ("lala", "d", (2, 3, 2)), ("al", "d", None)])
def test_loops(pattern, ffs, loop):
    cfg, w, model = make(pattern=pattern, ffs=ffs, loop=loop)
    assert len(model.cache_specs) == len(O.layer_runs(cfg))
    ids = toks(60, seed=2)
    want = O.forward(cfg, w, ids)
    if loop:                                                              # the map, its embedding half and the pass vectors count
        for name, edit in (("loop.step", lambda t: 0 * t), ("loop.in", lambda t: torch.cat([t[:, :64], 0 * t[:, 64:]], 1)),
                           ("loop.in", lambda t: torch.cat([0 * t[:, :64], t[:, 64:]], 1))):
            assert err(O.forward(cfg, dict(w, **{name: edit(w[name])}), ids), want) > 100 * TOL32
    assert err(in_portions(engine(model), ids, [31, 2, 1]), want) < TOL32


def test_the_pieces_of_the_latent_projection_are_folded_only_where_that_is_not_wider():
    for kw, q_rows, folded_q, folded_o in ((dict(kv_rank=16, vdim=16), 24, True, True), (dict(kv_rank=17, vdim=16), 24, False, False),
                                           (dict(kv_rank=14, vdim=12), 22, True, False), (dict(kv_rank=18, vdim=20), 24, False, True)):
        _, _, model = make(pattern="l", ffs="-", dim=16, rot_dim=8, loop=None, **kw)
        ly = model.layers[0]
        assert ly["q_rows"] == q_rows and (ly["ukT"] is None) == folded_q and (ly["uv"] is None) == folded_o
        assert ly["proj"].N % 8 == 0


@pytest.mark.parametrize("kw", [dict(), dict(kv_rank=12, vdim=20), dict(pattern="lala", ffs="d-d", loop=(1, 3, 2))])
def test_bf16_is_within_tolerance_everywhere(kw):
    cfg, w, model = make(dtype="bfloat16", **kw)
    ids = toks(150)
    want = O.forward(cfg, w, ids)
    assert err(in_portions(engine(model), ids, [70, 33, 1]), want) < TOL16
    assert err(whole(engine(model), ids), want) < TOL16


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kv_rank,rot_dim,dim,vdim,a_dim,keep", [(64, 32, 64, 40, 64, 4), (64, 64, 40, 72, 128, 70), (128, 32, 128, 128, 64, 1),
                                                                 (128, 64, 64, 64, 128, 0), (64, 0, 64, 64, 64, 140), (128, 0, 128, 40, 64, 64)])
def test_tensor_core_paths(dtype, kv_rank, rot_dim, dim, vdim, a_dim, keep):
    """Sizes at which prompt portions take the tiled attention kernels over bf16 pages and single tokens the shared-pool kernel,
    and the tcgen05 products (K a multiple of 64, more than 32 rows), with a window that ends inside a page."""
    cfg = O.random_config(width=128, pattern="al", heads=2, dim=dim, vdim=vdim, kv_rank=kv_rank, rot_dim=rot_dim, a_heads=4, a_kv=2,
                          a_dim=a_dim, a_rot=a_dim // 2, window=90, keep=keep, ff=128, loop=(0, 2, 1))
    cfg, w, model = make(cfg, dtype=dtype)
    ids = toks(300)
    e = rows_err(in_portions(engine(model), ids, [170, 80, 1]), O.forward(cfg, w, ids))
    assert float(e.max()) < (TOL32 if dtype == "float32" else TOL16)
    assert model.L.pieh_pipeline_error() == 0


# ---- prompts, decoding, portions, batches ---------------------------------------------------------------------------------------
def test_prefill_against_token_by_token_decoding():
    cfg, w, model = make()
    ids = toks(70)
    want = O.forward(cfg, w, ids)
    eng = engine(model)
    assert err(whole(eng, ids), want) < TOL32
    assert err(in_portions(eng, ids, [1]), want) < TOL32            # one token at a time from the first one (graph replay)
    assert err(in_portions(engine(model, graph=False), ids, [1]), want) < TOL32


@pytest.mark.parametrize("sizes", [[2], [3, 2, 5, 2, 64, 7, 2], [63, 2, 1], [64, 64, 2], [65, 1], [17, 16, 15, 2], [129, 2]])
def test_portions_of_several_sizes(sizes):
    cfg, w, model = make(pattern="lal", loop=(1, 3, 2))
    ids = toks(140, seed=3)
    assert err(in_portions(engine(model), ids, sizes), O.forward(cfg, w, ids)) < TOL32


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_match_each_alone(dtype):
    """bf16: latent and head sizes whose steps switch between the tile, shared-pool and run kernels with the mixture of the batch."""
    big = dict(width=128, dim=64, kv_rank=64, rot_dim=32, vdim=64, a_dim=64, a_rot=32) if dtype == "bfloat16" else {}
    cfg, w, model = make(pattern="al", dtype=dtype, window=21, keep=3, **big)
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
        assert err(torch.cat(got[k]), want[k]) < (TOL32 if dtype == "float32" else TOL16), k


def test_pages_and_slots_are_used_again():
    cfg, w, model = make()
    eng = engine(model, max_tokens=128, max_seqs=1)                  # two pages, one slot: everything is re-used
    for seed, n, sizes in ((11, 120, [50, 1]), (12, 100, [3, 64, 1]), (13, 128, [128]), (14, 9, [1]), (15, 2, [2]), (16, 1, [1])):
        ids = toks(n, seed=seed)
        assert err(in_portions(eng, ids, sizes, sid=seed), O.forward(cfg, w, ids)) < TOL32, seed
    assert eng.cache.allocator.get_num_free_pages() == 2 and len(eng.cache.free_slots) == 1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    cfg, w, model = make(window=50, keep=6, kv_rank=32, rot_dim=16, dtype=dtype)
    ids = toks(260, seed=9)
    assert err(in_portions(engine(model), ids, [20, 1]), O.forward(cfg, w, ids)) < (TOL32 if dtype == "float32" else TOL16)


def test_wanted_rows_in_any_order():
    cfg, w, model = make()
    ids, other = toks(40, seed=17), toks(9, seed=18)
    want, wo = O.forward(cfg, w, ids), O.forward(cfg, w, other)
    eng = engine(model)
    out = eng.forward([("s", ids, [39, 0, 7, 7]), ("t", other, []), ("u", other[:4], [3])])
    assert err(out, torch.cat([want[[39, 0, 7, 7]], wo[[3]]])) < TOL32
    assert eng.forward([("t", ids[:3], [])]).shape[0] == 0


# ---- inputs made so that one token stands out -----------------------------------------------------------------------------------
def _embed_as(w, tok, rows, target):
    """Makes the embedding of `tok` so that, after the first layer norm (made plain here), `rows` maps it onto `target`'s direction."""
    for k in ("l0.norm1", "l0.norm1.b"):
        w[k] = torch.full_like(w[k], 0.0 if k.endswith(".b") else 1.0)
    A = torch.cat([rows, torch.ones((1, rows.shape[1]), dtype=F)])          # ... and has no mean to take off
    e = torch.linalg.pinv(A) @ torch.cat([target, torch.zeros(1, dtype=F)])
    w["embed"][tok] = (e / e.pow(2).mean().sqrt()).to(BF)


def _plain_norm(v):
    d = v - v.mean()
    return d / d.pow(2).mean().sqrt()


def point_an_attention_key(w, cfg, q_tok, k_tok, gain):
    """The key of k_tok points where all query heads of q_tok look together, and the queries are raised: wherever both are visible
    that key takes most of the weight, so one key more or less shows."""
    m, f = cfg["layers"][0]["mixer"], lambda n: w[n].double()
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    w["l0.mix.k.b"] = torch.zeros_like(w["l0.mix.k.b"])
    q = (f("l0.mix.q") @ _plain_norm(f("embed")[q_tok]) + f("l0.mix.q.b")).view(G, H // G, d)
    look = O.unit_rms(q, 1e-5).sum(1) * f("l0.mix.q.norm") / f("l0.mix.k.norm")          # per kv head
    _embed_as(w, k_tok, f("l0.mix.k"), look.reshape(-1))
    w["l0.mix.q.norm"] = (gain * f("l0.mix.q.norm")).to(BF)


def point_a_latent_key(w, cfg, q_tok, k_tok, gain):
    m, f = cfg["layers"][0]["mixer"], lambda n: w[n].double()
    H, d, dr, r = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (f("l0.mix.q") @ _plain_norm(f("embed")[q_tok])).view(H, d + dr)[:, :d]
    look = torch.einsum("hdr,hd->r", f("l0.mix.uk").view(H, d, r), q) * f("l0.mix.dkv.norm")
    _embed_as(w, k_tok, f("l0.mix.dkv")[:r], look)
    qw = f("l0.mix.q").view(H, d + dr, -1).clone()
    qw[:, :d] *= gain                                                    # the rotated part keeps its size
    w["l0.mix.q"] = qw.reshape(H * (d + dr), -1).to(BF)


def _edge_cfg(**kw):
    return O.random_config(pattern="a", ffs="-", loop=None, a_heads=2, a_kv=1, a_rot=2, **kw)


def _other_mask(cfg, **kw):
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"].update(kw)
    return other


@pytest.mark.parametrize("window,probe,keep", [(6, 20, 3), (64, 64, 0), (64, 100, 4), (65, 130, 1), (90, 200, 70), (1, 9, 2), (2, 65, 0),
                                               (128, 191, 5)])
def test_keys_just_inside_and_just_outside_the_window(window, probe, keep):
    """One earlier token's key points at the probe's query, just inside the window or just outside it, so a window that is
    one token off changes the logits by far more than the tolerance."""
    cfg = _edge_cfg(window=window, keep=keep)
    cfg, w, model = make(cfg, edit=lambda w: point_an_attention_key(w, cfg, 89, 88, 3.0))
    for dist in (window - 1, window):
        ids = toks(probe + 6, seed=20 + dist, avoid=(88, 89))
        ids[probe - dist], ids[probe] = 88, 89
        want = O.forward(cfg, w, ids)
        size = window + (1 if dist == window else -1)
        if size > 0 and probe - dist >= keep and dist:
            assert float(rows_err(O.forward(_other_mask(cfg, size=size), w, ids), want)[probe]) > 50 * TOL32   # the case does show the edge
        assert err(whole(engine(model), ids), want) < TOL32                              # inside a prompt
        assert err(in_portions(engine(model), ids, [probe - 3, 1]), want) < TOL32        # decoded alone
        assert err(in_portions(engine(model), ids, [probe - dist + 1, 2]), want) < TOL32  # portions that start at the edge


@pytest.mark.parametrize("keep,window,probe", [(1, 5, 30), (3, 6, 64), (64, 7, 200), (65, 20, 129), (4, 64, 300), (63, 1, 100), (128, 10, 260)])
def test_the_first_tokens_that_stay_visible_and_the_next_ones(keep, window, probe):
    """The planted key sits at the last position that is kept, or at the first one that is not, the window long gone past it."""
    cfg = _edge_cfg(window=window, keep=keep)
    cfg, w, model = make(cfg, edit=lambda w: point_an_attention_key(w, cfg, 89, 88, 3.0))
    for at in (keep - 1, keep, 0):
        ids = toks(probe + 4, seed=50 + at, avoid=(88, 89))
        ids[at], ids[probe] = 88, 89
        want = O.forward(cfg, w, ids)
        off = {keep - 1: keep - 1, keep: keep + 1, 0: 0}[at]
        assert float(rows_err(O.forward(_other_mask(cfg, keep_first=off), w, ids), want)[probe]) > 50 * TOL32
        assert err(whole(engine(model), ids), want) < TOL32
        assert err(in_portions(engine(model), ids, [at + 1, 2, probe - at - 6, 1]), want) < TOL32
        assert err(in_portions(engine(model), ids, [2]), want) < TOL32


@pytest.mark.parametrize("a_dim", [64, 128])
@pytest.mark.parametrize("window,keep", [(70, 5), (70, 70), (20, 64), (3, 1)])
def test_window_and_kept_tokens_on_the_tiled_attention_kernel(a_dim, window, keep):
    """The same planted key in bf16 at head sizes where prompt portions run on 64-row tiles over whole pages: the edges fall inside
    a tile and inside a page."""
    cfg = O.random_config(width=160, pattern="a", ffs="-", loop=None, a_heads=2, a_kv=1, a_dim=a_dim, a_rot=2, window=window, keep=keep)
    cfg, w, model = make(cfg, dtype="bfloat16", edit=lambda w: point_an_attention_key(w, cfg, 89, 88, 2.0))
    probe = 150
    for at, off in ((probe - window + 1, dict(size=window - 1)), (probe - window, dict(size=window + 1)), (keep - 1, dict(keep_first=keep - 1)),
                    (keep, dict(keep_first=keep + 1))):
        ids = toks(probe + 40, seed=30 + at, avoid=(88, 89))
        ids[at], ids[probe] = 88, 89
        want = O.forward(cfg, w, ids)
        assert float(rows_err(O.forward(_other_mask(cfg, **off), w, ids), want)[probe]) > 3 * TOL16
        assert float(rows_err(whole(engine(model), ids), want)[probe]) < TOL16
        assert float(rows_err(in_portions(engine(model), ids, [100, 90]), want)[probe]) < TOL16
        assert float(rows_err(in_portions(engine(model), ids, [probe - 1, 1]), want)[probe]) < TOL16


@pytest.mark.parametrize("dtype,kv_rank,rot_dim", [("float32", 24, 8), ("bfloat16", 32, 16), ("bfloat16", 64, 32)])
@pytest.mark.parametrize("far,probe", [(0, 63), (0, 64), (63, 300), (64, 191), (128, 447)])
def test_a_latent_key_far_away(dtype, kv_rank, rot_dim, far, probe):
    """One key at a page's border or at the very start takes the probe's weight among hundreds of keys."""
    cfg = O.random_config(pattern="l", ffs="-", loop=None, width=96, heads=2, kv_rank=kv_rank, rot_dim=rot_dim, dim=32)
    cfg, w, model = make(cfg, dtype=dtype, edit=lambda w: point_a_latent_key(w, cfg, 89, 88, 6.0))
    tol = TOL32 if dtype == "float32" else TOL16
    ids = toks(probe + 3, seed=35 + far, avoid=(88, 89))
    ids[far], ids[probe] = 88, 89
    want = O.forward(cfg, w, ids)
    moved = list(ids)
    moved[far] = 3
    assert float(rows_err(O.forward(cfg, w, moved), want)[probe]) > 3 * TOL16
    for sizes in ([len(ids)], [far + 1, 50, 1] if far else [60, 1], [probe, 1]):
        e = rows_err(in_portions(engine(model), ids, sizes), want)
        assert float(e[probe]) < tol and float(e.max()) < 2 * tol, sizes


def test_looped_passes_keep_caches_of_their_own():
    """A far key planted in one pass only would be lost or doubled if passes shared pages: decode against whole prompts over three
    passes, the restatement shown to move when a pass is left out."""
    cfg, w, model = make(pattern="la", loop=(0, 2, 3), seed=4)
    ids = toks(100, seed=60)
    want = O.forward(cfg, w, ids)
    fewer = copy.deepcopy(cfg)
    fewer["loop"]["times"] = 2
    assert err(O.forward(fewer, w, ids), want) > 100 * TOL32
    eng = engine(model)
    assert err(in_portions(eng, ids, [66, 1]), want) < TOL32
    assert len({t["c"].data_ptr() for t in eng.cache.layers if "c" in t}) == 3


def test_gates_biases_and_norm_biases_count():
    cfg, w, model = make()
    ids = toks(50, seed=61)
    want = O.forward(cfg, w, ids)
    assert err(in_portions(engine(model), ids, [20, 2, 1]), want) < TOL32
    for name in ("l0.mix.g", "l1.mix.q.b", "l1.mix.k.b", "l0.norm1b.b", "l1.norm2b.b", "final.norm.b", "l0.norm1.b"):
        assert err(O.forward(cfg, dict(w, **{name: torch.zeros_like(w[name])}), ids), want) > 10 * TOL32, name


# ---- other sizes ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(heads=1, a_heads=1, a_kv=1), dict(heads=5, a_heads=9, a_kv=3), dict(a_heads=4, a_kv=4), dict(rot_dim=2, a_rot=2), dict(rot_dim=0, a_rot=0),
    dict(a_rot=16), dict(window=1, keep=0), dict(window=1000, keep=4), dict(window=5, keep=1000), dict(window=0), dict(keep=0), dict(keep=1),
    dict(scale=1.0, a_scale=1.0), dict(factor=1.0), dict(factor=32.0, a_base=100.0), dict(eps=1e-2), dict(loop=(1, 3, 3)), dict(loop=(3, 4, 2)),
    dict(loop=None), dict(loop=(0, 4, 1)), dict(width=72, dim=20, vdim=12, kv_rank=10, rot_dim=6, a_dim=12, a_rot=6, ff=28),
    dict(width=40, dim=4, vdim=4, kv_rank=8, rot_dim=8, a_dim=8, a_rot=4, ff=8), dict(width=65, vocab=91, dim=7, vdim=9, kv_rank=21, rot_dim=10,
                                                                                      a_dim=10, a_rot=6, ff=13),
    dict(dim=72, vdim=136, kv_rank=136, heads=1), dict(kv_rank=300, heads=2), dict(heads=17, dim=8, vdim=8, kv_rank=16, rot_dim=16),
    dict(dim=1, vdim=1, kv_rank=1, rot_dim=2, a_dim=2, a_rot=2), dict(vocab=513), dict(width=260, ff=300)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(kw, dtype):
    kw = dict(dict(loop=(0, 2, 2)), **kw)
    cfg, w, model = make(pattern="lala", ffs="d-dd", seed=2, dtype=dtype, **kw)
    ids = toks(75, vocab=cfg["vocab"], seed=4)
    e = rows_err(in_portions(engine(model), ids, [67, 2, 1]), O.forward(cfg, w, ids))
    assert float(e.max()) < (TOL32 if dtype == "float32" else 2 * TOL16)


# ---- the engine's own entry points ------------------------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler():
    cfg, w, model = make()
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
    cfg, w, model = make()
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
    cfg, w, _ = make(pattern="lal", loop=(1, 3, 2))
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
