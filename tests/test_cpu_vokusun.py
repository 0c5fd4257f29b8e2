"""CPU: the host side of the Vokusun family -- config reader and registry, the order of layer runs under a loop, the synthetic
checkpoint's tensor names, rotation frequencies, what the latent projection folds, one cache entry per run -- and checks of the
plain restatement itself (tests/vokusun_oracle.py) against closed forms, so that what the GPU tests compare with is pinned."""
import copy
import math

import pytest
import torch

import vokusun_oracle as O

F = torch.float64


def test_registry_and_config_reader():
    from proxy_inference_engine_b200.checkpoint import MODEL_REGISTRY, model_kind
    from proxy_inference_engine_b200.vokusun import VokusunArgs
    cfg = O.random_config(eps=3e-4)
    a = VokusunArgs.from_dict(cfg)
    assert (a.vocab, a.width, a.norm_eps, a.loop) == (90, 64, 3e-4, {"start": 0, "stop": 2, "times": 2})
    assert VokusunArgs.from_dict(a.to_dict()).layers == a.layers and VokusunArgs.from_dict(a.to_dict()).loop == a.loop
    assert model_kind(cfg) == "Vokusun" and "Vokusun" in MODEL_REGISTRY
    b = VokusunArgs.from_dict({k: v for k, v in cfg.items() if k not in ("loop", "norm")})
    assert b.loop is None and b.norm_eps == 1e-5
    for edit in (lambda c: c.pop("vocab"),
                 lambda c: c["layers"][0].update(type="parallel"),
                 lambda c: c["layers"][0]["mixer"].pop("kv_rank"),
                 lambda c: c["layers"][1]["mixer"].pop("scale"),
                 lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
                 lambda c: c["layers"][1]["mixer"].update(vdim=8),
                 lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
                 lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
                 lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1),
                 lambda c: c["layers"][0]["mlp"].update(kind="moe"),
                 lambda c: c["loop"].update(stop=3),
                 lambda c: c["loop"].update(start=2),
                 lambda c: c["loop"].update(times=0)):
        bad = copy.deepcopy(cfg)
        edit(bad)
        with pytest.raises(ValueError):
            VokusunArgs.from_dict(bad)


def test_order_of_layer_runs():
    from proxy_inference_engine_b200.vokusun import VokusunArgs
    runs = lambda **kw: VokusunArgs.from_dict(O.random_config(**kw)).runs()
    assert runs(pattern="lal", loop=None) == [(0, None), (1, None), (2, None)]
    assert runs(pattern="lal", loop=(0, 3, 1)) == [(0, 0), (1, None), (2, None)]
    assert runs(pattern="lal", loop=(1, 2, 3)) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]
    assert runs(pattern="lala", loop=(1, 3, 2)) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    for kw in (dict(pattern="lal", loop=None), dict(pattern="lala", loop=(1, 3, 2)), dict(pattern="la", loop=(1, 2, 4))):
        assert O.layer_runs(O.random_config(**kw)) == runs(**kw)                        # the restatement's own order agrees


def test_random_weights_cover_every_tensor_the_restatement_reads():
    from proxy_inference_engine_b200.vokusun import VokusunArgs, random_weights
    cfg = O.random_config(pattern="lala", ffs="d-d", loop=(1, 3, 2))
    w = random_weights(VokusunArgs.from_dict(cfg), seed=3)
    for name in ("embed", "head", "final.norm.b", "loop.in", "loop.step", "l0.norm1b.b", "l0.norm2b", "l0.mix.dkv.norm", "l0.mix.g",
                 "l1.mix.q.b", "l1.mix.k.norm", "l0.mlp.gate"):
        assert name in w, name
    assert "l1.norm2" not in w and "l1.mlp.up" not in w and "l1.mix.v" not in w
    assert w["loop.in"].shape == (64, 128) and w["loop.step"].shape == (2, 64) and w["l0.mix.dkv"].shape == (32, 64)
    trace = []
    logits = O.forward(cfg, w, [1, 2, 3, 4, 5, 6, 7, 8, 9], trace)
    assert logits.shape == (9, 90) and len(trace) == 6 and bool(torch.isfinite(logits).all())


def test_rotation_frequencies_carry_the_linear_scaling():
    from proxy_inference_engine_b200.latent import rotary_frequencies
    f = rotary_frequencies({"base": 100.0, "dims": 4, "scaling": {"factor": 8.0}})
    assert f == [1.0 / 8, 0.1 / 8] and rotary_frequencies({"base": 100.0, "dims": 4}) == [1.0, 0.1]


def test_the_bench_configurations_are_valid():
    from proxy_inference_engine_b200.hybrid_bench import SIZES, vokusun_config
    from proxy_inference_engine_b200.vokusun import VokusunArgs
    for size in SIZES:
        a = VokusunArgs.from_dict(vokusun_config(size))
        assert len(a.runs()) == len(SIZES[size]["pattern"])


def test_one_cache_entry_per_layer_run():
    from proxy_inference_engine_b200.cache import HybridCache

    class _Alloc:        # the allocator lives in the native library; this one hands out ids the same way
        def __init__(self, n, *_a, **_k): self.free = list(range(n - 1, -1, -1))
        def allocate_pages(self, n): return [self.free.pop() for _ in range(n)]
        def free_pages(self, ps): self.free += list(reversed(ps))
        def get_num_free_pages(self): return len(self.free)
    import proxy_inference_engine_b200.paging as paging
    lat, att = {"pages": {"c": (32,)}}, {"pages": {"k": (2, 16), "v": (2, 16)}}
    orig, paging.PageAllocator = paging.PageAllocator, _Alloc
    try:
        c = HybridCache([lat, att, lat, att], 130, 2, "cpu", torch.bfloat16)     # a looped pair: four runs
    finally:
        paging.PageAllocator = orig
    assert c.n_pages == 3 and c.layers[0]["c"].shape == (3, 64, 32) and c.layers[1]["v"].shape == (3, 64, 2, 16)
    assert c.layers[0]["c"].data_ptr() != c.layers[2]["c"].data_ptr()            # each pass has its own


# ---- the restatement against closed forms --------------------------------------------------------------------------------------
def test_layer_norm_takes_the_mean_off_first():
    x = torch.tensor([[1.0, 3.0], [5.0, 5.0]], dtype=F)
    w, b = torch.tensor([2.0, 3.0], dtype=F), torch.tensor([0.5, -0.5], dtype=F)
    y = O.layer_norm(x, w, b, 0.0 + 1e-12)
    assert torch.allclose(y[0], torch.tensor([-1.5, 2.5], dtype=F), atol=1e-9)
    assert torch.allclose(y[1], b, atol=1e-12)                                   # a constant row is its bias
    assert abs(float(O.layer_norm(x, w, b, 3.0)[0, 0]) - (0.5 - 2.0 / 2.0)) < 1e-12      # eps inside the root: 1 / sqrt(1 + 3)


def test_rotation_turns_neighbouring_features_and_is_slowed_by_the_factor():
    x = torch.zeros((3, 1, 6), dtype=F)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    y = O.rotate_pairs(x, torch.tensor([0, 1, 2]), 4, 100.0)
    assert torch.allclose(y[0], x[0]) and float(y[1, 0, 5]) == 7.0               # position 0 and unrotated features
    assert torch.allclose(y[2, 0, :4], torch.tensor([math.cos(2.0), math.sin(2.0), 0.0, 0.0], dtype=F), atol=1e-12)
    slow = O.rotate_pairs(x, torch.tensor([0, 4, 8]), 4, 100.0, factor=4.0)
    assert torch.allclose(slow, y, atol=1e-12)
    q, k = torch.randn((1, 1, 4), dtype=F), torch.randn((1, 1, 4), dtype=F)      # scores depend on the distance only
    dot = lambda a, b: float((O.rotate_pairs(q, torch.tensor([a]), 4, 50.0) * O.rotate_pairs(k, torch.tensor([b]), 4, 50.0)).sum())
    assert abs(dot(9, 4) - dot(25, 20)) < 1e-9


def test_which_keys_a_query_sees():
    assert O.visible(3, None) == [0, 1, 2, 3]
    assert O.visible(9, {"size": 3, "keep_first": 2}) == [0, 1, 7, 8, 9]
    assert O.visible(3, {"size": 3, "keep_first": 2}) == [0, 1, 2, 3]            # the window has not left the first ones yet
    assert O.visible(9, {"size": 1}) == [9] and O.visible(2, {"size": 1, "keep_first": 8}) == [0, 1, 2]


def test_attention_weights_and_head_groups():
    q = torch.zeros((3, 4, 2), dtype=F)
    k = torch.zeros((3, 2, 2), dtype=F)
    v = torch.tensor([[[1.0], [10.0]], [[2.0], [20.0]], [[6.0], [60.0]]], dtype=F)
    out = O.softmax_attention(q, k, v, 1.0, None)                                # equal scores: the plain mean
    assert torch.allclose(out[2, :, 0], torch.tensor([3.0, 3.0, 30.0, 30.0], dtype=F))
    q[2, 3, 0] = 1.0
    k[1, 1, 0] = 2.0 * math.log(3.0)                                             # head 3 reads group 1: weight 3 against 1 and 1
    out = O.softmax_attention(q, k, v, 0.5, None)
    assert abs(float(out[2, 3, 0]) - (10 + 3 * 20 + 60) / 5) < 1e-12 and abs(float(out[2, 2, 0]) - 30.0) < 1e-12


def test_values_are_the_projected_keys_and_the_latent_gate_is_per_head():
    W = d = 4
    z, eye = (lambda *s: torch.zeros(s, dtype=F)), torch.eye(4, dtype=F)
    w = {"q": z(d, W), "q.b": z(d), "k": 2 * eye, "k.b": torch.tensor([1.0, 0, 0, 0], dtype=F), "q.norm": torch.ones(d, dtype=F),
         "k.norm": torch.full((d,), 9.0, dtype=F), "o": eye}
    h = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=F)
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "scale": 1.0, "rot": {"base": 10.0, "dims": 4}, "mask": {"size": 5, "keep_first": 0}}
    assert torch.allclose(O.shared_kv_attention(h, w, "", m, 1e-6)[0], torch.tensor([3.0, 4.0, 6.0, 8.0], dtype=F))    # bias in, no norm
    w = {"q": z(2 * 2, W), "dkv": eye[:2], "dkv.norm": torch.tensor([1.0, 5.0], dtype=F), "uk": z(2, 2),
         "uv": torch.tensor([[1.0, 0], [0, 1.0]], dtype=F), "g": z(2, W), "o": torch.eye(W, 2, dtype=F)}
    w["g"][1, 0] = math.log(3.0)
    m = {"heads": 2, "dim": 1, "rot_dim": 0, "vdim": 1, "kv_rank": 2, "scale": 1.0}
    w["q"] = z(2, W)
    c = O.unit_rms(h[:, :2], 0.0)[0]
    out = O.latent_attention(h, w, "", m, 0.0)[0]
    assert abs(float(out[0]) - 0.5 * float(c[0])) < 1e-12                        # sigmoid(0)
    assert abs(float(out[1]) - 0.75 * 5 * float(c[1])) < 1e-12                   # sigmoid(log 3)


def test_loop_openings_and_the_sandwich_by_hand():
    """One attention layer run twice without a feed-forward: every pass starts from loop.in [x; x0] + its own vector."""
    from proxy_inference_engine_b200.vokusun import VokusunArgs, random_weights
    cfg = O.random_config(pattern="a", ffs="-", loop=(0, 1, 2), width=24, a_heads=2, a_kv=1, a_dim=8, a_rot=4)
    w = random_weights(VokusunArgs.from_dict(cfg), seed=1)
    trace = []
    logits = O.forward(cfg, w, [3, 4, 3], trace)
    f = lambda n: w[n].double()
    ln = lambda v, n: O.layer_norm(v, f(n), f(n + ".b"), 1e-5)
    mix = {k[len("l0.mix."):]: f(k) for k in w if k.startswith("l0.mix.")}
    x0 = f("embed")[[3, 4, 3]]
    x = x0
    for t in range(2):
        x = x @ f("loop.in")[:, :24].T + x0 @ f("loop.in")[:, 24:].T + f("loop.step")[t]
        x = x + ln(O.shared_kv_attention(ln(x, "l0.norm1"), mix, "", cfg["layers"][0]["mixer"], 1e-5), "l0.norm1b")
        assert torch.allclose(trace[t], x, atol=1e-12)
    assert torch.allclose(logits, ln(x, "final.norm") @ f("head").T, atol=1e-12)


def test_gated_feed_forward():
    w = {"gate": torch.tensor([[100.0], [-100.0]], dtype=F), "up": torch.tensor([[2.0], [3.0]], dtype=F), "down": torch.tensor([[1.0, 10.0]], dtype=F)}
    assert abs(float(O.gated_ff(torch.tensor([[1.0]], dtype=F), w, "")) - 200.0) < 1e-9      # gelu(100) = 100, gelu(-100) = 0
    z = torch.linspace(-4, 4, 9, dtype=F)
    assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)
