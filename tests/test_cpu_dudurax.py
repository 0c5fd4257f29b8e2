"""CPU: the host side of the Dudurax family -- config reader and registry, the synthetic checkpoint's tensor names, the cache
entries (latent pages, recurrent states, the last token of every slot) -- and checks of the plain restatement itself
(tests/dudurax_oracle.py) against closed forms, so that what the GPU tests compare with is pinned."""
import copy
import math

import pytest
import torch

import dudurax_oracle as O

F = torch.float64


def test_registry_and_config_reader():
    from proxy_inference_engine_b200.checkpoint import MODEL_REGISTRY, model_kind
    from proxy_inference_engine_b200.dudurax import DuduraxArgs
    cfg = O.random_config()
    a = DuduraxArgs.from_dict(cfg)
    assert (a.vocab, a.width, a.norm_eps, a.alpha, a.embed_scale) == (90, 64, 1e-5, 1.7, 2.0)
    assert a.bigram == {"buckets": 61, "mul_prev": 5, "mul_cur": 3}
    assert DuduraxArgs.from_dict(a.to_dict()).to_dict() == a.to_dict()
    assert model_kind(cfg) == "Dudurax" and "Dudurax" in MODEL_REGISTRY
    plain = {k: v for k, v in cfg.items() if k not in ("embedding", "postln_alpha", "norm")}
    b = DuduraxArgs.from_dict(plain)
    assert b.bigram is None and (b.alpha, b.embed_scale, b.norm_eps) == (1.0, 1.0, 1e-6) and "bigram" not in b.to_dict()["embedding"]
    for edit in (lambda c: c.pop("width"),
                 lambda c: c["layers"][0].update(type="attention"),
                 lambda c: c["layers"][0]["mixer"].pop("tau"),
                 lambda c: c["layers"][0]["mixer"].update(tau=0.0),
                 lambda c: c["layers"][1]["mixer"].pop("kv_rank"),
                 lambda c: c["layers"][1]["mixer"].pop("scale"),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10),
                 lambda c: c["layers"][0]["mlp"].update(kind="glu"),
                 lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3),
                 lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5),
                 lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
                 lambda c: c["embedding"]["bigram"].update(buckets=0)):
        bad = copy.deepcopy(cfg)
        edit(bad)
        with pytest.raises(ValueError):
            DuduraxArgs.from_dict(bad)


def test_random_weights_cover_every_tensor_the_restatement_reads():
    from proxy_inference_engine_b200.dudurax import DuduraxArgs, random_weights
    cfg = O.random_config(pattern="gahg", ffs="dm-m")
    w = random_weights(DuduraxArgs.from_dict(cfg), seed=3)
    for name in ("embed", "bigram", "head", "final.norm", "l0.norm2", "l0.mix.a1", "l0.mix.a2.b", "l0.mlp.up", "l1.mix.dkv.norm",
                 "l1.mix.uk", "l1.mlp.router", "l1.mlp.correction", "l1.mlp.e5.gate", "l2.mix.norm", "l3.mlp.e0.down"):
        assert name in w, name
    assert "l2.norm2" not in w and "l2.mlp.up" not in w and "l1.mlp.e6.gate" not in w       # no feed-forward; identity: no tensors
    assert w["bigram"].shape == (62, 64) and w["l1.mlp.router"].shape == (8, 64) and w["l1.mlp.correction"].shape == (8,)
    assert w["l1.mix.q"].shape == (4 * 24, 64) and w["l1.mix.dkv"].shape == (32, 64) and w["l2.mix.norm"].shape == (20,)
    trace = []
    logits = O.forward(cfg, w, [1, 2, 3, 4, 5, 6, 7, 8, 9], trace)
    assert logits.shape == (9, 90) and len(trace) == 4 and bool(torch.isfinite(logits).all())


def test_cache_entries_and_the_last_token_slot():
    from proxy_inference_engine_b200.cache import HybridCache

    class _Alloc:        # the allocator lives in the native library; this one hands out ids the same way
        def __init__(self, n, *_a, **_k): self.free = list(range(n - 1, -1, -1))
        def allocate_pages(self, n): return [self.free.pop() for _ in range(n)]
        def free_pages(self, ps): self.free += list(reversed(ps))
        def get_num_free_pages(self): return len(self.free)
    import proxy_inference_engine_b200.paging as paging
    orig, paging.PageAllocator = paging.PageAllocator, _Alloc
    try:
        c = HybridCache([{"slots": {"state": (2, 16, 24)}}, {"pages": {"c": (32,)}}, {"int_slots": {"last_token": ()}}], 130, 2, "cpu",
                        torch.bfloat16)
    finally:
        paging.PageAllocator = orig
    assert c.layers[1]["c"].shape == (3, 64, 32) and c.layers[1]["c"].dtype == torch.bfloat16
    assert c.layers[0]["state"].shape == (2, 2, 16, 24) and c.layers[0]["state"].dtype == torch.float32
    assert c.layers[2]["last_token"].shape == (2,) and c.layers[2]["last_token"].dtype == torch.int32
    assert {"state", "last_token"} <= c.slot_keys and "c" not in c.slot_keys      # what a replayed warm-up has to put back


# ---- the restatement against closed forms --------------------------------------------------------------------------------------
def test_pair_rows_and_embedding():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert O.pair_row(None, 7, b) == 10 and O.pair_row(2, 7, b) == 4 and O.pair_row(7, 2, b) == 9
    w = {"embed": torch.arange(8, dtype=F)[:, None].repeat(1, 2), "bigram": 100 * torch.arange(11, dtype=F)[:, None].repeat(1, 2)}
    x = O.embedding([7, 2, 7], w, {"scale": 0.5, "bigram": b})
    assert x[:, 0].tolist() == [3.5 + 1000, 1 + 900, 3.5 + 400]                  # the pair rows are not scaled
    assert O.embedding([7], w, {"scale": 0.5})[0, 0] == 3.5


def test_rotation_pairs_feature_i_with_i_plus_half():
    x = torch.zeros((3, 1, 6), dtype=F)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    y = O.rotate_half(x, torch.tensor([0, 1, 2]), 4, 100.0)
    assert torch.allclose(y[0], x[0]) and float(y[1, 0, 5]) == 7.0                    # position 0 and unrotated features
    assert torch.allclose(y[2, 0, :4], torch.tensor([math.cos(2.0), 0.0, math.sin(2.0), 0.0], dtype=F), atol=1e-12)


def test_window_counts_the_query_itself():
    q = k = torch.zeros((4, 1, 2), dtype=F)
    v = torch.tensor([1.0, 2.0, 4.0, 8.0], dtype=F).view(4, 1, 1)
    assert torch.allclose(O.window_softmax_attention(q, k, v, 1.0, 2)[:, 0, 0], torch.tensor([1.0, 1.5, 3.0, 6.0], dtype=F))
    assert torch.allclose(O.window_softmax_attention(q, k, v, 1.0, 1)[:, 0, 0], v[:, 0, 0])


def test_gated_linear_attention_closed_form():
    k = torch.tensor([[1.0, 1.0, 0.0], [0.0, 0.0, 1.0]], dtype=F).view(2, 1, 3)
    v = torch.tensor([[1.0, 2.0], [10.0, 20.0]], dtype=F).view(2, 1, 2)
    q = torch.tensor([[1.0, 0.0, 5.0], [1.0, 1.0, 1.0]], dtype=F).view(2, 1, 3)
    dec = torch.tensor([[9.0, 9.0, 9.0], [0.0, 0.5, 1.0]], dtype=F).view(2, 1, 3)    # the first decay meets an empty state
    o = O.gla_scan(q, k, v, dec)
    assert torch.allclose(o[0, 0], v[0, 0]) and torch.allclose(o[1, 0], 0.5 * v[0, 0] + v[1, 0])   # the decay acts per key channel
    w = {"a1": torch.eye(1, 2, dtype=F), "a2": torch.tensor([[1.0]], dtype=F), "a2.b": torch.tensor([-1.0], dtype=F)}
    d = O.channel_decays(torch.tensor([[1.0, 50.0]], dtype=F), w, "", 4.0)
    assert abs(float(d[0, 0]) - 0.5 ** 0.25) < 1e-12


def test_clamped_expert_and_gelu():
    w = {"gate": torch.tensor([[3.0]], dtype=F), "up": torch.tensor([[-5.0]], dtype=F), "down": torch.tensor([[2.0]], dtype=F)}
    y = O.clamped_expert(torch.tensor([1.0], dtype=F), w, "", 1.5)
    assert abs(float(y[0]) - 2 * 1.5 / (1 + math.exp(-1.702 * 1.5)) * (1 - 1.5)) < 1e-12
    y = O.clamped_expert(torch.tensor([-1.0], dtype=F), w, "", 1.5)                   # the gate is clamped from above only
    assert abs(float(y[0]) - 2 * -3.0 / (1 + math.exp(1.702 * 3.0)) * (1 + 1.5)) < 1e-12
    z = torch.linspace(-4, 4, 41, dtype=F)
    assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_router_choices():
    z = torch.log(torch.tensor([0.1, 0.2, 0.3, 0.05, 0.25, 0.1], dtype=F))
    r = {"top": 2, "scale": 10.0}
    pick, w, gap = O.route(z, torch.zeros(6, dtype=F), r)
    assert pick == [2, 4] and abs(w[0] - 3.0) < 1e-12 and abs(w[1] - 2.5) < 1e-12 and abs(gap - 0.05) < 1e-12    # not renormalised
    corr = torch.tensor([-1.0, -2.0, -2.0, -2.0, -2.0, -1.0], dtype=F)                # chooses, but does not weigh
    pick, w, _ = O.route(z, corr, r)
    assert pick == [0, 5] and abs(w[0] - 1.0) < 1e-12 and abs(w[1] - 1.0) < 1e-12
    # groups {0 1} {2 3} {4 5} score by their BEST choice score; negative scores do not lose to what is not eligible
    pick, w, _ = O.route(z, corr, dict(r, groups={"count": 3, "keep": 1}))
    assert pick == [0, 1]
    pick, _, gap = O.route(z, torch.zeros(6, dtype=F), dict(r, groups={"count": 3, "keep": 2}))
    assert pick == [2, 4] and abs(gap - 0.05) < 1e-12


def test_identity_experts_return_the_input():
    w = {"router": torch.zeros((3, 2), dtype=F), "correction": torch.tensor([0.0, 1.0, 2.0], dtype=F),
         "e0.gate": torch.ones((1, 2), dtype=F), "e0.up": torch.ones((1, 2), dtype=F), "e0.down": torch.ones((2, 1), dtype=F)}
    mlp = {"expert": {"ff": 1, "limit": 9.0}, "router": {"experts": 1, "identity": 2, "top": 2, "scale": 6.0}}
    h = torch.tensor([[2.0, -1.0]], dtype=F)
    assert torch.allclose(O.moe(h, w, "", mlp), 6.0 * (2 / 3) * h)                    # two identity experts of score 1/3 each


def test_the_norm_sits_on_the_residual():
    from proxy_inference_engine_b200.dudurax import DuduraxArgs, random_weights
    cfg = O.random_config(pattern="g", ffs="d", width=16, heads=1, dim=8, alpha=0.25)
    w = random_weights(DuduraxArgs.from_dict(cfg), seed=1)
    trace = []
    O.forward(cfg, w, [3, 4], trace)
    f = {k: v.double() for k, v in w.items()}
    x = O.embedding([3, 4], f, cfg["embedding"])
    y = 0.25 * x + O.gla_mixer(x, f, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)      # the mixer reads x itself
    x = y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-5) * f["l0.norm1"]
    y = 0.25 * x + O.gelu_tanh(x @ f["l0.mlp.up"].T) @ f["l0.mlp.down"].T
    assert torch.allclose(trace[0], y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-5) * f["l0.norm2"], atol=1e-12)
