"""Dudurax: a decoder-only model whose norms sit ON the residual -- ``x <- rms(alpha x + f(x)) w`` after every sublayer, the
sublayers reading x itself -- over a token embedding plus a hashed embedding of the (previous, current) token pair.  A
layer's mixer is one of
    gla, gla_2         gated linear attention: a matrix state per head with a decay per key channel (low-rank logits, the
                       tau-th root of a sigmoid), per-head output norm, silu gate; the two names carry sizes of their own
    latent_attention   sliding-window softmax attention whose keys and values are expanded from one small latent per token,
                       with one extra rotated key part shared by all heads; only latent and rotated part are cached
and its feed-forward is dense (tanh-form gelu) or a mixture of clamped gated experts: softmax scores over experts AND
identity experts (which return their input), a learned correction that takes part in choosing only, group-limited choice
(a group scores its best expert), weights not renormalised.
Served through the ragged step of libpie_b200_hybrid.so like the other hybrid families: same ``BatchDetails``, same
``cache.HybridCache`` (pages, state slots, and the last token of every sequence), same ``engine.HybridEngine``.

config.json: ``architecture`` "Dudurax"; ``vocab``, ``width``, ``norm.eps``, ``postln_alpha``, ``embedding`` {scale, bigram
{buckets, mul_prev, mul_cur} | absent} and ``layers``, a list of ``{"type": ..., "mixer": {...}, "mlp": {...} | null}`` with
    gla, gla_2:        heads, dim, vdim, tau
    latent_attention:  heads, dim, rot_dim, vdim, kv_rank, scale, mask.size (absent: all earlier tokens), rot {base, dims}
    mlp:               {"kind": "dense", "ff"}  or  {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts",
                       "identity", "top", "scale", "groups" {"count", "keep"} | absent}}
Tensors: ``embed``, ``bigram`` [buckets + 1, width], ``head``, ``final.norm``, per layer i ``l<i>.norm1|norm2``,
``l<i>.mix.q|k|v|g|o|norm|a1|a2|a2.b`` or ``l<i>.mix.q|dkv|dkv.norm|uk|uv|o``, ``l<i>.mlp.up|down`` or
``l<i>.mlp.router|correction`` and ``l<i>.mlp.e<j>.gate|up|down``.

One step over a ``ragged.BatchDetails`` (x: fp32 residual [T, W]; h: the same rows in the act dtype, what products read):

    x, h   = embed_pairs(tokens; last token of every sequence in its slot)
    per layer:
      gla:      p = linear(h; [q | k | v | g | a1] fused)
                one row per sequence: gla_step (decays, update, read-out, head norm, gate: one launch)
                otherwise:            gla_decay -> gla_scan (state in the slot; long portions in parallel segments)
                                      -> gated_group_norm (head norm, silu(g))
                y = linear(.; o)
      latent:   the queries go INTO the latent space, (uk^T q) . c = q . (uk c), so keys and values are never expanded:
                kv_rank <= dim:  uk^T q is one matrix formed at load;  p = linear(h; [per head: uk^T q | rotated part] [dkv])
                otherwise:       p = linear(h; [q | dkv]), then one batched product with the heads' uk^T
                latent_rot_prepare (latent norm, rotations, append to pages)
                bias_attn_run over the pages: one shared key "head" of kv_rank + rot_dim features whose values are its leading
                kv_rank features
                kv_rank <= vdim: o uv is one matrix formed at load;  otherwise a batched product with the heads' uv first
                y = linear(.; o)
      x, h   = sum_norm(alpha x + y; norm1)
      dense:    y = linear(linear_act(h; up, gelu); down)
      moe:      z = linear(h; router) -> moe_route -> two grouped products (clamped gated pair between them); the weighted sum is
                formed inside the norm, an identity expert contributing x itself
      x, h   = sum_norm(alpha x + y | mixture; norm2)
    logits   = linear(stream_norm(x[wanted rows]; final norm); head)                                     fp32

dtype "bfloat16": matrix-product inputs and the cached latents are bf16; accumulation, residual, norms, rotation angles,
attention scores and weights, routing, decays and the recurrence are fp32.  dtype "float32": weights are widened once and
every product is a plain fp32 multiply-add.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass, field

import torch

from . import _lib
from ._lib import DTYPE_BF16, DTYPE_F32, EPI_GELU, EPI_NONE, HybGla, HybMixSum, HybMoePlan
from .babodra import interleave_pairs
from .cache import HybridCache
from .golitar import _Linear, _p, _stream
from .latent import LatentMixin
from .ragged import BatchDetails

GLA = ("gla", "gla_2")
MIXERS = GLA + ("latent_attention",)
GLU_SLOPE, GLU_OFFSET = 1.702, 1.0     # expert: g sigmoid(1.702 g) (u + 1), both halves clamped


@dataclass
class DuduraxArgs:
    vocab: int
    width: int
    layers: list
    norm_eps: float = 1e-6
    alpha: float = 1.0
    embed_scale: float = 1.0
    bigram: dict | None = None
    architecture: str = "Dudurax"
    raw: dict = field(default_factory=dict)

    @classmethod
    def from_dict(cls, cfg: dict) -> "DuduraxArgs":
        for key in ("vocab", "width", "layers"):
            if key not in cfg:
                raise ValueError(f"Dudurax config: '{key}' is missing")
        for i, ly in enumerate(cfg["layers"]):
            if ly.get("type") not in MIXERS:
                raise ValueError(f"Dudurax config: layer {i} has unknown type {ly.get('type')!r}")
            m = ly.get("mixer") or {}
            need = ("heads", "dim", "vdim", "tau") if ly["type"] in GLA else ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale")
            for key in need:
                if key not in m:
                    raise ValueError(f"Dudurax config: layer {i} mixer lacks '{key}'")
            if ly["type"] in GLA:
                if not float(m["tau"]) > 0:
                    raise ValueError(f"Dudurax config: layer {i}: tau must be positive")
            else:
                rot = m.get("rot")
                if rot and (int(rot["dims"]) % 2 or int(rot["dims"]) > int(m["rot_dim"])):
                    raise ValueError(f"Dudurax config: layer {i}: rot.dims must be even and at most rot_dim")
            mlp = ly.get("mlp")
            if mlp:
                if mlp.get("kind") not in ("dense", "moe"):
                    raise ValueError(f"Dudurax config: layer {i} has unknown feed-forward kind {mlp.get('kind')!r}")
                if mlp["kind"] == "moe":
                    r = mlp["router"]
                    n, grp = int(r["experts"]) + int(r.get("identity") or 0), r.get("groups") or {"count": 1, "keep": 1}
                    if n % int(grp["count"]) or not 1 <= int(grp["keep"]) <= int(grp["count"]):
                        raise ValueError(f"Dudurax config: layer {i}: groups do not divide the router's outputs")
                    if n // int(grp["count"]) * int(grp["keep"]) < int(r["top"]):
                        raise ValueError(f"Dudurax config: layer {i}: the kept groups hold fewer than 'top' experts")
        emb = cfg.get("embedding") or {}
        bigram = emb.get("bigram") or None
        if bigram:
            bigram = {k: int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")}
            if bigram["buckets"] < 1:
                raise ValueError("Dudurax config: bigram.buckets must be positive")
        return cls(vocab=int(cfg["vocab"]), width=int(cfg["width"]), layers=list(cfg["layers"]),
                   norm_eps=float((cfg.get("norm") or {}).get("eps", 1e-6)), alpha=float(cfg.get("postln_alpha", 1.0)),
                   embed_scale=float(emb.get("scale", 1.0)), bigram=bigram,
                   architecture=cfg.get("architecture", "Dudurax"), raw=cfg)

    def to_dict(self) -> dict:
        emb = {"scale": self.embed_scale}
        if self.bigram:
            emb["bigram"] = dict(self.bigram)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "postln_alpha": self.alpha, "embedding": emb, "layers": self.layers}


class DuduraxModel(LatentMixin):
    def __init__(self, args: DuduraxArgs, weights: dict, device="cuda", dtype: str = "bfloat16"):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype must be 'bfloat16' or 'float32'")
        self.args, self.device, self.dtype = args, device, dtype
        self.exact = dtype == "float32"
        self.act_torch = torch.float32 if self.exact else torch.bfloat16
        self.act = DTYPE_F32 if self.exact else DTYPE_BF16
        self.L = _lib.load_hybrid(build_if_missing=True)
        self.W, W, self.S = args.width, args.width, 1        # one residual stream
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        get = lambda name: weights[name]
        lin = lambda w, b=None: _Linear(w, b, self.exact, device)
        act = lambda t: t.to(device=device, dtype=self.act_torch).contiguous()
        self.embed, self.head = act(get("embed")), lin(get("head"))
        self.final_norm = f32(get("final.norm"))
        self.pairs = None
        if args.bigram:
            self.pairs = act(get("bigram"))
            if tuple(self.pairs.shape) != (args.bigram["buckets"] + 1, W):
                raise ValueError(f"bigram has shape {tuple(self.pairs.shape)}, expected {(args.bigram['buckets'] + 1, W)}")
        self.layers, self.cache_specs, self.rot_tables = [], [], {}
        for i, cfg in enumerate(args.layers):
            p, m = f"l{i}.", cfg["mixer"]
            mw = lambda n: get(p + "mix." + n)
            ly = {"type": "gla" if cfg["type"] in GLA else cfg["type"], "norm1": f32(get(p + "norm1")), "mlp": None}
            if ly["type"] == "gla":
                H, n, dv, rank = int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(mw("a1").shape[0])
                ly["dims"] = (H, n, dv, rank)
                ly["proj"] = lin(torch.cat([mw("q"), mw("k"), mw("v"), mw("g"), mw("a1")], 0))
                ly["a2t"], ly["a2b"], ly["inv_tau"] = f32(mw("a2").float().t()), f32(mw("a2.b")), 1.0 / float(m["tau"])
                norm = f32(mw("norm"))
                ly["head_norm"], ly["all_norm"], ly["out"] = norm, norm.repeat(H).contiguous(), lin(mw("o"))
                self.cache_specs.append({"slots": {"state": (H, n, dv)}})
            else:
                self._latent_weights(ly, m, mw, lin, f32)
                self.cache_specs.append({"pages": {"c": (ly["dims"][4] + ly["dims"][2],)}})
            mlp = cfg.get("mlp")
            if mlp:
                q = p + "mlp."
                ly["norm2"] = f32(get(p + "norm2"))
                if mlp["kind"] == "dense":
                    ly["mlp"] = {"kind": "dense", "up": lin(get(q + "up")), "down": lin(get(q + "down"))}
                else:
                    r = mlp["router"]
                    E, idn, grp = int(r["experts"]), int(r.get("identity") or 0), r.get("groups") or {"count": 1, "keep": 1}
                    stack = lambda ts: torch.stack(ts, 0).to(device=device,
                                                             dtype=torch.float32 if self.exact else torch.bfloat16).contiguous()
                    ly["mlp"] = {"kind": "moe", "E": E, "identity": idn, "top": int(r["top"]), "scale": float(r.get("scale", 1.0)),
                                 "groups": (int(grp["count"]), int(grp["keep"])), "limit": float(mlp["expert"].get("limit") or 0.0),
                                 "router": lin(get(q + "router")),
                                 "correction": f32(get(q + "correction")) if (q + "correction") in weights else None,
                                 "gu": stack([interleave_pairs(get(f"{q}e{e}.gate"), get(f"{q}e{e}.up")) for e in range(E)]),
                                 "down": stack([get(f"{q}e{e}.down") for e in range(E)]),
                                 "counters": torch.zeros(2 * E + 2, dtype=torch.int32, device=device)}
            self.layers.append(ly)
        if self.pairs is not None:
            self.cache_specs.append({"int_slots": {"last_token": ()}})     # belongs to the embedding, after the layers' entries

    # ------------------------------------------------------------------------------------------------
    def make_cache(self, max_tokens: int, max_seqs: int = 4) -> HybridCache:
        return HybridCache(self.cache_specs, max_tokens, max_seqs, self.device, self.act_torch, lib=self.L)

    def _empty(self, shape, dtype=None):
        return torch.empty(shape, dtype=dtype or torch.float32, device=self.device)

    def _linear(self, lin: _Linear, x, M, out_dtype=None, act=EPI_NONE):
        out_dtype = DTYPE_F32 if out_dtype is None else out_dtype
        out = self._empty((M, lin.N), torch.float32 if out_dtype == DTYPE_F32 else torch.bfloat16)
        _lib.check_hybrid(self.L.pieh_linear_act(_p(out), out_dtype, out.stride(0), _p(x), self.act, x.stride(0), _p(lin.w),
                                                 lin.w_dtype, _p(lin.bias), M, lin.N, lin.K, act, 0.0, 0.0, _stream()), "linear")
        return out

    def _sum_norm(self, x, h, y, mix, w, T):
        """x <- rms(alpha x + y | mixture) w, h <- x in the act dtype (exact mode: h is x)."""
        _lib.check_hybrid(self.L.pieh_sum_norm(_p(x), None if self.exact else _p(h), self.act, _p(y), C.byref(mix) if mix else None,
                                               _p(w), float(self.args.alpha), float(self.args.norm_eps), T, self.W, _stream()),
                          "sum_norm")

    def _segment_tiles(self, desc, H, dv):
        """64-row tiles per segment of the scan: enough segments that all heads' column blocks fill the GPU about four times."""
        return max(1, min(16, H * ((dv + 63) // 64) * desc.n_tiles // 592))

    def _gla(self, ly, st, h, desc, T):
        L, eps = self.L, float(self.args.norm_eps)
        H, n, dv, rank = ly["dims"]
        proj = self._linear(ly["proj"], h, T)                  # [q | k | v | g | a1]
        ld = proj.stride(0)
        g_off, low_off = 2 * H * n + H * dv, 2 * H * n + 2 * H * dv
        gl = HybGla(H, n, dv, 0, H * n, 2 * H * n, float(n) ** -0.5, _p(st["state"]))
        mixed = self._empty((T, H * dv), self.act_torch)
        if desc.T == desc.n_seq and dv <= 1024:                # every sequence brings one row
            _lib.check_hybrid(L.pieh_gla_step(_p(mixed), self.act, _p(proj), ld, low_off, rank, _p(ly["a2t"]), _p(ly["a2b"]),
                                              ly["inv_tau"], g_off, _p(ly["head_norm"]), eps, C.byref(gl), C.byref(desc),
                                              _stream()), "gla_step")
            return self._linear(ly["out"], mixed, T)
        decay = self._empty((T, H * n))
        _lib.check_hybrid(L.pieh_gla_decay(_p(decay), _p(proj), ld, low_off, rank, _p(ly["a2t"]), _p(ly["a2b"]), ly["inv_tau"],
                                           H * n, T, _stream()), "gla_decay")
        seg, scratch = self._segment_tiles(desc, H, dv), None
        if desc.n_tiles > desc.n_seq:                          # some portion spans several tiles
            scratch = self._empty((((desc.n_tiles - 1) // seg + desc.n_seq) * H * n * (dv + 1),))
        o = self._empty((T, H * dv))
        _lib.check_hybrid(L.pieh_gla_scan(_p(o), _p(proj), ld, _p(decay), C.byref(gl), C.byref(desc), _p(scratch), seg,
                                          _stream()), "gla_scan")
        _lib.check_hybrid(L.pieh_gated_group_norm(_p(mixed), self.act, _p(o), o.stride(0), C.c_void_p(proj.data_ptr() + 4 * g_off),
                                                  ld, _p(ly["all_norm"]), H, dv, eps, 2, 0, T, _stream()), "gated_group_norm")
        return self._linear(ly["out"], mixed, T)

    def _moe(self, ml, h, T):
        """-> (pieh_mix_sum describing the feed-forward's output, tensors to keep alive until it is consumed)."""
        L, E, top, W = self.L, ml["E"], ml["top"], self.W
        P = T * top
        z = self._linear(ml["router"], h, T)                       # [T, E + identity] fp32 logits
        i32 = lambda n: self._empty((n,), torch.int32)
        bufs = [i32(P), i32(P), i32(P), self._empty((P,)), i32(1 + 3 * (P // 64 + E)), i32(1 + 3 * (P // 128 + E))]
        plan = HybMoePlan(E, top, ml["groups"][0], ml["groups"][1], ml["scale"], *[b.data_ptr() for b in bufs],
                          ml["counters"].data_ptr(), 0, 1, _p(ml["correction"]), 1, ml["identity"])
        _lib.check_hybrid(L.pieh_moe_route(_p(z), z.stride(0), C.byref(plan), T, _stream()), "moe_route")
        wdt = DTYPE_F32 if self.exact else DTYPE_BF16
        ff2, ff = ml["gu"].shape[1], ml["gu"].shape[1] // 2
        hid = self._empty((P, ff), self.act_torch)
        _lib.check_hybrid(L.pieh_moe_linear(_p(hid), self.act, ff, _p(h), self.act, h.stride(0), _p(ml["gu"]), wdt, ff2 * W, P,
                                            ff2, W, 1, 1, GLU_SLOPE, ml["limit"], GLU_OFFSET, C.byref(plan), _stream()),
                          "moe_gate_up")
        ys = self._empty((P, W))
        _lib.check_hybrid(L.pieh_moe_linear(_p(ys), DTYPE_F32, W, _p(hid), self.act, ff, _p(ml["down"]), wdt, W * ff, P, W, ff,
                                            0, 0, 1.0, 0.0, 0.0, C.byref(plan), _stream()), "moe_down")
        mix = HybMixSum(ys.data_ptr(), bufs[2].data_ptr(), bufs[3].data_ptr(), top, None, None, 0)
        return mix, (z, bufs, hid, ys)

    def step(self, batch: BatchDetails, cache: HybridCache, rows: torch.Tensor | None = None, trace: list | None = None):
        """One forward step over ``batch``; pages and state slots come from ``cache`` through the batch's block table and
        ``state_slots``.  rows: int32 device tensor of the token rows whose logits are wanted (None: each sequence's last
        row).  Returns fp32 logits [len(rows), vocab].  trace: if a list, the residual after every layer is appended."""
        batch.validate()
        L, T, W, a = self.L, batch.total_tokens_in_step, self.W, self.args
        desc, keep = batch.hybrid_descriptor()
        x = self._empty((T, W))
        h = x if self.exact else self._empty((T, W), self.act_torch)
        bg = a.bigram or {"buckets": 0, "mul_prev": 0, "mul_cur": 0}
        last = cache.layers[-1]["last_token"] if self.pairs is not None else None
        _lib.check_hybrid(L.pieh_embed_pairs(_p(x), None if self.exact else _p(h), self.act, _p(self.embed), _p(self.pairs), self.act,
                                             _p(batch.token_ids), float(a.embed_scale), bg["mul_prev"], bg["mul_cur"],
                                             bg["buckets"], _p(last), W, a.vocab, C.byref(desc), _stream()), "embed_pairs")
        rot_cache = {}
        for ly, st in zip(self.layers, cache.layers):
            if ly["type"] == "gla":
                y = self._gla(ly, st, h, desc, T)
            else:
                y = self._latent(ly, st, h, batch, desc, T, rot_cache)
            self._sum_norm(x, h, y, None, ly["norm1"], T)
            ml = ly["mlp"]
            if ml and ml["kind"] == "dense":
                hid = self._linear(ml["up"], h, T, out_dtype=self.act, act=EPI_GELU)
                self._sum_norm(x, h, self._linear(ml["down"], hid, T), None, ly["norm2"], T)
            elif ml:
                mix, alive = self._moe(ml, h, T)
                self._sum_norm(x, h, None, mix, ly["norm2"], T)
                del alive
            if trace is not None:
                trace.append(x.clone())
        if rows is None:
            rows = batch.last_token_rows().to(torch.int32)
        R = int(rows.numel())
        xn = self._empty((R, W), self.act_torch)
        _lib.check_hybrid(L.pieh_stream_norm(_p(xn), self.act, _p(x), _p(rows), None, _p(self.final_norm), 0.0,
                                             float(a.norm_eps), R, 1, W, _stream()), "final_norm")
        logits = self._linear(self.head, xn, R)
        del keep
        return logits


def random_weights(args: DuduraxArgs, seed: int = 0, device="cpu") -> dict:
    """A synthetic checkpoint of this design (bf16 tensors): matrices U(-1, 1) scaled by 1 / sqrt(in), norm weights around
    1, decay biases spread so that some channels forget within a few tokens and others hardly at all, corrections of the
    size of the scores, router rows large enough that choices are rarely near ties."""
    g = torch.Generator(device=device).manual_seed(seed)
    bf = torch.bfloat16
    rnd = lambda *s: torch.rand(s, generator=g, device=device) * 2 - 1
    lin = lambda o, i, gain=1.0: (gain * rnd(o, i) / math.sqrt(i)).to(bf)
    W = args.width
    w = {"embed": (torch.randn((args.vocab, W), generator=g, device=device) / args.embed_scale).to(bf),
         "head": lin(args.vocab, W), "final.norm": (1 + 0.1 * rnd(W)).to(bf)}
    if args.bigram:
        w["bigram"] = (0.7 * torch.randn((args.bigram["buckets"] + 1, W), generator=g, device=device)).to(bf)
    for i, cfg in enumerate(args.layers):
        p, m = f"l{i}.", cfg["mixer"]
        q = p + "mix."
        w[p + "norm1"] = (1 + 0.2 * rnd(W)).to(bf)
        if cfg["type"] in GLA:
            H, n, dv = m["heads"], m["dim"], m["vdim"]
            low = max(4, min(16, W // 8))
            w[q + "q"], w[q + "k"], w[q + "v"] = lin(H * n, W, 2.0), lin(H * n, W, 2.0), lin(H * dv, W, 2.0)
            w[q + "g"], w[q + "o"] = lin(H * dv, W, 2.0), lin(W, H * dv, 2.0)
            w[q + "a1"], w[q + "a2"], w[q + "a2.b"] = lin(low, W, 2.0), lin(H * n, low, 2.0), (3 * rnd(H * n)).to(bf)
            w[q + "norm"] = (1 + 0.2 * rnd(dv)).to(bf)
        else:
            H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[q + "q"], w[q + "dkv"] = lin(H * (d + dr), W, 2.0), lin(r + dr, W, 2.0)
            w[q + "dkv.norm"] = (1 + 0.2 * rnd(r)).to(bf)
            w[q + "uk"], w[q + "uv"], w[q + "o"] = lin(H * d, r, 2.0), lin(H * dv, r, 2.0), lin(W, H * dv, 2.0)
        mlp = cfg.get("mlp")
        if not mlp:
            continue
        q = p + "mlp."
        w[p + "norm2"] = (1 + 0.2 * rnd(W)).to(bf)
        if mlp["kind"] == "dense":
            w[q + "up"], w[q + "down"] = lin(mlp["ff"], W, 2.0), lin(W, mlp["ff"], 2.0)
        else:
            E = mlp["router"]["experts"]
            n, ff = E + (mlp["router"].get("identity") or 0), mlp["expert"]["ff"]
            w[q + "router"], w[q + "correction"] = lin(n, W, 3.0), (rnd(n) / n).to(bf)
            for e in range(E):
                w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = lin(ff, W, 2.0), lin(ff, W, 2.0), lin(W, ff, 2.0)
    return w
