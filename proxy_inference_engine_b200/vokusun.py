"""Vokusun: a decoder-only model of sandwich blocks built on LAYER norm -- ``x <- x + ln(f(ln(x)))`` for every sublayer -- with
an optional LOOP: a run of layers is applied several times with the same weights (each pass with a cache of its own), and
every pass opens with a linear map of the current residual AND the embedding, plus a learned per-pass vector.  A layer's
mixer is one of
    latent_attention   causal softmax attention over one cached latent per token with a rotated key part shared by all heads,
                       every head's output multiplied by the sigmoid of a gate logit of its own
    attention          grouped-head softmax attention whose VALUES are its projected keys; queries and keys get a bias, an rms
                       norm per head and a (linearly scaled) rotation; a sliding window, and the first tokens stay visible
and its feed-forward is dense, gated by the tanh form of gelu, or absent.  Rotations pair neighbouring features.
Served through the ragged step of libpie_b200_hybrid.so like the other hybrid families: same ``BatchDetails``, same
``cache.HybridCache`` (one entry per layer RUN, so a looped layer holds one per pass), same ``engine.HybridEngine``.

config.json: ``architecture`` "Vokusun"; ``vocab``, ``width``, ``norm.eps``, ``loop`` {start, stop, times} | absent, and
``layers``, a list of ``{"type": "latent_attention" | "attention", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}``:
    latent_attention:  heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}
    attention:         heads, kv_heads, dim, vdim (= dim), scale, mask {size, keep_first} (absent: all earlier tokens),
                       rot {base, dims, scaling.factor}
Tensors: ``embed``, ``head``, ``final.norm[.b]``, ``loop.in`` [width, 2 width], ``loop.step`` [times, width], per layer i
``l<i>.norm1|norm1b|norm2|norm2b[.b]``, ``l<i>.mix.q|dkv|dkv.norm|uk|uv|g|o`` or ``l<i>.mix.q|q.b|k|k.b|q.norm|k.norm|o``,
``l<i>.mlp.gate|up|down``.

One step over a ``ragged.BatchDetails`` (x: fp32 residual [T, W]; h: what the next product reads, act dtype; loop.in = [A | B]):

    x, h   = embed(tokens)
    e      = linear(h; B), once per step: what the embedding adds to every pass (start 0: from one product with [A; B])
    per layer run:
      opening a pass:   x, h = layernorm_add(x <- linear(h; A) + e + pass vector; norm1)
      latent_attention: latent.LatentMixin (queries taken into the latent space; gate inside the attention kernel)
      attention:        p = linear(h; [q | k] + biases)
                        bias_attn_prepare (per-head norms, rotation; k' and the plain k appended to the pages)
                        bias_attn_run (window + kept first keys);  y = linear(.; o)
      x, h   = layernorm_add(x += ln(y; norm1b); norm2)
      y      = linear(linear_glu_act(h; gate, up, gelu); down)
      x, h   = layernorm_add(x += ln(y; norm2b); the next run's norm1 | x itself if a pass opens | the final norm of the
               wanted rows)
    logits = linear(h; head)                                                                      fp32

dtype "bfloat16": matrix-product inputs and the pages are bf16; accumulation, residual, norms, rotation angles, attention
scores and weights and gates are fp32.  dtype "float32": weights are widened once and every product is a plain fp32
multiply-add.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass, field

import torch

from . import _lib
from ._lib import DTYPE_BF16, DTYPE_F32, EPI_GELU, EPI_NONE, HybBiasAttn
from .babodra import interleave_pairs
from .cache import HybridCache
from .golitar import _Linear, _p, _stream
from .latent import LatentMixin
from .ragged import BatchDetails

MIXER_KEYS = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"),
              "attention": ("heads", "kv_heads", "dim", "scale")}


@dataclass
class VokusunArgs:
    vocab: int
    width: int
    layers: list
    norm_eps: float = 1e-5
    loop: dict | None = None
    architecture: str = "Vokusun"
    raw: dict = field(default_factory=dict)

    @classmethod
    def from_dict(cls, cfg: dict) -> "VokusunArgs":
        bad = lambda what: ValueError(f"Vokusun config: {what}")
        for key in ("vocab", "width", "layers"):
            if key not in cfg:
                raise bad(f"'{key}' is missing")
        for i, ly in enumerate(cfg["layers"]):
            kind, m = ly.get("type"), ly.get("mixer") or {}
            if kind not in MIXER_KEYS:
                raise bad(f"layer {i} has unknown type {kind!r}")
            for key in MIXER_KEYS[kind]:
                if key not in m:
                    raise bad(f"layer {i} mixer lacks '{key}'")
            if kind == "attention":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise bad(f"layer {i}: heads is not a multiple of kv_heads")
                if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                    raise bad(f"layer {i}: the values are the keys, so vdim must equal dim")
            rot, room = m.get("rot"), int(m["rot_dim"] if kind == "latent_attention" else m["dim"])
            if rot and (int(rot["dims"]) % 2 or int(rot["dims"]) > room):
                raise bad(f"layer {i}: rot.dims must be even and at most {room}")
            mask = m.get("mask")
            if mask and (int(mask["size"]) < 1 or int(mask.get("keep_first") or 0) < 0):
                raise bad(f"layer {i}: mask.size must be positive and mask.keep_first not negative")
            mlp = ly.get("mlp")
            if mlp and mlp.get("kind") != "dense":
                raise bad(f"layer {i} has unknown feed-forward kind {mlp.get('kind')!r}")
        loop = cfg.get("loop") or None
        if loop:
            a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
            if not (0 <= a < b <= len(cfg["layers"])) or times < 1:
                raise bad("loop needs 0 <= start < stop <= number of layers and times >= 1")
            loop = {"start": a, "stop": b, "times": times}
        return cls(vocab=int(cfg["vocab"]), width=int(cfg["width"]), layers=list(cfg["layers"]),
                   norm_eps=float((cfg.get("norm") or {}).get("eps", 1e-5)), loop=loop,
                   architecture=cfg.get("architecture", "Vokusun"), raw=cfg)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": self.layers}
        if self.loop:
            out["loop"] = dict(self.loop)
        return out

    def runs(self) -> list:
        """The order the layers run in: [(layer index, number of the pass this run OPENS or None)]."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        out = [(i, None) for i in range(a)]
        for t in range(times):
            out += [(i, t if i == a else None) for i in range(a, b)]
        return out + [(i, None) for i in range(b, n)]


class VokusunModel(LatentMixin):
    rot_pairs = 1

    def __init__(self, args: VokusunArgs, weights: dict, device="cuda", dtype: str = "bfloat16"):
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
        norm = lambda name: (f32(get(name)), f32(get(name + ".b")))

        def shaped(name, shape):
            if tuple(get(name).shape) != shape:
                raise ValueError(f"{name} has shape {tuple(get(name).shape)}, expected {shape}")
            return get(name)
        self.embed = shaped("embed", (args.vocab, W)).to(device=device, dtype=self.act_torch).contiguous()
        self.head, self.final_norm = lin(shaped("head", (args.vocab, W))), norm("final.norm")
        self.loop_step = None
        if args.loop:
            self.loop_step = f32(shaped("loop.step", (args.loop["times"], W)))
            both = shaped("loop.in", (W, 2 * W))
            self.loop_in = lin(torch.cat([both[:, :W], both[:, W:]], 0))      # [A; B]: rows 0 .. W - 1 read x, the rest x0
            self.loop_x, self.loop_x0 = lin(self.loop_in.w[:W]), lin(self.loop_in.w[W:])      # views of the same storage
        self.layer_weights, self.rot_tables = [], {}
        for i, cfg in enumerate(args.layers):
            p, m, kind = f"l{i}.", cfg["mixer"], cfg["type"]
            mw = lambda n: get(p + "mix." + n)
            ly = {"type": kind, "norm1": norm(p + "norm1"), "norm1b": norm(p + "norm1b"), "mlp": None}
            if kind == "latent_attention":
                self._latent_weights(ly, m, mw, lin, f32, gate=mw("g"))
                ly["cache"] = {"pages": {"c": (ly["dims"][4] + ly["dims"][2],)}}
            else:
                H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
                ly["dims"], ly["scale"] = (H, G, d), float(m["scale"])
                ly["proj"] = lin(torch.cat([mw("q"), mw("k")], 0), torch.cat([mw("q.b"), mw("k.b")], 0))
                ly["q_norm"], ly["k_norm"], ly["out"] = f32(mw("q.norm")), f32(mw("k.norm")), lin(mw("o"))
                mask = m.get("mask") or {}
                ly["window"], ly["keep"] = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
                ly["rot"] = self._rot_key(m.get("rot"))
                ly["cache"] = {"pages": {"k": (G, d), "v": (G, d)}}
            if cfg.get("mlp"):
                q = p + "mlp."
                ly["norm2"], ly["norm2b"] = norm(p + "norm2"), norm(p + "norm2b")
                ly["mlp"] = {"gu": lin(interleave_pairs(get(q + "gate"), get(q + "up"))), "down": lin(get(q + "down"))}
            self.layer_weights.append(ly)
        # one entry per layer RUN: a looped layer appears once per pass, with the same weights and its own cache entry
        self.runs = args.runs()
        self.layers = [self.layer_weights[i] for i, _ in self.runs]
        self.cache_specs = [ly["cache"] for ly in self.layers]

    # ------------------------------------------------------------------------------------------------
    def make_cache(self, max_tokens: int, max_seqs: int = 4) -> HybridCache:
        return HybridCache(self.cache_specs, max_tokens, max_seqs, self.device, self.act_torch, lib=self.L)

    def _empty(self, shape, dtype=None):
        return torch.empty(shape, dtype=dtype or torch.float32, device=self.device)

    def _linear(self, lin: _Linear, x, M):
        out = self._empty((M, lin.N))
        _lib.check_hybrid(self.L.pieh_linear_act(_p(out), DTYPE_F32, out.stride(0), _p(x), self.act, x.stride(0), _p(lin.w),
                                                 lin.w_dtype, _p(lin.bias), M, lin.N, lin.K, EPI_NONE, 0.0, 0.0, _stream()),
                          "linear")
        return out

    def _norm_add(self, x, y, post, h, nxt, n, e=None, vec=None, rows=None):
        """x <- x + ln(y; post) (post None: x <- y), + e + vec; h <- ln(x; nxt) (nxt None: x).  rows: only h of these rows."""
        (pw, pb), (nw, nb) = post or (None, None), nxt or (None, None)
        _lib.check_hybrid(self.L.pieh_layernorm_add(_p(x), _p(y), y.stride(0) if y is not None else 0, _p(pw), _p(pb), _p(e),
                                                    e.stride(0) if e is not None else 0, _p(vec), _p(h), self.act, _p(nw),
                                                    _p(nb), _p(rows), float(self.args.norm_eps), n, self.W, _stream()),
                          "layernorm_add")

    def _attention(self, ly, st, h, batch, bref, T, rot_cache):
        L, eps = self.L, float(self.args.norm_eps)
        H, G, d = ly["dims"]
        proj = self._linear(ly["proj"], h, T)                  # [q | k]
        ld = proj.stride(0)
        cs = self._rot(ly["rot"], batch, T, rot_cache) if ly["rot"] else None
        at = HybBiasAttn(H=H, G=G, d=d, dv=d, k_off=H * d, v_off=H * d, g_off=-1, q_norm=_p(ly["q_norm"]), k_norm=_p(ly["k_norm"]),
                         eps=eps, scale=ly["scale"], window=ly["window"], keep_first=ly["keep"], k_pages=_p(st["k"]),
                         v_pages=_p(st["v"]), kv_dtype=self.act, rot_dims=ly["rot"][0] if ly["rot"] else 0, rot_cs=_p(cs),
                         head_norm=1, rot_pairs=self.rot_pairs)
        q = self._empty((T, H * d))
        _lib.check_hybrid(L.pieh_bias_attn_prepare(_p(q), _p(proj), ld, C.byref(at), bref, _stream()), "attn_prepare")
        o = self._empty((T, H * d), self.act_torch)
        _lib.check_hybrid(L.pieh_bias_attn_run(_p(o), self.act, _p(q), None, 0, C.byref(at), bref, _stream()), "attn_run")
        return self._linear(ly["out"], o, T)

    def _feed_forward(self, ml, h, T):
        g = ml["gu"]
        hid = self._empty((T, g.N // 2), self.act_torch)
        _lib.check_hybrid(self.L.pieh_linear_glu_act(_p(hid), self.act, hid.stride(0), _p(h), self.act, h.stride(0), _p(g.w),
                                                     g.w_dtype, T, g.N, g.K, EPI_GELU, 0.0, 0.0, _stream()), "linear_glu")
        return self._linear(ml["down"], hid, T)

    def step(self, batch: BatchDetails, cache: HybridCache, rows: torch.Tensor | None = None, trace: list | None = None):
        """One forward step over ``batch``; pages come from ``cache`` through the batch's block table.  rows: int32 device
        tensor of the token rows whose logits are wanted (None: each sequence's last row).  Returns fp32 logits
        [len(rows), vocab].  trace: if a list, the residual after every layer run is appended."""
        batch.validate()
        L, T, W, a = self.L, batch.total_tokens_in_step, self.W, self.args
        desc, keep = batch.hybrid_descriptor()
        if rows is None:
            rows = batch.last_token_rows().to(torch.int32)
        R, nruns = int(rows.numel()), len(self.layers)
        x, h = self._empty((T, W)), self._empty((T, W), self.act_torch)
        out = self._empty((R, W), self.act_torch)
        _lib.check_hybrid(L.pieh_embed_positions(_p(x), _p(h), self.act, _p(self.embed), None, self.act, _p(batch.token_ids), None,
                                                 T, W, a.vocab, 0, _stream()), "embed")
        e = y = None                                           # e: the embedding's part of every pass opening
        opens = [t for _, t in self.runs]
        if a.loop:
            if opens[0] is not None:                           # the first run opens pass 0: x is x0, one product gives both parts
                both = self._linear(self.loop_in, h, T)
                y, e = both[:, :W], both[:, W:]
            else:
                e = self._linear(self.loop_x0, h, T)
        vec = self.loop_step[opens[0]] if y is not None else None
        self._norm_add(x, y, None, h, self.layers[0]["norm1"], T, e if y is not None else None, vec)
        rot_cache = {}
        for r, (ly, st) in enumerate(zip(self.layers, cache.layers)):
            if ly["type"] == "latent_attention":
                y = self._latent(ly, st, h, batch, desc, T, rot_cache)
            else:
                y = self._attention(ly, st, h, batch, C.byref(desc), T, rot_cache)
            post = ly["norm1b"]
            if ly["mlp"]:
                self._norm_add(x, y, post, h, ly["norm2"], T)
                y, post = self._feed_forward(ly["mlp"], h, T), ly["norm2b"]
            if trace is not None:                              # the residual by itself first
                self._norm_add(x, y, post, None, None, T)
                trace.append(x.clone())
                y = post = None
            if r + 1 == nruns:
                self._norm_add(x, y, post, out, self.final_norm, R, rows=rows)
            elif opens[r + 1] is None:
                self._norm_add(x, y, post, h, self.layers[r + 1]["norm1"], T)
            else:
                self._norm_add(x, y, post, h, None, T)
                y = self._linear(self.loop_x, h, T)
                self._norm_add(x, y, None, h, self.layers[r + 1]["norm1"], T, e, self.loop_step[opens[r + 1]])
        logits = self._linear(self.head, out, R)
        del keep
        return logits


def random_weights(args: VokusunArgs, seed: int = 0, device="cpu") -> dict:
    """A synthetic checkpoint of this design (bf16 tensors): matrices U(-1, 1) scaled by 1 / sqrt(in), norm weights around 1
    and small biases."""
    g = torch.Generator(device=device).manual_seed(seed)
    bf = torch.bfloat16
    rnd = lambda *s: torch.rand(s, generator=g, device=device) * 2 - 1
    lin = lambda o, i, gain=1.0: (gain * rnd(o, i) / math.sqrt(i)).to(bf)
    W = args.width
    w = {"embed": torch.randn((args.vocab, W), generator=g, device=device).to(bf), "head": lin(args.vocab, W)}

    def norm(name):
        w[name], w[name + ".b"] = (1 + 0.2 * rnd(W)).to(bf), (0.2 * rnd(W)).to(bf)
    norm("final.norm")
    if args.loop:
        w["loop.in"], w["loop.step"] = lin(W, 2 * W, 2.0), (0.5 * rnd(args.loop["times"], W)).to(bf)
    for i, cfg in enumerate(args.layers):
        p, m = f"l{i}.", cfg["mixer"]
        q = p + "mix."
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if cfg.get("mlp") else ()):
            norm(p + nm)
        if cfg["type"] == "latent_attention":
            H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[q + "q"], w[q + "dkv"] = lin(H * (d + dr), W, 2.0), lin(r + dr, W, 2.0)
            w[q + "dkv.norm"], w[q + "g"] = (1 + 0.2 * rnd(r)).to(bf), lin(H, W, 2.0)
            w[q + "uk"], w[q + "uv"], w[q + "o"] = lin(H * d, r, 2.0), lin(H * dv, r, 2.0), lin(W, H * dv, 2.0)
        else:
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            w[q + "q"], w[q + "k"], w[q + "o"] = lin(H * d, W, 2.0), lin(G * d, W, 2.0), lin(W, H * d, 2.0)
            w[q + "q.b"], w[q + "k.b"] = (0.5 * rnd(H * d)).to(bf), (0.5 * rnd(G * d)).to(bf)
            w[q + "q.norm"], w[q + "k.norm"] = (1 + 0.3 * rnd(d)).to(bf), (1 + 0.3 * rnd(d)).to(bf)
        mlp = cfg.get("mlp")
        if mlp:
            q = p + "mlp."
            w[q + "gate"], w[q + "up"], w[q + "down"] = lin(mlp["ff"], W, 2.0), lin(mlp["ff"], W, 2.0), lin(W, mlp["ff"], 2.0)
    return w
