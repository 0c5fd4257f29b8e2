"""Plain, slow restatement of the Dudurax design, one function per mechanism, in float64 on the CPU.  It takes a whole
sequence at once (no cache, no batching, token-by-token loops) and shares no code with the package: the tests compare the
engine's steps (portions, decoding, mixed batches) against it."""
from __future__ import annotations

import math

import torch

F = torch.float64


def unit_rms(x, eps):
    """x [.., n] / sqrt(mean(x^2) + eps)"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def pair_row(prev, cur, bigram):
    """Row of the pair table: the hash of (previous, current), or the extra last row when there is no previous token."""
    n = bigram["buckets"]
    return n if prev is None else (prev * bigram["mul_prev"] + cur * bigram["mul_cur"]) % n


def embedding(tokens, w, emb):
    """Token row times the scale, plus the (unscaled) row of the pair table."""
    rows = []
    for t, cur in enumerate(tokens):
        x = w["embed"][cur] * emb.get("scale", 1.0)
        if emb.get("bigram"):
            x = x + w["bigram"][pair_row(tokens[t - 1] if t else None, cur, emb["bigram"])]
        rows.append(x)
    return torch.stack(rows)


def rotate_half(x, positions, dims, base):
    """x [L, heads, d]: feature i < dims/2 pairs with i + dims/2 and turns by position * base^(-2i/dims); features from
    `dims` on pass through."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        ang = positions.to(F) * (base ** (-2.0 * i / dims))
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def window_softmax_attention(q, k, v, scale, window):
    """q, k [L, H, d], v [L, H, dv]: query i weighs the keys j with 0 <= i - j < window by the softmax of their scores."""
    L, H, _ = q.shape
    out = torch.zeros((L, H, v.shape[2]), dtype=F)
    for i in range(L):
        lo = max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1]) * scale
        out[i] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[lo:i + 1])
    return out


def latent_attention(h, w, p, m, eps):
    """Keys and values of every head are expanded from the normed latent; one rotated key part serves all heads."""
    L = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(L)
    q = (h @ w[p + "q"].T).view(L, H, d + dr)
    low = h @ w[p + "dkv"].T
    c = unit_rms(low[:, :r], eps) * w[p + "dkv.norm"]
    k_rot = low[:, r:].view(L, 1, dr)
    q_rot = q[:, :, d:]
    if dr:
        q_rot = rotate_half(q_rot, pos, m["rot"]["dims"], m["rot"]["base"])
        k_rot = rotate_half(k_rot, pos, m["rot"]["dims"], m["rot"]["base"])
    k = (c @ w[p + "uk"].T).view(L, H, d)
    v = (c @ w[p + "uv"].T).view(L, H, dv)
    qq = torch.cat([q[:, :, :d], q_rot], -1)
    kk = torch.cat([k, k_rot.expand(L, H, dr)], -1)
    window = (m.get("mask") or {}).get("size") or L
    o = window_softmax_attention(qq, kk, v, m["scale"], window)
    return o.reshape(L, H * dv) @ w[p + "o"].T


def channel_decays(h, w, p, tau):
    """sigmoid(z)^(1 / tau) from the low-rank logits z."""
    return torch.sigmoid((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]) ** (1.0 / tau)


def gla_scan(q, k, v, decay):
    """q, k, decay [L, H, n], v [L, H, dv]:  S <- diag(decay) S + k v^T  (S [n, dv] per head, zero at the start), o = S^T q."""
    L, H, n = q.shape
    S = torch.zeros((H, n, v.shape[2]), dtype=F)
    o = torch.zeros((L, H, v.shape[2]), dtype=F)
    for t in range(L):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hnd,hn->hd", S, q[t])
    return o


def gla_mixer(h, w, p, m, eps):
    L = h.shape[0]
    H, n, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(L, H, n) * n ** -0.5
    k = (h @ w[p + "k"].T).view(L, H, n)
    v = (h @ w[p + "v"].T).view(L, H, dv)
    o = gla_scan(q, k, v, channel_decays(h, w, p, m["tau"]).view(L, H, n))
    o = (unit_rms(o, eps) * w[p + "norm"]).reshape(L, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def clamped_expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z, correction, r):
    """Logits z [E + identity] of one token -> (chosen output numbers, their weights, gap to the nearest other choice)."""
    n, top = z.shape[0], r["top"]
    s = torch.softmax(z, -1)
    c = s + correction
    groups = r.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]
    gs = torch.stack([c[g * per:(g + 1) * per].max() for g in range(groups["count"])])
    gorder = torch.argsort(gs, descending=True, stable=True)
    kept = gorder[:groups["keep"]].tolist()
    gap = math.inf
    if groups["keep"] < groups["count"]:
        gap = float(gs[gorder[groups["keep"] - 1]] - gs[gorder[groups["keep"]]])
    masked = torch.full_like(c, -math.inf)
    for g in kept:
        masked[g * per:(g + 1) * per] = c[g * per:(g + 1) * per]
    order = torch.argsort(masked, descending=True, stable=True)
    if top < n and masked[order[top]] > -math.inf:
        gap = min(gap, float(masked[order[top - 1]] - masked[order[top]]))
    pick = order[:top].tolist()
    return pick, [float(s[e]) * r["scale"] for e in pick], gap


def moe(h, w, p, mlp, margins=None):
    """margins: if a list, the smallest gap between a taken and a rejected choice (or group) of every token is appended."""
    r = mlp["router"]
    E, limit = r["experts"], mlp["expert"]["limit"]
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        pick, wts, gap = route(z[t], w[p + "correction"], r)
        if margins is not None:
            margins.append(gap)
        for e, c in zip(pick, wts):
            out[t] += c * (h[t] if e >= E else clamped_expert(h[t], w, f"{p}e{e}.", limit))
    return out


def dense_ff(h, w, p):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def forward(cfg, weights, tokens, trace=None, margins=None):
    """tokens: list of ids of ONE sequence from its start -> logits [L, vocab] (float64).  trace: if a list, the residual
    after every layer is appended."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = embedding(tokens, w, cfg["embedding"])
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = latent_attention if ly["type"] == "latent_attention" else gla_mixer
        x = unit_rms(alpha * x + mixer(x, w, p + "mix.", ly["mixer"], eps), eps) * w[p + "norm1"]
        mlp = ly.get("mlp")
        if mlp:
            y = dense_ff(x, w, p + "mlp.") if mlp["kind"] == "dense" else moe(x, w, p + "mlp.", mlp, margins)
            x = unit_rms(alpha * x + y, eps) * w[p + "norm2"]
        if trace is not None:
            trace.append(x.clone())
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T


def random_config(vocab=90, width=64, pattern="gal", ffs="dmm", heads=2, dim=16, vdim=24, tau=8.0, heads2=3, dim2=8, vdim2=20,
                  tau2=2.0, a_heads=4, a_dim=16, a_vdim=12, rot_dim=8, kv_rank=24, rot_base=10000.0, window=6, scale=None, ff=48,
                  experts=6, identity=2, top=3, groups=(4, 3), expert_ff=24, limit=1.0, router_scale=1.5, alpha=1.7, eps=1e-5,
                  embed_scale=2.0, buckets=61, mul_prev=5, mul_cur=3):
    """A small configuration: pattern 'g' = gla, 'h' = gla_2, 'a' or 'l' = latent_attention; ffs per layer 'd' dense, 'm'
    experts, '-' none (the last letter repeats); buckets 0 = no pair table; window 0 = no mask; groups None = no groups."""
    layers = []
    for i, c in enumerate(pattern):
        if c == "g":
            kind, mixer = "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}
        elif c == "h":
            kind, mixer = "gla_2", {"heads": heads2, "dim": dim2, "vdim": vdim2, "tau": tau2}
        else:
            kind = "latent_attention"
            mixer = {"heads": a_heads, "dim": a_dim, "vdim": a_vdim, "rot_dim": rot_dim, "kv_rank": kv_rank,
                     "scale": scale if scale is not None else (a_dim + rot_dim) ** -0.5,
                     "rot": {"base": rot_base, "dims": rot_dim}}
            if window:
                mixer["mask"] = {"size": window}
        f = ffs[min(i, len(ffs) - 1)]
        mlp = None
        if f == "d":
            mlp = {"kind": "dense", "ff": ff}
        elif f == "m":
            mlp = {"kind": "moe", "expert": {"ff": expert_ff, "limit": limit},
                   "router": {"experts": experts, "identity": identity, "top": top, "scale": router_scale}}
            if groups:
                mlp["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    emb = {"scale": embed_scale}
    if buckets:
        emb["bigram"] = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    return {"architecture": "Dudurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": emb, "layers": layers}
