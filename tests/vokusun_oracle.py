"""Plain, slow restatement of the Vokusun design, one function per mechanism, in float64 on the CPU.  It takes a whole
sequence at once (no cache, no batching, a loop over the tokens) and shares no code with the package: the tests compare the
engine's steps (portions, decoding, mixed batches) against it."""
from __future__ import annotations

import math

import torch

F = torch.float64


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * w + b"""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x, eps):
    """x [.., n] / sqrt(mean(x^2) + eps)"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, positions, dims, base, factor=1.0):
    """x [L, heads, d]: features 2i and 2i + 1 of the leading `dims` turn together by position * base^(-2i/dims) / factor;
    features from `dims` on pass through."""
    out = x.clone()
    for i in range(dims // 2):
        ang = positions.to(F) * (base ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def rotate(x, positions, rot):
    if not rot or not rot["dims"]:
        return x
    return rotate_pairs(x, positions, rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor", 1.0))


def visible(i, mask):
    """The key positions query i sees, as a list: all of 0 .. i, or the last `size` of them plus the first `keep_first`."""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < (mask.get("keep_first") or 0)]


def softmax_attention(q, k, v, scale, mask):
    """q [L, H, d], k [L, G, d], v [L, G, dv]; query head h reads key / value head h // (H / G).  -> [L, H, dv]"""
    L, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros((L, H, v.shape[2]), dtype=F)
    kk, vv = k.repeat_interleave(per, 1), v.repeat_interleave(per, 1)
    for i in range(L):
        js = torch.tensor(visible(i, mask))
        p = torch.softmax(torch.einsum("hd,jhd->hj", q[i], kk[js]) * scale, -1)
        out[i] = torch.einsum("hj,jhd->hd", p, vv[js])
    return out


def latent_attention(h, w, p, m, eps):
    """Keys and values of every head are expanded from the normed latent; one rotated key part serves all heads; each head's
    output is multiplied by the sigmoid of its own gate logit."""
    L = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(L)
    q = (h @ w[p + "q"].T).view(L, H, d + dr)
    low = h @ w[p + "dkv"].T
    c = unit_rms(low[:, :r], eps) * w[p + "dkv.norm"]
    q_rot, k_rot = rotate(q[:, :, d:], pos, m.get("rot")), rotate(low[:, r:].view(L, 1, dr), pos, m.get("rot"))
    k = torch.cat([(c @ w[p + "uk"].T).view(L, H, d), k_rot.expand(L, H, dr)], -1)
    v = (c @ w[p + "uv"].T).view(L, H, dv)
    o = softmax_attention(torch.cat([q[:, :, :d], q_rot], -1), k, v, m["scale"], m.get("mask"))
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(L, H * dv) @ w[p + "o"].T


def shared_kv_attention(h, w, p, m, eps):
    """The values are the keys as projected; queries and keys then get an RMS norm per head and the rotation."""
    L = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(L)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(L, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(L, G, d)
    v = k.clone()
    q = rotate(unit_rms(q, eps) * w[p + "q.norm"], pos, m.get("rot"))
    k = rotate(unit_rms(k, eps) * w[p + "k.norm"], pos, m.get("rot"))
    return softmax_attention(q, k, v, m["scale"], m.get("mask")).reshape(L, H * d) @ w[p + "o"].T


def gated_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer_runs(cfg):
    """[(layer index, pass this run opens or None)] in the order the layers run."""
    n = len(cfg["layers"])
    lp = cfg.get("loop") or None
    if not lp:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        runs += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, None) for i in range(lp["stop"], n)]


def open_pass(x, x0, t, w):
    """What happens to the residual right before pass t of the looped layers."""
    return torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, weights, tokens, trace=None):
    """tokens: list of ids of ONE sequence from its start -> logits [L, vocab] (float64).  trace: if a list, the residual
    after every layer run is appended."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: layer_norm(x, w[name], w[name + ".b"], eps)
    x0 = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = x0.clone()
    for i, t in layer_runs(cfg):
        ly, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = open_pass(x, x0, t, w)
        mixer = {"latent_attention": latent_attention, "attention": shared_kv_attention}[ly["type"]]
        x = x + norm(mixer(norm(x, p + "norm1"), w, p + "mix.", ly["mixer"], eps), p + "norm1b")
        if ly.get("mlp"):
            x = x + norm(gated_ff(norm(x, p + "norm2"), w, p + "mlp."), p + "norm2b")
        if trace is not None:
            trace.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T


def random_config(vocab=90, width=64, pattern="la", ffs="d", heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=24, rot_base=10000.0,
                  a_heads=6, a_kv=2, a_dim=16, a_rot=8, a_base=50000.0, factor=4.0, window=6, keep=3, scale=None, a_scale=None,
                  ff=48, loop=(0, 2, 2), eps=1e-5):
    """A small configuration: pattern 'l' = latent_attention, 'a' = attention; ffs per layer 'd' dense, '-' none (the last
    letter repeats); loop None = no loop; window 0 = no mask."""
    layers = []
    for i, c in enumerate(pattern):
        if c == "l":
            kind, mixer = "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                               "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
                                               "rot": {"base": rot_base, "dims": rot_dim}}
        else:
            kind, mixer = "attention", {"heads": a_heads, "kv_heads": a_kv, "dim": a_dim, "vdim": a_dim,
                                        "scale": a_scale if a_scale is not None else a_dim ** -0.5,
                                        "rot": {"base": a_base, "dims": a_rot, "scaling": {"factor": factor}}}
            if window:
                mixer["mask"] = {"size": window, "keep_first": keep}
        f = ffs[min(i, len(ffs) - 1)]
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if f == "d" else None})
    cfg = {"architecture": "Vokusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg
