"""Latent attention with a rotated part, shared by the families that have it (``dudurax.DuduraxModel``,
``vokusun.VokusunModel``): per head a query [unrotated | rotated], per token ONE cached row [latent c (rms-normed) | rotated key
part].  The head's unrotated key is U c and its value V c, but neither is ever formed: (U^T q) . c = q . (U c), so queries go
into the latent space, the attention runs over the cached rows with one shared key "head" whose values are its leading
kv_rank features, and V is applied to what comes out.

    kv_rank <= dim:   U^T W_q is one matrix formed at load;  p = linear(h; [per head: U^T q | rotated part] [dkv] [gate])
    otherwise:        p = linear(h; [q | dkv | gate]), then one batched product with the heads' U^T
    latent_rot_prepare (latent norm, rotations, append to pages)
    bias_attn_run over the pages (optional: window with kept first keys, one sigmoid gate per head)
    kv_rank <= vdim:  W_o V is one matrix formed at load;  otherwise a batched product with the heads' V first
    y = linear(.; o)
"""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib
from ._lib import DTYPE_BF16, DTYPE_F32, EPI_NONE, HybBiasAttn, HybLatentRot
from .golitar import _p, _stream


def rotary_frequencies(rot: dict) -> list:
    """Angle per position of rotated pair i: base^(-2 i / dims), over the linear scaling factor if there is one."""
    dims = int(rot["dims"])
    factor = float((rot.get("scaling") or {}).get("factor") or 1.0)
    return [float(rot["base"]) ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


class LatentMixin:
    """For a model class with W, L, act, act_torch, exact, device, args.norm_eps, rot_tables, _empty and _linear."""

    rot_pairs = 0     # 1: features 2 i and 2 i + 1 rotate together; 0: i and i + dims / 2

    def _rot_key(self, rot):
        """Registers the frequencies of one rotation; -> its key in the tables (None: nothing rotates)."""
        if not rot or int(rot["dims"]) <= 0:
            return None
        key = (int(rot["dims"]), float(rot["base"]), float((rot.get("scaling") or {}).get("factor") or 1.0))
        if key not in self.rot_tables:
            self.rot_tables[key] = torch.tensor(rotary_frequencies(rot), dtype=torch.float64).to(self.device)
        return key

    def _rot(self, key, batch, T, cache):
        """(cos, sin) table of this step for one rotation, formed once and shared by the layers that use it."""
        if key not in cache:
            cs = self._empty((T, key[0] // 2, 2))
            _lib.check_hybrid(self.L.pieh_rot_table(_p(cs), _p(batch.positions), _p(self.rot_tables[key]), T, key[0] // 2,
                                                    _stream()), "rot_table")
            cache[key] = cs
        return cache[key]

    def _heads(self, out, out_dtype, out_head, x, w, M, nb, N, K):
        """nb per-head products in one launch: x [M, nb * K] (head-major columns), w [nb, N, K] -> head z at out + z * out_head."""
        wd = DTYPE_F32 if self.exact else DTYPE_BF16
        _lib.check_hybrid(self.L.pieh_linear_batched(_p(out), out_dtype, out.stride(0), out_head, _p(x), self.act, x.stride(0), K,
                                                     _p(w), wd, N * K, nb, M, N, K, EPI_NONE, None, 0, 0, _stream()),
                          "linear_batched")
        return out

    def _latent_weights(self, ly, m, mw, lin, f32, gate=None):
        """Fills ly with the fused projection of one layer.  mw(name): the layer's mixer tensor; gate: [H, W] or None."""
        H, d, dr, dv, r = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        if r > 512 or r + dr > 1024:
            raise ValueError(f"kv_rank {r} + rot_dim {dr} is beyond what the latent attention kernel holds (512 + 512)")
        W, wdt = self.W, torch.float32 if self.exact else torch.bfloat16
        ly["dims"] = (H, d, dr, dv, r)
        ukT = mw("uk").reshape(H, d, r).transpose(1, 2)                       # [H, r, d]
        qh = mw("q").reshape(H, d + dr, W)
        ly["ukT"] = ly["uv"] = None
        if r <= d:
            q_lat = torch.bmm(ukT.double(), qh[:, :d].double()).float()
            qw = torch.cat([q_lat, qh[:, d:].float()], 1)                     # [H, r + dr, W]
        else:
            qw, ly["ukT"] = qh.float(), ukT.to(device=self.device, dtype=wdt).contiguous()
        rows = [qw.reshape(-1, W), mw("dkv").float()]
        ly["q_rows"], ly["g_off"] = qw.shape[1], -1                           # projection rows per head
        if gate is not None:
            ly["g_off"] = H * qw.shape[1] + r + dr
            pad = -(ly["g_off"] + H) % 8                                      # rows of the product stay 16-byte aligned
            rows += [gate.float(), torch.zeros((pad, W), dtype=torch.float32, device=gate.device)]
        ly["proj"] = lin(torch.cat(rows, 0))
        uv = mw("uv").reshape(H, dv, r)
        if r <= dv:
            o = mw("o").reshape(W, H, dv).permute(1, 0, 2)                    # [H, W, dv]
            ly["out"] = lin(torch.bmm(o.double(), uv.double()).permute(1, 0, 2).reshape(W, H * r).float())
        else:
            ly["uv"], ly["out"] = uv.to(device=self.device, dtype=wdt).contiguous(), lin(mw("o"))
        ly["kv_norm"], ly["scale"] = f32(mw("dkv.norm")), float(m["scale"])
        mask = m.get("mask") or {}
        ly["window"], ly["keep"] = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
        ly["rot"] = self._rot_key(m.get("rot"))

    def _latent(self, ly, st, h, batch, desc, T, rot_cache):
        L, eps = self.L, float(self.args.norm_eps)
        H, d, dr, dv, r = ly["dims"]
        bref, D = C.byref(desc), r + dr
        proj = self._linear(ly["proj"], h, T)                  # per head [query | rotated part], [latent | shared key part], [gate]
        ld, kv_off = proj.stride(0), H * ly["q_rows"]
        rot_n = ly["rot"][0] if ly["rot"] else 0
        cs = self._rot(ly["rot"], batch, T, rot_cache) if ly["rot"] else None
        if ly["ukT"] is None:                                  # queries are in the latent space already: rotate them in place
            q, q_ld, plain, rot_at = proj, ld, None, r
        else:
            q, plain, rot_at = self._empty((T, H * D)), self._empty((T, H * d), self.act_torch), d
            q_ld = q.stride(0)
        lr = HybLatentRot(H, r, dr, rot_n, 0, ly["q_rows"], rot_at, kv_off, _p(ly["kv_norm"]), eps, _p(cs),
                          C.c_void_p(q.data_ptr() + 4 * r), q_ld, D, _p(plain), self.act, _p(st["c"]), self.act, self.rot_pairs)
        _lib.check_hybrid(L.pieh_latent_rot_prepare(_p(proj), ld, C.byref(lr), bref, _stream()), "latent_rot_prepare")
        if plain is not None:
            self._heads(q, DTYPE_F32, D, plain, ly["ukT"], T, H, r, d)
        at = HybBiasAttn(H=H, G=1, d=D, dv=r, g_off=ly["g_off"], gate_heads=1 if ly["g_off"] >= 0 else 0, eps=eps,
                         scale=ly["scale"], window=ly["window"], keep_first=ly["keep"], k_pages=_p(st["c"]), v_pages=_p(st["c"]),
                         kv_dtype=self.act, q_ld=q_ld, v_ld=D)
        mixed = self._empty((T, H * r), self.act_torch)
        _lib.check_hybrid(L.pieh_bias_attn_run(_p(mixed), self.act, _p(q), _p(proj), ld, C.byref(at), bref, _stream()), "attn_run")
        if ly["uv"] is not None:
            mixed = self._heads(self._empty((T, H * dv), self.act_torch), self.act, dv, mixed, ly["uv"], T, H, dv, r)
        return self._linear(ly["out"], mixed, T)
