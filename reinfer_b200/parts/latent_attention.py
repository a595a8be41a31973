"""Attention whose keys and values are rebuilt from one small latent vector per token:

    a   = rms(W_dq h) * w_q                       the queries' bottleneck (`q_rank`), an RMS norm with a plain weight inside
    q   = W_uq a                                  per head [dim unrotated | rot_dim rotated]
    c,r = split(W_dkv h)                          c (`kv_rank`) is normalised, rms(c) * w_kv; r (`rot_dim`) is rotated and is
                                                  ONE key part for all heads
    k_h = [W_uk,h c | rot(r)],   v_h = W_uv,h c
    score_h(i, j) = (q_h,plain . W_uk,h c_j + rot(q_h,rot) . rot(r_j)) * scale,   j <= i,   ordinary softmax
    `window`: position i sees only the j with i - j < window (pages that the window has passed go back to the pool)
    `gate`:   the heads' outputs are multiplied by sigmoid(W_g h) (tensor `g`) before W_o - element by element (True) or
              by one number a head ("heads")
    `own_kv=False`: the layer has no W_dkv; it reads the latents that an earlier layer of the same `kv_rank` cached (the
              layer's description names that layer, `cache_from`) with its own maps
    `rot_dim=0`: no rotated part; a token's cached row is c alone
    `sink`:   one learned number a head (tensor `sink`) joins the softmax's denominator as exp(sink_h), without key or value
    `out_scale`: a factor on the output (in 32-bit, on the heads' outputs behind which W_o stands)

Only [c | rot(r)] of a token is cached: kv_rank + rot_dim numbers, whatever the head count.  The per-head maps are
moved to the query's side (q_h,plain . W_uk,h c = (W_uk,h^T q_h,plain) . c, and sum_j p_j W_uv,h c_j = W_uv,h sum_j p_j c_j),
so the attention kernels see ONE key/value head of size kv_rank + rot_dim whose values are the first kv_rank columns of
its keys (`AttentionExtras(v_in_k=True)`), shared by all query heads: each cached row is read once for all heads.  The
rotation is a registered position encoding (kind `rope_pairs`: neighbouring or half-split pairs, optional frequency stretching).
`scale` is used as given.

Launches: fused projection [W_dq; W_dkv] -> `latent_prep` (both norms, the shared key's rotation, the cache store) ->
W_uq -> per-head W_uk^T on the plain part with the rotation of the rotated part behind it (`heads_linear`, one launch for
all heads) -> attention -> per-head W_uv (`heads_linear`, whose epilogue applies the gate) -> output projection.  The
bottleneck rows (and the gate's) reach their readers as 32-bit sums.

A prompt portion does the same work many times over in that form: every query head meets keys of kv_rank where the head itself
is smaller.  With heads of 128, no rotated part, no sink and no window, bfloat16 portions of REBUILD_FROM tokens or more (on average over
the step's portions) therefore take the keys and values rebuilt per head, once for the positions that the portions see
(`ops.kv_pages_from_latents`), and the tcgen05 kernel over them with the gate in its epilogue; single tokens of the same
step keep the latent form.
"""
from __future__ import annotations

import os
from typing import Optional

import torch

from .. import ops
from ..weights.params import ParamSpec
from .base import Mixer, PagedKVSpec, build_part, register_part
from .linear import matmul, matmul_into_residual, takes_row_scaled
from .spec import PartSpec


REBUILD = os.environ.get("REINFER_B200_LATENT_REBUILD", "1") != "0"    # 0: the latent form for every token (a development switch)
REBUILD_FROM = 64                            # tokens a portion from which rebuilding keys and values pays


class LatentAttention(Mixer):
    def __init__(self, hidden: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float,
                 eps: float, position: Optional[dict] = None, window: Optional[int] = None, gate=False, own_kv: bool = True, out_scale: float = 1.0,
                 sink: bool = False):
        self.hidden, self.H, self.dn, self.dr, self.dv = int(hidden), int(heads), int(dim), int(rot_dim), int(vdim)
        self.rq, self.rkv, self.scale, self.eps = int(q_rank), int(kv_rank), float(scale), float(eps)
        if min(self.H, self.dn, self.dv, self.rq, self.rkv) <= 0 or self.dr < 0:
            raise ValueError("latent attention: sizes must be positive")
        if gate not in (False, True, "heads", None):
            raise ValueError(f"latent attention: gate {gate!r} (False, True or 'heads')")
        self.window, self.gates = (int(window) if window else None), 0 if not gate else self.H if gate == "heads" else self.H * self.dv
        self.own_kv, self.out_scale, self.has_sink = bool(own_kv), float(out_scale), bool(sink)
        if self.window is not None and self.window <= 0:
            raise ValueError(f"latent attention: a window of {window} positions")
        pos = dict(position) if position else None
        self.position = build_part("position", PartSpec(pos.pop("kind"), pos)) if pos else None
        self.rot = int(getattr(self.position, "dims", 0)) if self.position is not None else 0
        self.half_split = bool(getattr(self.position, "half_split", False))
        if self.rot > self.dr:
            raise ValueError(f"latent attention: {self.rot} rotated dimensions in a part of {self.dr}")
        self.w_in = self.w_uq = self.w_absorb = self.w_uv = self.w_kv = self.w_o = self.qw = self.kvw = self.sink = None

    def param_specs(self):
        h, H = self.hidden, self.H
        out = {"dq": ParamSpec((self.rq, h)), "dq.norm": ParamSpec((self.rq,), init="norm"),
               "uq": ParamSpec((H * (self.dn + self.dr), self.rq)),
               "uk": ParamSpec((H * self.dn, self.rkv)), "uv": ParamSpec((H * self.dv, self.rkv)),
               "o": ParamSpec((h, H * self.dv))}
        if self.own_kv:
            out.update({"dkv": ParamSpec((self.rkv + self.dr, h)), "dkv.norm": ParamSpec((self.rkv,), init="norm")})
        if self.gates:
            out["g"] = ParamSpec((self.gates, h))
        if self.has_sink:
            out["sink"] = ParamSpec((H,), std=1.0)
        return out

    def cache_spec(self):
        # one head of [c | rot(r)]; no value rows of their own
        return PagedKVSpec(1, self.rkv + self.dr, self.window, 0)

    def bind(self, t):
        mats = [t["dq"]] + ([t["dkv"]] if self.own_kv else []) + ([t["g"]] if self.gates else [])
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.w_uq = t["uq"]
        # the keys' per-head map on the query's side: [H, kv_rank, dim] so that q_abs = w_absorb[h] q_plain
        self.w_absorb = t["uk"].view(self.H, self.dn, self.rkv).transpose(1, 2).contiguous()
        self.w_uv = t["uv"].view(self.H, self.dv, self.rkv).contiguous()
        self.w_kv = None
        if self.dn == self.dv == 128 and self.dr == 0 and self.window is None and not self.has_sink and self.rkv % 8 == 0 and t["uk"].is_cuda and \
                t["uk"].dtype == t["uv"].dtype == torch.bfloat16:
            self.w_kv = torch.cat([t["uk"], t["uv"]], dim=0).contiguous()       # for prompts whose keys and values are rebuilt per head
        self.w_o = t["o"]
        self.qw = t["dq.norm"].float().contiguous()
        self.kvw = t["dkv.norm"].float().contiguous() if self.own_kv else None
        self.sink = t["sink"].float().contiguous() if self.has_sink else None

    def prepare(self, device, dtype) -> None:
        if self.position is not None:
            self.position.prepare(device)

    @property
    def takes_row_scaled(self) -> bool:
        return takes_row_scaled(self.w_in)

    def forward(self, ctx, xn, residual, cache):
        T, H, dn, dr, dv, rq, rkv = xn.shape[0], self.H, self.dn, self.dr, self.dv, self.rq, self.rkv
        g = cache.group
        act, dev = ctx.dtype, ctx.device
        freq = self.position.freq if self.position is not None else None
        mag = self.position.magnitude if self.position is not None else 1.0
        if cache.write != self.own_kv:
            raise ValueError("latent attention: a layer without a latent of its own reads another layer's cache, and only such a layer")
        proj = matmul(ctx, xn, self.w_in, out_dtype=torch.float32)                 # [T, q_rank (| kv_rank | rot_dim) (| gate)], 32-bit sums
        a = torch.empty((T, rq), dtype=act, device=dev)
        nc, nr = (rkv, dr) if self.own_kv else (0, 0)
        ops.latent_prep(proj, rq, nc, nr, self.qw, self.kvw, self.eps, ctx.positions, freq, self.rot if self.own_kv else 0, mag,
                        g.kv_slot if self.own_kv else None, a, cache.kv, g.page_size, half_split=self.half_split)
        q = matmul(ctx, a, self.w_uq).view(T, H, dn + dr)
        heads = torch.empty((T, H, dv), dtype=act, device=dev)
        at = rq + nc + nr
        gate = proj[:, at:at + self.gates] if self.gates else None
        n_dec = ctx.q_start[ctx.n_decode] if self._rebuilds(ctx, act) else T     # tokens that take the latent form: all, or the single ones
        if n_dec:
            self._latent_form(ctx, q[:n_dec], cache, heads[:n_dec], gate[:n_dec] if gate is not None else None, decode_only=n_dec < T)
        if n_dec < T:
            pages, table = ops.kv_pages_from_latents(ctx, cache.kv, g, self.w_kv, H)
            ops.prompt_attention_128(ctx, q, pages, table, heads, H, H, self.scale, gate, self.out_scale)
        return matmul_into_residual(ctx, heads.view(T, H * dv), self.w_o, residual)

    def _rebuilds(self, ctx, act) -> bool:
        """Whether the step's prompt portions work on keys and values rebuilt per head (heads of 128, no rotated part, bfloat16)."""
        if self.w_kv is None or act != torch.bfloat16 or ctx.n_entries == ctx.n_decode or self.gates not in (0, self.H) or not REBUILD:
            return False
        tokens = ctx.n_tokens - ctx.q_start[ctx.n_decode]
        return tokens >= REBUILD_FROM * (ctx.n_entries - ctx.n_decode)

    def _latent_form(self, ctx, q, cache, heads, gate, decode_only: bool) -> None:
        T, H, dn, dr, rkv = q.shape[0], self.H, self.dn, self.dr, self.rkv
        act, dev = ctx.dtype, ctx.device
        freq = self.position.freq if self.position is not None else None
        mag = self.position.magnitude if self.position is not None else 1.0
        qf = torch.empty((T, H, rkv + dr), dtype=act, device=dev)                  # [W_uk^T q_plain | rot(q_rot)] per head
        ops.heads_linear(q, self.w_absorb, qf, tail=(ctx.positions, freq, self.rot, mag, self.half_split))     # the rotated part rides along
        lat = torch.empty((T, H, rkv), dtype=act, device=dev)
        ops.biased_attention(ctx, qf, cache.kv, cache.group, lat, H, 1, rkv + dr, rkv, self.window or 0, self.scale, None,
                             more=ops.AttentionExtras(v_in_k=True, sink=self.sink), decode_only=decode_only)
        ops.heads_linear(lat, self.w_uv, heads, gate=gate, out_scale=self.out_scale)


register_part("mixer", "latent_attention", LatentAttention)
