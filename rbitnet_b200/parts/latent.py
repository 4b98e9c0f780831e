"""``LatentAttention``: causal softmax attention whose keys and values are made from one small vector per position,
the only thing the cache keeps.

From the input rows h, without biases and (unless ``rot_dim`` is given) without a position encoding:

    c_q = rmsnorm(W_dq h) * w_dq          [q_rank]      the queries' latent
    q   = W_uq c_q                        [n_heads, head_dim]
    c   = rmsnorm(W_dkv h) * w_dkv        [kv_rank]     the latent that is cached
    k_j = W_uk c_j,  v_j = W_uv c_j       per head: [head_dim], [value_dim]
    score_ij = (q_i . k_j) * scale, j <= i;  softmax over j;  o_i = sum_j p_ij v_j;  result = W_o o

Because k_j and v_j are linear in c_j, the sums over positions can be taken over the latents themselves:
q_i . k_j = (W_uk^T q_i) . c_j and sum_j p_ij v_j = W_uv (sum_j p_ij c_j), head by head.  So a step turns every
query head into the latent's space (a small product per head), runs the library's attention with ONE key/value head
whose keys and values are both the cached latents, and turns every head's result back (another small product per
head).  Nothing but c is stored per position, whole prompts and single tokens take the same path, and every attention
kernel of the library serves it as it serves grouped attention with one key head.  Norms, scores and softmax are
float32 as everywhere.

Options, each off by default:
  q_rank = 0    the queries come straight from the input rows: q = W_q h ("q"), no latent and no norm of their own
  rot_dim > 0   every query head has ``rot_dim`` more values after its ``head_dim`` ones, and W_dkv ``rot_dim`` more
                rows after the latent's (not normed): one key part per position that all heads share.  Both are turned
                by position (``position``: a rotary encoding over ``rot_dim`` values) and the score is
                (q_c . W_uk c + rot(q_r) . rot(k_r)) * scale.  The cache row is [c | rot(k_r)]; a query head enters
                the attention as [W_uk^T q_c | rot(q_r)], and the result's columns beyond the latent meet no row of W_uv
  sinks         the softmax's denominator also holds exp(s_h), a stored number per head ("sink")
  value_gate    the joined heads are multiplied value by value with sigmoid(W_g h) ("g", a row per value), read from the
                same input rows; its float32 sums come out of the same product as the latents, and the sigmoid is applied
                where the heads' results leave their matrices W_uv

  window        a position sees itself and the window - 1 positions before it; the pages behind it are given back
  head_gate     head h's result is multiplied by sigmoid(W_g h)_h, one number per head ("g", a row per head), made and applied
                as the gate per value is

All options go together (one kind of gate at a time).  With queries through a latent AND a turned part, the turned part of the queries exists only
after W_uq: the step that takes the query heads into the latent's space turns it (``ops.latent_queries``).
"""
from __future__ import annotations

import dataclasses

import torch

from .base import Mixer, CacheNeed
from .registry import register_part, build_part
from .spec import PartSpec


class LatentAttention(Mixer):
    def __init__(self, width: int, n_heads: int, head_dim: int, value_dim: int, q_rank: int, kv_rank: int,
                 scale: float, norm_eps: float, rot_dim: int = 0, position: dict = None, sinks: bool = False,
                 value_gate: bool = False, window: int = None, head_gate: bool = False):
        self.width, self.n_heads, self.head_dim, self.value_dim = int(width), int(n_heads), int(head_dim), int(value_dim)
        self.q_rank, self.kv_rank = int(q_rank or 0), int(kv_rank)
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.rot_dim, self.sinks, self.value_gate = int(rot_dim or 0), bool(sinks), bool(value_gate)
        self.window, self.head_gate = (int(window) if window else None), bool(head_gate)
        if self.head_gate and self.value_gate:
            raise ValueError("latent attention: a gate per head or a gate per value, not both")
        if min(self.n_heads, self.head_dim, self.value_dim, self.kv_rank) < 1 or self.q_rank < 0 or self.rot_dim < 0:
            raise ValueError("latent attention: heads, sizes and ranks are at least 1")
        self.position = None
        if self.rot_dim:
            if not position or position.get("kind") != "rotary":
                raise ValueError("latent attention: a turned key part needs a rotary position encoding")
            self.position = build_part("position", PartSpec(position["kind"], dict(position.get("params", {}))))
            if self.position.head_dim != self.rot_dim or self.position.rot_dim != self.rot_dim:
                raise ValueError("latent attention: the position encoding turns the whole turned part")
        self.direct = self.q_rank == 0
        #: the float32 column of the stacked product at which the gate's sums begin
        self.gate_at = (self.q_rank or self.n_heads * (self.head_dim + self.rot_dim)) + self.kv_rank + self.rot_dim
        self.sink_w = None
        self.cache_width = self.kv_rank + self.rot_dim
        self.w_down = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = self.q_norm_w = self.kv_norm_w = None

    def weight_shapes(self):
        H, D, Dv, E, Rq, R = self.n_heads, self.head_dim, self.value_dim, self.width, self.q_rank, self.kv_rank
        shapes = {"dkv": ((R + self.rot_dim, E), "matrix"), "dkv.norm": ((R,), "norm"), "uk": ((H * D, R), "matrix"),
                  "uv": ((H * Dv, R), "matrix"), "o": ((E, H * Dv), "matrix")}
        if Rq:
            shapes.update({"dq": ((Rq, E), "matrix"), "dq.norm": ((Rq,), "norm"),
                           "uq": ((H * (D + self.rot_dim), Rq), "matrix")})
        else:
            shapes["q"] = ((H * (D + self.rot_dim), E), "matrix")
        if self.sinks:
            shapes["sink"] = ((H,), "matrix")
        if self.value_gate:
            shapes["g"] = ((H * Dv, E), "matrix")
        if self.head_gate:
            shapes["g"] = ((H, E), "matrix")
        return shapes

    def cache_need(self):
        return CacheNeed(1, self.cache_width, self.window, streams=((1, self.cache_width),))

    def bind(self, weights, ops):
        H, D, Dv, R, Rr = self.n_heads, self.head_dim, self.value_dim, self.kv_rank, self.rot_dim
        self.cache_width = Rc = ops.cache_head_width(R + Rr, R + Rr)
        gate = [weights["g"]] if self.value_gate or self.head_gate else []
        if self.q_rank:
            self.w_down = ops.prepare_linear([weights["dq"], weights["dkv"]] + gate)
            self.w_uq = ops.prepare_linear([weights["uq"]])
        else:
            self.w_down = ops.prepare_linear([weights["q"], weights["dkv"]] + gate)
        if self.position is not None:
            self.position.bind({}, ops)
        if self.sinks:
            self.sink_w = weights["sink"].to(device=ops.device, dtype=torch.float32).contiguous()
        self.w_o = ops.prepare_linear([weights["o"]])
        # per head W_uk of the head, transposed, and W_uv.  Where the queries are turned before they enter the latent's
        # space, the first carries an identity block that passes the turned part on, and rows of zeros up to the cache's
        # width: [Rc, D + Rr]; else it is [R, D]
        if self.direct:
            uk = torch.zeros((H, Rc, D + Rr), dtype=weights["uk"].dtype, device=weights["uk"].device)
            uk[:, :R, :D] = weights["uk"].view(H, D, R).transpose(1, 2)
            if Rr:
                uk[:, R:R + Rr, D:] = torch.eye(Rr, dtype=uk.dtype, device=uk.device)
        else:
            uk = weights["uk"].view(H, D, R).transpose(1, 2).contiguous()
        self.w_uk_t = ops.prepare_per_head(uk)
        self.w_uv = ops.prepare_per_head(weights["uv"].view(H, Dv, R))
        f32 = dict(device=ops.device, dtype=torch.float32)
        self.q_norm_w = weights["dq.norm"].to(**f32).contiguous() if self.q_rank else None
        self.kv_norm_w = weights["dkv.norm"].to(**f32).contiguous()

    #: ``h`` may be rows with their norm pending, and ``then_norm`` is handed to the last product
    folds_norms = True

    def forward(self, ctx, h, entry, accumulate_into=None, then_norm=None):
        ops = ctx.ops
        view = ctx.cache_view(entry)
        if not view.writes:
            raise ValueError("latent attention reads only its own cache")
        H = self.n_heads
        # float32 [T, W_dq h (or W_q h) | W_dkv h | W_g h]
        down = ops.linear(h, self.w_down, out_dtype=torch.float32)
        table = self.position.table() if self.position is not None else None
        if self.direct:
            q = ops.latent_rotate_append(down, H, self.head_dim, self.rot_dim, self.kv_rank, table, self.kv_norm_w,
                                         self.norm_eps, ctx.meta, view)            # [T, H * (D + Rr)]; [c | k_r] is cached
            ql = ops.per_head_linear(q, self.w_uk_t)                                # [T, H * Rc]: W_uk^T q per head
        else:
            cq = ops.latent_norm_append(down, self.q_rank, self.kv_rank, self.q_norm_w, self.kv_norm_w, self.norm_eps,
                                        ctx.meta, view, rot_dim=self.rot_dim, table=table)    # [T, q_rank]; [c | k_r] is cached
            q = ops.linear(cq, self.w_uq)                                           # [T, H * (D + Rr)]
            ql = ops.latent_queries(q, self.w_uk_t, self.rot_dim, view.head_dim, table, ctx.meta)
        both = dataclasses.replace(view, v=view.k)                                  # keys and values: the latents
        if self.sinks:
            a = ops.attention(ql.view(ql.shape[0], H, view.head_dim), ctx.meta, both, H, self.scale, self.window,
                              sinks=self.sink_w)
        else:
            a = ops.attention(ql.view(ql.shape[0], H, view.head_dim), ctx.meta, both, H, self.scale, self.window)
        gate = (down, self.gate_at) if self.value_gate else (down, self.gate_at, "head") if self.head_gate else None
        o = ops.per_head_linear(a, self.w_uv, gate=gate)                            # [T, H * Dv]
        if accumulate_into is None:
            return ops.linear(o, self.w_o, out_dtype=torch.float32)
        if then_norm is None:
            return ops.linear(o, self.w_o, accumulate_into=accumulate_into)
        return ops.linear(o, self.w_o, accumulate_into=accumulate_into, then_norm=then_norm)


register_part("mixer", "latent_attention", LatentAttention)
