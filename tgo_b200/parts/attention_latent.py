"""Causal softmax attention over a compressed cache (the latent attention of DeepSeek-V2):
every token keeps ONE small row instead of keys and values per head.

    c_q = norm(W_dq x) * g_q                     the queries' latent (query_rank wide)
    q_h = W_uq,h c_q = [q_h,nope (head_dim), q_h,rope (rope_dim)]
    [c', r'] = W_dkv x;   c = norm(c') * g_kv    the latent (latent_rank wide)
                          r = rotated r'         one rotated key part for all heads (rope_dim)
    k_h,nope(j) = W_uk,h c(j),   v_h(j) = W_uv,h c(j)
    score_h(i, j) = (q_h,nope(i) . k_h,nope(j) + rotated q_h,rope(i) . r(j)) * scale,  j <= i
    out = W_o concat_h softmax_j(score_h(i, .)) v_h

The cache holds [c, r] per token, one plane, rows latent_rank + rope_dim wide. Keys and values
are never expanded: since q_nope . (W_uk c) = (W_uk^T q_nope) . c and sum_j w_j W_uv c(j) =
W_uv sum_j w_j c(j), the expansion matrices are applied to the query and to the attention's
result, a product per head, and the attention itself has one key/value head whose key is the
whole cached row and whose value is its first latent_rank channels. It runs in the kernels of
`sink_attention` (`parts/attention_sink.py`), which take such a row. Norms, rotation, scores
and softmax are float32. Tensor roles: q_down, q_down_norm, q_up, kv_down, kv_norm, k_up, v_up, o.

What the spec may change: `query_rank` 0, q_h straight from x by one matrix (role q instead of the
three of the queries' latent); `window`, a query reads itself and the window - 1 rows before it;
`sink` (role sink), exp(sink_h) joins every softmax's denominator, unscaled and without a value;
`output_gate` (role gate), the concatenated heads are multiplied by the logistic function of
W_g x; `borrows_latent`, the layer has no W_dkv and reads the rows that the call whose cache it
borrows has written (`cache_row` wide; channels past the latent meet zeros in the query).
Matrices that read x itself (q, kv_down, gate) are joined into one product at bind time.
"""
from __future__ import annotations

import math
from typing import List

import torch

from ..config.spec import MixerSpec, tensor_names
from ..kernels import ops
from ..registry import MIXERS, POSITIONS
from ..weights.binder import WeightSpec
from .attention import step_tiles
from .attention_sink import sink_attention, tile_form
from .base import CacheNeed, LayerCache, Part


class LatentAttention(Part):
    out_dtype = None                 # dtype of the output product's rows (None: activations')

    def __init__(self, spec: MixerSpec, hidden: int, prefix: str, device=None):
        self.hidden = hidden
        self.H, self.dn, self.dr = spec.num_heads, spec.head_dim, spec.rope_dim
        self.dv = spec.value_dim or spec.head_dim
        self.rank, self.q_rank = spec.latent_rank, spec.query_rank
        if min(self.H, self.dn, self.dv, self.rank) <= 0 or min(self.dr, self.q_rank) < 0:
            raise ValueError("latent attention: heads, head_dim, value_dim and latent_rank must be "
                             "positive")
        self.borrows = bool(getattr(spec, "borrows_latent", False))
        self.row = int(getattr(spec, "cache_row", 0)) or self.rank + self.dr   # a token's cached row
        if self.row < self.rank + self.dr or (self.row != self.rank + self.dr and not self.borrows):
            raise ValueError(f"latent attention: cached rows of {self.row} for a latent of {self.rank} "
                             f"and a rotated part of {self.dr}")
        self.window = spec.window
        self.sink, self.gated = bool(spec.sink), bool(spec.output_gate)
        if self.gated and spec.gate_activation != "sigmoid":
            raise ValueError("latent attention: the output gate is a logistic one")
        self.eps = float(spec.norm_eps)
        self.scale = spec.scale if spec.scale is not None else 1.0 / math.sqrt(self.dn + self.dr)
        pos = spec.position
        self.position = POSITIONS.get(pos.kind)(pos, self.dr, device) \
            if pos is not None and self.dr else None
        if self.position is not None and not hasattr(self.position, "table"):
            raise ValueError("latent attention: the rotation is done inside its kernels and needs "
                             "a position encoding that offers a table of cosines and sines")
        roles = (["q_down", "q_down_norm", "q_up"] if self.q_rank else ["q"]) + \
            ([] if self.borrows else ["kv_down", "kv_norm"]) + ["k_up", "v_up", "o"] + \
            (["sink"] if self.sink else []) + (["gate"] if self.gated else [])
        self.names = tensor_names(spec.tensors, prefix, roles, "latent attention")
        self.w_dq = self.w_uq = self.w_in = self.w_uk_t = self.w_uv = self.w_o = None
        self.q_gain = self.kv_gain = self.sinks = None
        # columns of the joined product: q, or nothing when q has a latent; then the row to
        # cache; then the gate
        self.qw = 0 if self.q_rank else self.H * (self.dn + self.dr)
        self.kvw = 0 if self.borrows else self.rank + self.dr
        self.gw = self.H * self.dv if self.gated else 0

    def weight_specs(self):
        n, d, H = self.names, self.hidden, self.H
        qw = H * (self.dn + self.dr)
        out = [WeightSpec(n["q_down"], (self.q_rank, d)),
               WeightSpec(n["q_down_norm"], (self.q_rank,), "gain"),
               WeightSpec(n["q_up"], (qw, self.q_rank))] if self.q_rank else [WeightSpec(n["q"], (qw, d))]
        if not self.borrows:
            out += [WeightSpec(n["kv_down"], (self.rank + self.dr, d)),
                    WeightSpec(n["kv_norm"], (self.rank,), "gain")]
        out += [WeightSpec(n["k_up"], (H * self.dn, self.rank)),
                WeightSpec(n["v_up"], (H * self.dv, self.rank)),
                WeightSpec(n["o"], (d, H * self.dv))]
        if self.sink:
            out.append(WeightSpec(n["sink"], (H,), "gain"))
        if self.gated:
            out.append(WeightSpec(n["gate"], (H * self.dv, d)))
        return out

    def cache_need(self):
        return CacheNeed("full" if self.window is None else "window", self.window, 1, (1, self.row))

    def state_need(self):
        return None

    def bind(self, weights):
        n, H = self.names, self.H
        first = []                       # what reads x itself, in the order of the joined columns
        if self.q_rank:
            self.w_dq = weights.pop(n["q_down"]).contiguous()
            self.w_uq = weights.pop(n["q_up"]).contiguous()
            self.q_gain = weights.pop(n["q_down_norm"]).to(torch.float32).contiguous()
        else:
            first.append(weights.pop(n["q"]))
        if not self.borrows:
            first.append(weights.pop(n["kv_down"]))
            self.kv_gain = weights.pop(n["kv_norm"]).to(torch.float32).contiguous()
        if self.gated:
            first.append(weights.pop(n["gate"]))
        if first:
            self.w_in = torch.cat(first, dim=0).contiguous()
        if self.sink:
            self.sinks = weights.pop(n["sink"]).to(torch.float32).contiguous()
        # per head: W_uk,h^T [latent_rank, head_dim] (applied to the query) and W_uv,h
        # [value_dim, latent_rank] (applied to the attention's result)
        self.w_uk_t = weights.pop(n["k_up"]).reshape(H, self.dn, self.rank).transpose(1, 2).contiguous()
        self.w_uv = weights.pop(n["v_up"]).reshape(H, self.dv, self.rank).contiguous()
        self.w_o = weights.pop(n["o"]).contiguous()

    def libraries(self, dtype, page_size) -> List[str]:
        names = ["sgemm" if dtype == torch.float32 else "gemm_skinny", "elementwise", "layer_ops",
                 "latent", "attention_generic"]
        if dtype == torch.bfloat16:
            names.append("attention_sink")
        return names

    def prepare_capture(self, ctx, cache) -> None:
        form, tokens = tile_form(self.H, 1, self.row, self.rank, self.row, ctx.act_dtype)
        if not ctx.decode_only and cache is not None and form is not None:
            step_tiles(ctx, tokens)

    def flops(self, extents, first_positions, writes_cache: bool = True) -> float:
        n, H, d = sum(extents), self.H, self.hidden
        per_token = d * (self.qw + self.kvw + self.gw + self.q_rank) + \
            self.q_rank * H * (self.dn + self.dr) + H * self.dn * self.rank + H * self.dv * self.rank + \
            H * self.dv * d
        reach = self.window or max((f + e for f, e in zip(first_positions, extents)), default=0)
        keys = 0
        for first, extent in zip(first_positions, extents):
            short = max(0, min(extent, reach - first))           # queries that see every earlier key
            keys += short * first + short * (short + 1) // 2 + (extent - short) * reach
        return 2.0 * n * per_token + 2.0 * H * (self.row + self.rank) * keys

    def cache_bytes_read(self, context_len: float, width: int) -> float:
        return self.row * width * (min(context_len, self.window) if self.window else context_len)

    def forward(self, x, ctx, cache: LayerCache):
        H, dn, dr, dv, rank, row = self.H, self.dn, self.dr, self.dv, self.rank, self.row
        x = ops.rows_of(x)
        T, dev = x.shape[0], x.device
        if cache.writable == self.borrows or cache.k.shape[-1] != row:
            raise ValueError("latent attention: a layer that borrows its latent must be called with the "
                             f"cache of another call whose rows are {row} wide, any other with its own")
        y = ops.linear(x, self.w_in) if self.w_in is not None else None
        if self.q_rank:
            # the queries' latent: product in float32 rows, norm, then the up product
            cq_raw = ops.linear(x, self.w_dq, out_dtype=torch.float32)
            cq = torch.empty((T, self.q_rank), dtype=x.dtype, device=dev)
            ops.gated_group_norm(cq_raw, None, self.q_gain, cq, 1, self.eps, None, False)
            q = ops.linear(cq, self.w_uq)                               # [T, H (dn + dr)]
        else:
            q = y[:, :self.qw]
        gate = y[:, self.qw + self.kvw:] if self.gated else None
        table, rot, interleaved = None, 0, False
        if self.position is not None:
            table, rot = self.position.table(ctx), self.position.rotary_dim
            interleaved = getattr(self.position, "pairing", "half_split") == "interleaved"
        if not self.borrows:
            ops.latent_row_cache(y[:, self.qw:self.qw + self.kvw], rank, dr, self.kv_gain, self.eps, table,
                                 rot, interleaved, cache.slots, cache.k, cache.page_size)
        # the query as the cache sees it: [W_uk^T q_nope, rotated q_rope] per head, zeros where the
        # cached row has channels this layer does not know
        fill = torch.zeros if row > rank + dr else torch.empty
        qa = fill((T, H * row), dtype=x.dtype, device=dev)
        ops.head_linear(q, dn + dr, self.w_uk_t, qa, row)
        if dr:
            ops.rope_slice(q, dn + dr, dn, qa, row, rank, H, dr, table, rot, interleaved)
        lat = torch.empty((T, H * rank), dtype=x.dtype, device=dev)
        sink_attention(qa, lat, H, 1, row, rank, cache, ctx, self.scale, self.window or 0, self.sinks,
                       value_row=row)
        a = torch.empty((T, H * dv), dtype=x.dtype, device=dev)
        ops.head_linear(lat, rank, self.w_uv, a, dv, gate)
        return ops.linear(a, self.w_o, out_dtype=self.out_dtype)


MIXERS.register("latent_attention", LatentAttention)
