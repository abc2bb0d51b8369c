"""A gated delta-rule mixer: H value heads of `value_dim` channels over G query/key heads of
`head_dim`, a matrix memory S [head_dim, value_dim] per head that is corrected by the error of its
own recall:

    q, k, v <- silu(causal convolution per channel, `conv_taps` taps, no bias) of W_q x, W_k x, W_v x
    q, k    <- divided by sqrt(sum of squares + 1e-6) per head; q also by sqrt(head_dim)
    beta     = sigmoid(W_b x)                                            one per head
    g        = exp(-exp(A_log) softplus(W_a x + dt_bias))                one per head
    S       <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
    out      = W_o ( gain * rmsnorm(o, each head alone) * silu(W_g x) )

Head h uses the q and k of head floor(h / (H / G)); the gain has value_dim entries that all heads
share. The projections are in the activation type (one joined product); everything from the
convolution to the norm is float32. Per request the mixer keeps, as one float32 state row, S [H,
head_dim, value_dim] and the convolution's last taps - 1 inputs [taps - 1, C] (q, k, v side by side).

A step of single tokens runs two kernels between the products (`delta_prepare`, `delta_step`), any
other step three (`delta_prepare`, `delta_scan`, the gated norm).

Spec fields: num_heads = H, num_kv_heads = G, head_dim, value_dim, conv_taps, norm_eps. Tensor roles:
q, k, v, q_conv, k_conv, v_conv, a, b, gate, a_log, dt_bias, norm, o.
"""
from __future__ import annotations

from typing import List

import torch

from ..config.spec import MixerSpec, tensor_names
from ..kernels import ops
from ..registry import MIXERS
from ..weights.binder import WeightSpec
from .base import LayerCache, Part, StateNeed

USE_STEP_KERNEL = True           # steps of single tokens on their own kernel


class GatedDelta(Part):
    out_dtype = None                 # dtype of the output product's rows (None: activations')

    def __init__(self, spec: MixerSpec, hidden: int, prefix: str, device=None):
        self.hidden = hidden
        self.H, self.G, self.dk = spec.num_heads, spec.num_kv_heads, spec.head_dim
        self.dv = spec.value_dim or spec.head_dim
        self.taps = int(spec.conv_taps)
        if min(self.H, self.G, self.dk, self.dv, self.taps) <= 0 or self.H % self.G:
            raise ValueError(f"delta mixer: heads {self.H} over {self.G}, keys {self.dk}, values {self.dv}, "
                             f"taps {self.taps}")
        self.eps = float(spec.norm_eps)
        self.kw, self.vw = self.G * self.dk, self.H * self.dv
        self.C = 2 * self.kw + self.vw                       # channels through the convolution
        self.mem_floats = self.H * self.dk * self.dv
        self.conv_at = (self.mem_floats + 3) // 4 * 4        # 16-byte places in the state row
        self.names = tensor_names(spec.tensors, prefix,
                                  ["q", "k", "v", "q_conv", "k_conv", "v_conv", "a", "b", "gate", "a_log",
                                   "dt_bias", "norm", "o"], "delta mixer")
        self.w_in = self.w_o = self.conv = self.decay = self.dt_bias = self.gain = self.gain_row = None

    def weight_specs(self):
        n, d, H, t = self.names, self.hidden, self.H, self.taps
        return [WeightSpec(n["q"], (self.kw, d)), WeightSpec(n["k"], (self.kw, d)), WeightSpec(n["v"], (self.vw, d)),
                WeightSpec(n["q_conv"], (self.kw, t), "constant"), WeightSpec(n["k_conv"], (self.kw, t), "constant"),
                WeightSpec(n["v_conv"], (self.vw, t), "constant"), WeightSpec(n["a"], (H, d)),
                WeightSpec(n["b"], (H, d)), WeightSpec(n["gate"], (self.vw, d)),
                WeightSpec(n["a_log"], (H,), "gain"), WeightSpec(n["dt_bias"], (H,), "gain"),
                WeightSpec(n["norm"], (self.dv,), "gain"), WeightSpec(n["o"], (d, self.vw))]

    def cache_need(self):
        return None

    def state_need(self):
        return StateNeed(((self.conv_at + (self.taps - 1) * self.C + 3) // 4 * 4,))

    def bind(self, weights):
        n = self.names
        rows = [weights.pop(n[r]) for r in ("q", "k", "v", "gate", "b", "a")]
        count = sum(r.shape[0] for r in rows)
        if count % 8:                                # whole 16-byte rows for the products
            rows.append(rows[0].new_zeros((8 - count % 8, self.hidden)))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = weights.pop(n["o"]).contiguous()
        self.conv = torch.cat([weights.pop(n[r]).to(torch.float32) for r in ("q_conv", "k_conv", "v_conv")],
                              dim=0).t().contiguous()                            # [taps, C]
        # the factor on the step, made in float64 and rounded once
        self.decay = torch.exp(weights.pop(n["a_log"]).double()).float().contiguous()
        self.dt_bias = weights.pop(n["dt_bias"]).to(torch.float32).contiguous()
        self.gain = weights.pop(n["norm"]).to(torch.float32).contiguous()
        self.gain_row = self.gain.repeat(self.H).contiguous()                    # all heads' gains side by side

    def libraries(self, dtype, page_size) -> List[str]:
        return ["sgemm" if dtype == torch.float32 else "gemm_skinny", "layer_ops", "delta"]

    def flops(self, extents, first_positions, writes_cache: bool = True) -> float:
        n = sum(extents)
        products = 2.0 * n * self.hidden * (2 * self.kw + 3 * self.vw + 2 * self.H)
        return products + 2.0 * n * self.C * self.taps + 6.0 * n * self.mem_floats

    def cache_bytes_read(self, context_len: float, width: int) -> float:
        return 4.0 * (self.mem_floats + (self.taps - 1) * self.C)       # the state, whatever the length

    def forward(self, x, ctx, cache: LayerCache):
        x = ops.rows_of(x)
        T, C, H, vw = x.shape[0], self.C, self.H, self.vw
        rows = ops.linear(x, self.w_in)
        raw, z = rows[:, :C], rows[:, C:C + vw]
        b, a = rows[:, C + vw:C + vw + H], rows[:, C + vw + H:C + vw + 2 * H]
        sizes = (ctx.num_seqs, H, self.G, self.dk, self.dv)
        state = cache.state
        prepared = ops.delta_prepare(raw, self.conv, b, a, self.dt_bias, self.decay, *sizes, ctx.seq_ids,
                                     ctx.q_start, ctx.state_slots, state, self.conv_at)
        n = torch.empty((T, vw), dtype=x.dtype, device=x.device)
        if ctx.decode_only and USE_STEP_KERNEL and ops.delta_step_supports(*sizes[1:], state, 0):
            ops.delta_step(prepared, z, self.gain, self.eps, n, *sizes, ctx.q_start, ctx.state_slots, state, 0,
                           raw, self.taps, self.conv_at)
        else:
            y = torch.empty((T, vw), dtype=torch.float32, device=x.device)
            ops.delta_scan(prepared, y, *sizes, ctx.q_start, ctx.state_slots, state, 0, raw, self.taps,
                           self.conv_at)
            ops.gated_group_norm(y, z, self.gain_row, n, H, self.eps, "silu", False)
        return ops.linear(n, self.w_o, out_dtype=self.out_dtype)


MIXERS.register("gated_delta", GatedDelta)
