"""The gated delta rule as a mixer: with a decay per key channel ("channel delta") or one per head ("head delta").

Per token, from the mixer's input h (H value heads on G query/key heads; head h reads
query/key head h // (H / G)):

    q, k, v   = silu(conv(W h))           short causal convolutions over time, one filter per channel
    q         = q / |q| * D^-1/2,  k = k / |k|                     |x| = sqrt(sum x^2 + 1e-6), per head
    beta      = sigmoid(W_b h)                                      one per head
    g         = exp(-exp(A_log) * softplus(W_a2 W_a1 h + dt_bias))   one per head and key channel
    S        <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          per head, S [D, Dv]
    out       = W_o (o / rms(o) * w_norm * sigmoid(W_g2 W_g1 h))

With one decay per head, g = exp(-exp(A_log) * softplus(W_a h + dt_bias)) is one number per head, and the output
gate is silu(W_g h) (no low-rank projections); everything else is the same.

What a request carries from token to token is one float32 vector in its state slot: S of
every head, then the last taps - 1 inputs of the convolutions.  The four wide projections of h
are one product, the two narrow ones (into the low ranks) another.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import FixedState
from ..weights import VECTOR, TensorSpec
from .base import Part, register_part


class ChannelDelta(Part):
    graph_safe = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, head_dim: int, v_head_dim: int, taps: int, rank_a: int,
                 rank_g: int, eps: float):
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads are no multiple of {n_kv_heads} key heads")
        self.width, self.n_heads, self.n_kv_heads = width, n_heads, n_kv_heads
        self.head_dim, self.v_head_dim, self.taps = head_dim, v_head_dim, int(taps)
        self.rank_a, self.rank_g, self.eps = int(rank_a), int(rank_g), float(eps)
        self.channels = 2 * n_kv_heads * head_dim + n_heads * v_head_dim
        self.state_floats = n_heads * head_dim * v_head_dim            # S of every head; the convolutions' inputs follow
        self.w_in = self.w_low = self.w_a2 = self.w_g2 = self.wo = self.conv_w = self.a_log = self.dt_bias = self.norm_w = None

    def cache_spec(self):
        return FixedState((self.state_floats + (self.taps - 1) * self.channels,), torch.float32)

    def tensor_specs(self, prefix):
        H, G, D, Dv, E = self.n_heads, self.n_kv_heads, self.head_dim, self.v_head_dim, self.width
        return [
            TensorSpec(prefix + ".q", (G * D, E)), TensorSpec(prefix + ".q.conv", (G * D, self.taps), VECTOR, init=(0.0, 10.0)),
            TensorSpec(prefix + ".k", (G * D, E)), TensorSpec(prefix + ".k.conv", (G * D, self.taps), VECTOR, init=(0.0, 10.0)),
            TensorSpec(prefix + ".v", (H * Dv, E)), TensorSpec(prefix + ".v.conv", (H * Dv, self.taps), VECTOR, init=(0.0, 10.0)),
            TensorSpec(prefix + ".b", (H, E)), TensorSpec(prefix + ".A_log", (H,), VECTOR),
            TensorSpec(prefix + ".norm", (Dv,), VECTOR, init=(1.0, 1.0)),
            TensorSpec(prefix + ".a1", (self.rank_a, E)), TensorSpec(prefix + ".a2", (H * D, self.rank_a)),
            TensorSpec(prefix + ".dt_bias", (H * D,), VECTOR),
            TensorSpec(prefix + ".g1", (self.rank_g, E)), TensorSpec(prefix + ".g2", (H * Dv, self.rank_g)),
            TensorSpec(prefix + ".o", (E, H * Dv)),
        ]

    def bind(self, prefix, tensors, rt):
        t = lambda n: tensors[prefix + n]
        self.w_in = torch.cat([t(".q"), t(".k"), t(".v"), t(".b")], dim=0).contiguous()
        self.w_low = torch.cat([t(".a1"), t(".g1")], dim=0).contiguous()
        self.w_a2, self.w_g2, self.wo = t(".a2"), t(".g2"), t(".o")
        self.conv_w = torch.cat([t(".q.conv"), t(".k.conv"), t(".v.conv")], dim=0).float().contiguous()
        self.a_log, self.dt_bias, self.norm_w = t(".A_log"), t(".dt_bias"), t(".norm")

    def first_weights(self):
        return [self.w_in]

    def forward(self, rt, h, batch, cache):
        H, G, D, Dv = self.n_heads, self.n_kv_heads, self.head_dim, self.v_head_dim
        proj = rt.linear(h, self.w_in, out_dtype=torch.float32)
        low = rt.linear(h, self.w_low)
        a_pre = rt.linear(low[:, :self.rank_a], self.w_a2, out_dtype=torch.float32)
        g_pre = rt.linear(low[:, self.rank_a:], self.w_g2, out_dtype=torch.float32)
        qkv_c, gb = ops.delta_prepare(proj, a_pre, self.conv_w, cache.state, self.state_floats, batch.seq_of_token,
                                      batch.seq_start, batch.slots, self.a_log, self.dt_bias, H, G, D, Dv)
        o = ops.delta_scan(qkv_c, gb, cache.state, batch.seq_start, batch.slots, H, G, D, Dv)
        y = ops.delta_output(o, self.norm_w, g_pre, self.eps, rt.dtype, H)
        return rt.linear(y, self.wo, partials_ok=True)


class HeadDelta(Part):
    """One decay per head, a full-rank output gate with silu.  Every projection of h is one product (``in_rows``)."""

    graph_safe = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, head_dim: int, v_head_dim: int, taps: int, eps: float):
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads are no multiple of {n_kv_heads} key heads")
        if not 1 <= taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"a convolution of {taps} taps (1 to {ops.CONV_MAX_TAPS})")
        self.width, self.n_heads, self.n_kv_heads = width, n_heads, n_kv_heads
        self.head_dim, self.v_head_dim, self.taps, self.eps = head_dim, v_head_dim, int(taps), float(eps)
        self.channels = 2 * n_kv_heads * head_dim + n_heads * v_head_dim
        self.conv_off = -(-(n_heads * head_dim * v_head_dim) // 4) * 4        # S of every head, then the convolutions' inputs (from a 16-byte boundary)
        self.w_in = self.wo = self.conv_w = self.a_log = self.dt_bias = self.norm_w = None

    def cache_spec(self):
        return FixedState((-(-(self.conv_off + (self.taps - 1) * self.channels) // 4) * 4,), torch.float32)

    def tensor_specs(self, prefix):
        H, G, D, Dv, E = self.n_heads, self.n_kv_heads, self.head_dim, self.v_head_dim, self.width
        conv = lambda n, c: TensorSpec(prefix + n, (c, self.taps), VECTOR, init=(0.0, 10.0))
        return [
            TensorSpec(prefix + ".q", (G * D, E)), conv(".q.conv", G * D), TensorSpec(prefix + ".k", (G * D, E)), conv(".k.conv", G * D),
            TensorSpec(prefix + ".v", (H * Dv, E)), conv(".v.conv", H * Dv), TensorSpec(prefix + ".b", (H, E)), TensorSpec(prefix + ".a", (H, E)),
            TensorSpec(prefix + ".A_log", (H,), VECTOR), TensorSpec(prefix + ".dt_bias", (H,), VECTOR),
            TensorSpec(prefix + ".norm", (Dv,), VECTOR, init=(1.0, 1.0)), TensorSpec(prefix + ".g", (H * Dv, E)), TensorSpec(prefix + ".o", (E, H * Dv)),
        ]

    def bind(self, prefix, tensors, rt):
        t = lambda n: tensors[prefix + n]
        self.w_in = torch.cat([t(".q"), t(".k"), t(".v"), t(".g"), t(".b"), t(".a")], dim=0).contiguous()
        self.conv_w = torch.cat([t(".q.conv"), t(".k.conv"), t(".v.conv")], dim=0).float().t().contiguous()      # [taps, channels]
        self.wo = t(".o")
        self.a_log, self.dt_bias, self.norm_w = (t(n).float().contiguous() for n in (".A_log", ".dt_bias", ".norm"))

    def in_rows(self):
        return self.w_in, None

    def first_weights(self):
        return [self.w_in]

    def forward_projected(self, rt, proj, batch, cache):
        H, G, D, Dv, C = self.n_heads, self.n_kv_heads, self.head_dim, self.v_head_dim, self.channels
        qkv = torch.empty((proj.shape[0], C), dtype=torch.float32, device=proj.device)
        ops.short_conv(proj[:, :C], self.conv_w, None, cache.state[:, self.conv_off:] if self.taps > 1 else None, batch.seq_of_token, batch.seq_start,
                       batch.slots, qkv, act="silu")
        g0, b0, a0 = C, C + H * Dv, C + H * Dv + H
        gb = ops.delta_head_prepare(qkv, proj[:, a0:a0 + H], proj[:, b0:b0 + H], self.a_log, self.dt_bias, H, G, D)
        chunks = batch.scan_chunks(ops.CHUNK_TOKENS, ops.CHUNK_FROM) if batch.max_q_len > ops.CHUNK_FROM else None
        o = ops.delta_scan(qkv, gb, cache.state, batch.seq_start, batch.slots, H, G, D, Dv, chunks=chunks)
        y = ops.delta_output(o, self.norm_w, proj[:, g0:g0 + H * Dv], self.eps, rt.dtype, H, act="silu")
        return rt.linear(y, self.wo, partials_ok=True)

    def forward(self, rt, h, batch, cache):
        return self.forward_projected(rt, rt.linear(h, self.w_in, out_dtype=torch.float32), batch, cache)


register_part("mixer", "channel_delta", ChannelDelta)
register_part("mixer", "head_delta", HeadDelta)
