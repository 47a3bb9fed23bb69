"""A recurrent block with a real-gated linear recurrent unit as a mixer.

    u_t   = conv(W_x h + b_x)                       a short causal convolution per channel, with a bias
    y_t   = gelu_tanh(W_y h + b_y)
    r_t   = sigmoid(R_b u + b),   i_t = sigmoid(I_b u + b)      a square matrix per equal part b of the channels
    a_t   = exp(-8 r_t softplus(lam))
    S_t   = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t   element by element, S_(-1) = 0
    out_t = W_o (S_t y_t)

Neither gate reads the state, so a portion's gates are products over all its tokens, and the recurrence is a scan over float32
numbers (in pieces side by side for long portions).  A request carries S and the convolution's last inputs, float32, in its state
slot.  A step of one token a request runs everything between the two projections as one kernel.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import FixedState
from ..weights import MATRIX, VECTOR, TensorSpec
from .base import Part, register_part

# portions of a request longer than this run the recurrence in pieces side by side
RGLRU_PIECES_FROM = 64
# tokens of a step from which the gates' products run on tensor cores (bfloat16)
RGLRU_PRODUCTS_FROM = 32


class RealGatedLRU(Part):
    graph_safe = True

    def __init__(self, width: int, inner: int, blocks: int, taps: int):
        if inner % blocks:
            raise ValueError(f"{inner} channels do not fall into {blocks} equal parts")
        self.width, self.inner, self.blocks, self.taps = width, inner, blocks, taps
        self.w_in = self.b_in = self.wo = self.conv_w = self.conv_b = self.sp8 = None
        self.ra = self.ri = self.ra_b = self.ri_b = self.w_gates = None
        self._tiles = {}

    def cache_spec(self):
        return FixedState((ops.rglru_state_floats(self.inner, self.taps),), torch.float32)

    def tensor_specs(self, prefix):
        E, C, B = self.width, self.inner, self.blocks
        P = C // B
        t = lambda name, shape, kind=MATRIX, init=(0.0, 1.0): TensorSpec(prefix + name, shape, kind, init=init)
        return [t(".y", (C, E)), t(".y.b", (C,), VECTOR), t(".x", (C, E)), t(".x.b", (C,), VECTOR),
                t(".conv", (C, self.taps), VECTOR, (1.0 / self.taps, 2.0)), t(".conv.b", (C,), VECTOR),
                t(".ra", (B, P, P)), t(".ra.b", (B, P), VECTOR), t(".ri", (B, P, P)), t(".ri.b", (B, P), VECTOR),
                t(".lam", (C,), VECTOR, (-4.0, 10.0)), t(".o", (E, C))]

    def bind(self, prefix, tensors, rt):
        t = lambda n: tensors[prefix + n]
        self.w_in = torch.cat([t(".x"), t(".y")], dim=0).contiguous()
        self.b_in = torch.cat([t(".x.b"), t(".y.b")]).contiguous()
        self.conv_w, self.conv_b = t(".conv").t().contiguous(), t(".conv.b").contiguous()
        self.ra, self.ri = t(".ra").contiguous(), t(".ri").contiguous()
        self.ra_b, self.ri_b = t(".ra.b").reshape(-1).contiguous(), t(".ri.b").reshape(-1).contiguous()
        self.w_gates = ops.rglru_pieces_matrices(self.ra, self.ri) if rt.dtype == torch.bfloat16 and (self.inner // self.blocks) % 8 == 0 else None
        # 8 softplus(lam), from double precision
        self.sp8 = (8.0 * torch.nn.functional.softplus(t(".lam").double())).float().contiguous()
        self.wo = t(".o")

    def first_weights(self):
        return [self.w_in]

    def _part_tiles(self, n: int, device) -> torch.Tensor:
        """The grouped product's tile list for n tokens: the part of every tile, then how many tiles (made once per number of tiles)."""
        rows, tile = ops.rglru_pieces_rows(n)
        per = rows // tile
        got = self._tiles.get(per)
        if got is None:
            flat = [v for b in range(self.blocks) for _ in range(per) for v in (b, 0, 0)] + [self.blocks * per]
            got = self._tiles[per] = torch.tensor(flat, dtype=torch.int32).to(device)
        return got

    def forward(self, rt, h, batch, cache):
        proj = rt.linear(h, self.w_in, bias=self.b_in, out_dtype=torch.float32)         # [tokens, x | y]
        if batch.max_q_len == 1:
            out = ops.rglru_step(proj, self.conv_w, self.conv_b, cache.state, batch.slots, batch.positions, self.ra, self.ra_b, self.ri, self.ri_b, self.sp8)
            return rt.linear(out, self.wo, partials_ok=True)
        n = h.shape[0]
        chunks = chunk_start = ends = None
        if batch.max_q_len > RGLRU_PIECES_FROM:
            chunks, chunk_start = batch.scan_pieces(ops.rglru_chunk_tokens())
        products = self.w_gates is not None and n >= RGLRU_PRODUCTS_FROM
        u = ops.rglru_conv(proj, self.conv_w, self.conv_b, cache.state, batch.seq_of_token, batch.seq_start, batch.slots, batch.positions,
                           part=self.inner // self.blocks if products else 0)
        if products:
            ab, ends = ops.rglru_gates_pieces(u, n, self.w_gates, self._part_tiles(n, h.device), self.ra_b, self.ri_b, self.sp8, rt.status, chunks=chunks)
        else:
            ab = ops.rglru_gates(u, self.ra, self.ra_b, self.ri, self.ri_b, self.sp8)
        out = torch.empty((n, self.inner), dtype=rt.dtype, device=h.device)
        ops.rglru_scan(ab, proj, cache.state, batch.seq_start, batch.slots, out, chunks, chunk_start, ends=ends)
        return rt.linear(out, self.wo, partials_ok=True)


register_part("mixer", "rglru", RealGatedLRU)
