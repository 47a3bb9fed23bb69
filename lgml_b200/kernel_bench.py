"""Time one kernel of the engine alone, at sizes given on the command line.

    python -m lgml_b200.kernel_bench gemm --m 8 --n 28672 --k 4096 [--swiglu] [--f32-out]
    python -m lgml_b200.kernel_bench decode_attention --batch 8 --context 2176 --heads 32 --kv-heads 8 --head-dim 128
    python -m lgml_b200.kernel_bench prefill_attention --tokens 2048 --heads 32 --kv-heads 8 --head-dim 128
    python -m lgml_b200.kernel_bench rmsnorm --rows 8 --width 4096 --parts 9
    python -m lgml_b200.kernel_bench token_shift --rows 2048 --width 4096
    python -m lgml_b200.kernel_bench mingru --rows 2048 --width 4096 [--requests 8]
    python -m lgml_b200.kernel_bench token_side --rows 8 --width 4096 --dim 64
    python -m lgml_b200.kernel_bench chunk_scan --rows 2048 --heads 16 --kv-heads 8 --dim 128 --vdim 128 [--memory]
    python -m lgml_b200.kernel_bench stream_norm --rows 2048 --width 4096 --streams 2
    python -m lgml_b200.kernel_bench scaled_norm --rows 2048 --width 4096 [--top 2] [--parts 9]
    python -m lgml_b200.kernel_bench rglru --rows 2048 --width 4096 --part 256 [--requests 8]

Each case is run over a ring of input buffers larger than the L2 cache, so that weights and
cache pages come from HBM as they do in a decode step; warm-up launches first, then the timed
launches between two CUDA events.  It prints the time per launch and the bytes or flops per
second that the kernel's own inputs and outputs amount to.  The same commands are what the
profiles under ``profiles/`` were captured from.
"""
from __future__ import annotations

import argparse
import sys

import torch

from . import ops

DEV = "cuda:0"
L2_BYTES = 126 << 20


USE_GRAPH = True


def timed(fn, n_buffers: int, warmup: int, iters: int) -> float:
    """Microseconds per call of fn(i), i cycling over the buffers.  The timed calls are
    captured into one CUDA graph and replayed, so that the host's launch cost (tens of
    microseconds from Python) does not sit between kernels that take less than that; launches
    follow one another as they do inside a captured decode step."""
    for i in range(warmup):
        fn(i % n_buffers)
    torch.cuda.synchronize()
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if USE_GRAPH:
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, capture_error_mode="relaxed"):
            for i in range(iters):
                fn(i % n_buffers)
        g.replay()
        torch.cuda.synchronize()
        start.record()
        g.replay()
        end.record()
    else:
        start.record()
        for i in range(iters):
            fn(i % n_buffers)
        end.record()
    torch.cuda.synchronize()
    return start.elapsed_time(end) * 1e3 / iters


def ring(bytes_per_buffer: int) -> int:
    return max(2, -(-2 * L2_BYTES // max(bytes_per_buffer, 1)))


def case_gemm(a) -> None:
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    M, N, K = a.m, a.n, a.k
    nb = min(ring(N * K * 2), 24)
    ws = [(torch.randn(N, K, device=DEV) * 0.02).to(torch.bfloat16) for _ in range(nb)]
    x = torch.randn(M, K, device=DEV).to(torch.bfloat16)
    n_out = N // 2 if a.swiglu else N
    out = torch.empty(M, n_out, dtype=torch.float32 if a.f32_out else torch.bfloat16, device=DEV)
    splits = None if a.splits < 0 else a.splits
    scratch = torch.empty(max(64 * M * N, 1), dtype=torch.float32, device=DEV) if not a.swiglu else None

    def run(i):
        if a.library:
            torch.mm(x, ws[i].t())
        elif a.swiglu:
            ops.gemm_tcgen05(x, ws[i], out, None, status, swiglu=True)
        else:
            ops.gemm_tcgen05(x, ws[i], out, None, status, n_splits=splits, scratch=scratch, partials_ok=a.partials)

    us = timed(run, nb, a.warmup, a.iters)
    byts = (N * K + M * K) * 2 + M * n_out * out.element_size()
    print(f"gemm M={M} N={N} K={K} swiglu={a.swiglu} library={a.library} splits={ops.tcgen05_splits(M, N, K) if splits is None else splits}: "
          f"{us:.2f} us, {byts / us / 1e3:.0f} GB/s, {2.0 * M * N * K / us / 1e6:.1f} TFLOP/s, status {int(status.item())}")


def case_decode_attention(a) -> None:
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    B, ctx, H, G, D = a.batch, a.context, a.heads, a.kv_heads, a.head_dim
    pages_per_seq = -(-ctx // 64)
    per_set = B * pages_per_seq
    nb = ring(per_set * G * 64 * D * 2 * 2)
    n_pages = per_set * nb
    k = torch.randn(n_pages, G, 64, D, device=DEV).to(torch.bfloat16)
    v = torch.randn(n_pages, G, 64, D, device=DEV).to(torch.bfloat16)
    q = torch.randn(B, H * D, device=DEV).to(torch.bfloat16)
    out = torch.empty_like(q)
    positions = torch.full((B,), ctx - 1, dtype=torch.int32, device=DEV)
    seq_of = torch.arange(B, dtype=torch.int32, device=DEV)
    tables = [(torch.randperm(per_set) + i * per_set).to(torch.int32).reshape(B, pages_per_seq).to(DEV) for i in range(nb)]
    n_splits = a.splits if a.splits > 0 else ops.decode_splits(B, G, H // G, ctx)
    scratch = torch.empty(max(B * H * n_splits * (D + 2), 1), dtype=torch.float32, device=DEV)
    us = timed(lambda i: ops.decode_attention(q, positions, seq_of, tables[i], k, v, out, H, D ** -0.5, 0, status, n_splits, scratch),
               nb, a.warmup, a.iters)
    byts = B * ctx * G * D * 2 * 2
    print(f"decode_attention batch={B} context={ctx} heads={H}/{G} head_dim={D} splits={n_splits}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s, status {int(status.item())}")


def case_prefill_attention(a) -> None:
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    T, H, G, D = a.tokens, a.heads, a.kv_heads, a.head_dim
    n_pages = -(-T // 64)
    k = torch.randn(n_pages, G, 64, D, device=DEV).to(torch.bfloat16)
    v = torch.randn(n_pages, G, 64, D, device=DEV).to(torch.bfloat16)
    q = torch.randn(T, H * D, device=DEV).to(torch.bfloat16)
    out = torch.empty_like(q)
    positions = torch.arange(T, dtype=torch.int32, device=DEV)
    table = torch.randperm(n_pages).to(torch.int32).reshape(1, n_pages).to(DEV)
    tt = ops.prefill_tile_tokens(H, G) if a.mma else (ops.prefill_tc_tile_tokens(H, G) if a.single else ops.prefill_twin_tile_tokens(H, G))
    tiles = torch.tensor([(0, t0, min(tt, T - t0), 0) for t0 in reversed(range(0, T, tt))], dtype=torch.int32, device=DEV)   # longest first
    fn = ops.prefill_attention if a.mma else (ops.prefill_attention_tc if a.single else ops.prefill_attention_twin)
    us = timed(lambda i: fn(q, positions, tiles, table, k, v, out, H, D ** -0.5, 0, status), 1, a.warmup, a.iters)
    flops = 4.0 * H * D * T * (T + 1) / 2
    print(f"prefill_attention ({'mma.sync' if a.mma else 'tcgen05'}) tokens={T} heads={H}/{G} head_dim={D}: {us:.2f} us, {flops / us / 1e6:.1f} TFLOP/s (causal), status {int(status.item())}")


def case_rmsnorm(a) -> None:
    rows, width, parts = a.rows, a.width, a.parts
    nb = min(ring(rows * width * 4), 16)
    xs = [torch.randn(rows, width, device=DEV) for _ in range(nb)]
    w = torch.ones(width, device=DEV)
    out = torch.empty(rows, width, dtype=torch.bfloat16, device=DEV)
    if a.bf16_delta:
        deltas = [torch.randn(rows, width, device=DEV).to(torch.bfloat16) for _ in range(nb)]
    elif parts > 0:
        deltas = [ops.Partials(torch.randn(parts, rows, width, device=DEV)) for _ in range(min(nb, 4))]
    else:
        deltas = [None]
    us = timed(lambda i: ops.rmsnorm(xs[i], w, 1e-5, out, delta=deltas[i % len(deltas)]), nb, a.warmup, a.iters)
    byts = rows * width * (4 + 2) + (rows * width * (4 + (2 if a.bf16_delta else 4 * parts)) if deltas[0] is not None else 0)
    print(f"rmsnorm rows={rows} width={width} parts={parts} bf16_delta={a.bf16_delta}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")


def case_token_shift(a) -> None:
    rows, width, reqs = a.rows, a.width, a.requests
    nb = min(ring(rows * width * 4), 16)
    hs = [torch.randn(rows, width, device=DEV) for _ in range(nb)]
    mu = torch.rand(width, device=DEV)
    out = torch.empty(rows, width, dtype=torch.bfloat16, device=DEV)
    state = torch.zeros(reqs, width, device=DEV)
    per = rows // reqs
    seq_start = torch.arange(0, reqs * per + 1, per, dtype=torch.int32, device=DEV)
    seq_of = torch.arange(reqs, dtype=torch.int32, device=DEV).repeat_interleave(per).contiguous()
    slots = torch.arange(reqs, dtype=torch.int32, device=DEV)
    n = reqs * per
    us = timed(lambda i: ops.token_shift(hs[i][:n], mu, state, seq_of, seq_start, slots, out[:n]), nb, a.warmup, a.iters)
    byts = n * width * (4 + 2)
    print(f"token_shift rows={n} width={width} requests={reqs}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")


def case_mingru(a) -> None:
    """The recurrence alone (the projections are a product of the framework's): sequential per channel for
    short portions, in pieces side by side beyond ``MINGRU_PIECES_FROM`` tokens."""
    rows, width, reqs = a.rows, a.width, a.requests
    per = rows // reqs
    n = reqs * per
    nb = min(ring(n * 3 * width * 4), 8)
    projs = [torch.randn(n, 3 * width, device=DEV) for _ in range(nb)]
    out = torch.empty(n, width, dtype=torch.bfloat16, device=DEV)
    state = torch.zeros(reqs, width, device=DEV)
    seq_start = torch.arange(0, n + 1, per, dtype=torch.int32, device=DEV)
    slots = torch.arange(reqs, dtype=torch.int32, device=DEV)
    chunks = chunk_start = None
    passes = 3
    from .parts.mingru import MINGRU_PIECES_FROM

    if per > MINGRU_PIECES_FROM:
        c = ops.mingru_chunk_tokens()
        pieces, first = [], [0]
        for r in range(reqs):
            pieces += [(r * per + t0, r * per + min(t0 + c, per)) for t0 in range(0, per, c)]
            first.append(len(pieces))
        chunks = torch.tensor(pieces, dtype=torch.int32, device=DEV)
        chunk_start = torch.tensor(first, dtype=torch.int32, device=DEV)
        passes = 5                           # z and u in the first pass, z, u and g in the last
    us = timed(lambda i: ops.mingru_scan(projs[i], state, seq_start, slots, out, chunks, chunk_start), nb, a.warmup, a.iters)
    byts = n * width * (4 * passes + 2)
    print(f"mingru rows={n} width={width} requests={reqs} pieces={'yes' if chunks is not None else 'no'}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")


def case_token_side(a) -> None:
    """The token input: for few rows the one kernel (its traffic is the two small matrices, read once per
    launch when they come from HBM); for many, the three small kernels around the two products."""
    rows, width, dim, vocab = a.rows, a.width, a.dim, 32000
    nb = max(min(ring(2 * dim * width * 2), 64), 2)
    gates = [(torch.randn(dim, width, device=DEV) * 0.02).to(torch.bfloat16) for _ in range(nb)]
    projs = [(torch.randn(width, dim, device=DEV) * 0.02).to(torch.bfloat16) for _ in range(nb)]
    table = torch.randn(vocab, dim, device=DEV).to(torch.bfloat16)
    ids = torch.randint(0, vocab, (rows,), dtype=torch.int32, device=DEV)
    norm_w = torch.ones(width, device=DEV)
    nx = min(ring(rows * width * 4), 16)
    xs = [torch.randn(rows, width, device=DEV) for _ in range(nx)]
    deltas = [torch.randn(rows, width, device=DEV) for _ in range(nx)]
    if rows < 64:
        us = timed(lambda i: ops.token_side(xs[i % nx], deltas[i % nx], 0.5, ids, table, 0, gates[i], projs[i], norm_w, 1e-6, 0.5), nb, a.warmup, a.iters)
        byts = 2 * dim * width * 2 + rows * width * 12
        print(f"token_side rows={rows} width={width} dim={dim}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")
        return
    ys = [torch.randn(rows, width, device=DEV) for _ in range(nx)]
    gl = [torch.randn(rows, dim, device=DEV) for _ in range(nx)]
    us = timed(lambda i: ops.residual_fold(xs[i], deltas[i], 0.5, copy_dtype=torch.bfloat16), nx, a.warmup, a.iters)
    print(f"side_fold rows={rows} width={width}: {us:.2f} us, {rows * width * 14 / us / 1e3:.0f} GB/s")
    us = timed(lambda i: ops.side_gate(gl[i], ids, table, 0, torch.bfloat16), nx, a.warmup, a.iters)
    print(f"side_gate rows={rows} dim={dim}: {us:.2f} us, {rows * dim * 8 / us / 1e3:.0f} GB/s")
    us = timed(lambda i: ops.side_add(xs[i], ys[i], norm_w, 1e-6, 0.5), nx, a.warmup, a.iters)
    print(f"side_add rows={rows} width={width}: {us:.2f} us, {rows * width * 12 / us / 1e3:.0f} GB/s")


def case_chunk_scan(a) -> None:
    """A recurrence with one decay per head over one request's tokens, 64 at a time (the row factors' kernel and the scan): the delta
    rule, or the matrix memory with its extra column (``--memory``)."""
    from .engine.batch import ScanChunks

    n, H, G, D, Dv = a.rows, a.heads, (a.heads if a.memory else a.kv_heads), a.dim, a.vdim
    P = Dv + 1 if a.memory else Dv
    C = 2 * G * D + H * Dv
    nb = min(ring(n * C * 4), 8)
    bufs = [torch.nn.functional.normalize(torch.randn(n, C // 4, 4, device=DEV), dim=1).view(n, C) for _ in range(nb)]
    gb = torch.rand(n, 4 * H, device=DEV) * 0.5
    gb[:, 3::4] = -gb[:, 3::4]
    gb[:, 2::4] = -gb[:, 2::4]
    state = torch.zeros(1, H * D * P, device=DEV)
    rows = torch.tensor([(t, min(t + 64, n)) for t in range(0, n, 64)], dtype=torch.int32, device=DEV)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)
    chunks = ScanChunks(rows, i32(0, rows.shape[0]), i32(0), 16, False)
    out = torch.empty(n, H * P, device=DEV)
    slots = i32(0)

    def run(i):
        x = bufs[i]
        v, k, q = x[:, :H * Dv], x[:, H * Dv:H * Dv + G * D], x[:, H * Dv + G * D:]
        ops.chunk_scan(q, k, v, gb[:, 2:], gb[:, 1:], 4, state, *((1, D) if a.memory else (P, 1)), chunks, slots, out, H, G, D, Dv, P, not a.memory)

    us = timed(run, nb, a.warmup, a.iters)
    seq = 2.0 * n * H * P * D * (2 if a.memory else 3)         # the recurrence's own multiply-adds, token by token
    print(f"chunk_scan {'memory' if a.memory else 'delta'} rows={n} heads={H}/{G} dim={D} vdim={Dv}: {us:.2f} us, {seq / us / 1e6:.2f} TFLOP/s of the recurrence itself")


def case_stream_norm(a) -> None:
    n, E, R = a.rows, a.width, a.streams
    nb = min(ring(n * E * 4 * (R + 2)), 8)
    xs = [torch.randn(n, R, E, device=DEV) for _ in range(nb)]
    ds = [torch.randn(n, E, device=DEV) for _ in range(nb)]
    gs = [torch.randn(n, E, device=DEV) for _ in range(nb)]
    w, w_in, w_out, mix = torch.ones(E, device=DEV), torch.ones(R, device=DEV), torch.ones(R, device=DEV), torch.eye(R, device=DEV)
    out = torch.empty(n, E, dtype=torch.bfloat16, device=DEV)
    us = timed(lambda i: ops.stream_norm(xs[i], 1e-6, out, w, w_in=w_in, delta=ds[i], gate=gs[i], w_out=w_out, mix=mix), nb, a.warmup, a.iters)
    byts = n * E * (8 * R + 8 + 2)
    print(f"stream_norm rows={n} width={E} streams={R}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")


def case_scaled_norm(a) -> None:
    """The seam between two parallel layers: a product (or its partial sums) and each token's experts, scaled channel by channel, into the
    stream; the norm; its rows again into the experts' tiles."""
    n, E, top = a.rows, a.width, a.top
    nb = min(ring(n * E * 4 * (a.parts + top + 1)), 8)
    xs = [torch.randn(n, E, device=DEV) for _ in range(nb)]
    ds = [torch.randn(a.parts, n, E, device=DEV) for _ in range(nb)]
    ys = [torch.randn(n * top, E, device=DEV) for _ in range(nb)]
    places = torch.randperm(n * top, device=DEV).to(torch.int32).view(n, top)
    w, s1, s2 = (torch.ones(E, device=DEV) for _ in range(3))
    out = torch.empty(n, E, dtype=torch.bfloat16, device=DEV)
    tiles = torch.empty(n * top, E, dtype=torch.bfloat16, device=DEV)

    def run(i):
        value = ops.Partials(ds[i]) if a.parts > 1 else ds[i][0]
        ops.scaled_norm(xs[i], (ops.Term(value, s1), ops.Term(ops.ExpertRows(ys[i], places, 1.0 / top), s2)), 1e-6, w, out, tiles=tiles, places=places)

    us = timed(run, nb, a.warmup, a.iters)
    byts = n * E * (8 + 4 * a.parts + 4 * top + 2 + 2 * top)
    print(f"scaled_norm rows={n} width={E} parts={a.parts} experts={top}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")


def case_rglru(a) -> None:
    """The gated linear recurrence between its projections: one token of every request (one kernel), or one request's portion
    (convolution, the gates' product, the gates and the chunks' ends, the chain, the scan)."""
    C, P, taps = a.width, a.part, 4
    B = C // P
    n = a.requests if a.requests > 1 else a.rows
    nb = min(ring(n * C * 8), 8)
    bufs = [torch.randn(n, 2 * C, device=DEV) for _ in range(nb)]
    conv_w, conv_b = torch.randn(taps, C, device=DEV), torch.zeros(C, device=DEV)
    ra, ri = ((torch.randn(B, P, P, device=DEV) / P ** 0.5).to(torch.bfloat16) for _ in range(2))
    rb, sp8 = torch.zeros(C, device=DEV), torch.full((C,), 0.2, device=DEV)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    slots = i32(list(range(a.requests)))
    state = torch.zeros(a.requests, ops.rglru_state_floats(C, taps), device=DEV)
    if a.requests > 1:
        pos = i32([9] * n)
        us = timed(lambda i: ops.rglru_step(bufs[i], conv_w, conv_b, state, slots, pos, ra, rb, ri, rb, sp8), nb, a.warmup, a.iters)
        byts = 4 * B * P * P + n * C * (8 + 8 + 4 * taps + 2)
        print(f"rglru step requests={n} channels={C} parts of {P}: {us:.2f} us, {byts / us / 1e3:.0f} GB/s")
        return
    rows, tile = ops.rglru_pieces_rows(n)
    w = ops.rglru_pieces_matrices(ra, ri)
    tiles = i32([v for b in range(B) for _ in range(rows // tile) for v in (b, 0, 0)] + [B * (rows // tile)])
    status, step = torch.zeros(1, dtype=torch.int32, device=DEV), ops.rglru_chunk_tokens()
    chunks = i32([(t, min(t + step, n)) for t in range(0, n, step)])
    first, seq, start, pos = i32([0, chunks.shape[0]]), i32([0] * n), i32([0, n]), i32(list(range(n)))
    out = torch.empty(n, C, dtype=torch.bfloat16, device=DEV)
    conv = lambda i: ops.rglru_conv(bufs[i], conv_w, conv_b, state, seq, start, slots, pos, part=P)
    u = conv(0)
    gates = lambda i: ops.rglru_gates_pieces(u, n, w, tiles, rb, rb, sp8, status, chunks=chunks)
    ab, ends = gates(0)
    scan = lambda i: ops.rglru_scan(ab, bufs[i], state, start, slots, out, chunks, first, ends=ends.clone())
    t_conv, t_gates, t_scan = (timed(f, nb, a.warmup, a.iters) for f in (conv, gates, scan))
    print(f"rglru rows={n} channels={C} parts of {P}: convolution {t_conv:.2f} us ({n * C * 10 / t_conv / 1e3:.0f} GB/s), gates {t_gates:.2f} us "
          f"({4.0 * n * C * P / t_gates / 1e6:.0f} TFLOP/s of float32 products, three times that on the tensor cores), scan {t_scan:.2f} us "
          f"({n * C * 14 / t_scan / 1e3:.0f} GB/s)")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m lgml_b200.kernel_bench")
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--iters", type=int, default=50)
    ap.add_argument("--no-graph", action="store_true", help="launch the timed calls one by one from the host")
    sub = ap.add_subparsers(dest="case", required=True)
    g = sub.add_parser("gemm")
    g.add_argument("--m", type=int, default=8)
    g.add_argument("--n", type=int, default=28672)
    g.add_argument("--k", type=int, default=4096)
    g.add_argument("--swiglu", action="store_true")
    g.add_argument("--f32-out", action="store_true")
    g.add_argument("--library", action="store_true", help="time the library product on the same operands instead")
    g.add_argument("--partials", action="store_true", help="leave the K splits' partial sums to the next kernel")
    g.add_argument("--splits", type=int, default=-1)
    d = sub.add_parser("decode_attention")
    d.add_argument("--batch", type=int, default=8)
    d.add_argument("--context", type=int, default=2176)
    d.add_argument("--heads", type=int, default=32)
    d.add_argument("--kv-heads", type=int, default=8)
    d.add_argument("--head-dim", type=int, default=128)
    d.add_argument("--splits", type=int, default=0)
    p = sub.add_parser("prefill_attention")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--heads", type=int, default=32)
    p.add_argument("--kv-heads", type=int, default=8)
    p.add_argument("--head-dim", type=int, default=128)
    p.add_argument("--mma", action="store_true", help="the mma.sync kernel instead of the tcgen05 one")
    p.add_argument("--single", action="store_true", help="the tcgen05 kernel with one tile per CTA and one page per step")
    r = sub.add_parser("rmsnorm")
    r.add_argument("--rows", type=int, default=8)
    r.add_argument("--width", type=int, default=4096)
    r.add_argument("--parts", type=int, default=9)
    r.add_argument("--bf16-delta", action="store_true", help="add a bfloat16 delta (a product's output) instead of float32 partial sums")
    for name in ("token_shift", "mingru", "token_side"):
        t = sub.add_parser(name)
        t.add_argument("--rows", type=int, default=2048)
        t.add_argument("--width", type=int, default=4096)
        t.add_argument("--requests", type=int, default=1)
        t.add_argument("--dim", type=int, default=64)
    c = sub.add_parser("chunk_scan")
    for name, size in (("rows", 2048), ("heads", 16), ("kv-heads", 8), ("dim", 128), ("vdim", 128)):
        c.add_argument("--" + name, type=int, default=size)
    c.add_argument("--memory", action="store_true", help="the matrix memory instead of the delta rule")
    c = sub.add_parser("stream_norm")
    for name, size in (("rows", 2048), ("width", 4096), ("streams", 2)):
        c.add_argument("--" + name, type=int, default=size)
    c = sub.add_parser("scaled_norm")
    for name, size in (("rows", 2048), ("width", 4096), ("top", 2), ("parts", 1)):
        c.add_argument("--" + name, type=int, default=size)
    c = sub.add_parser("rglru")
    for name, size in (("rows", 2048), ("width", 4096), ("part", 256), ("requests", 1)):
        c.add_argument("--" + name, type=int, default=size)
    a = ap.parse_args(argv)
    global USE_GRAPH
    USE_GRAPH = not a.no_graph
    if not torch.cuda.is_available():
        print("kernel_bench needs a CUDA device", file=sys.stderr)
        return 1
    {"gemm": case_gemm, "decode_attention": case_decode_attention, "prefill_attention": case_prefill_attention, "rmsnorm": case_rmsnorm,
     "token_shift": case_token_shift, "mingru": case_mingru, "token_side": case_token_side, "chunk_scan": case_chunk_scan,
     "stream_norm": case_stream_norm, "scaled_norm": case_scaled_norm, "rglru": case_rglru}[a.case](a)
    return 0


if __name__ == "__main__":
    sys.exit(main())
