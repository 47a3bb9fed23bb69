"""Tedisun in the engine against the plain implementation: every mechanism alone, then whole models under every way of
cutting the work.

The models are small and differ from each other in every size and option (one to four streams, one to eight heads of 5 to
128 entries, values shorter and longer than keys, windows of 1 to 70 tokens and none, 0 to 67 kept first tokens, one to 37
experts with none to four that return their input, convolutions of 1 to 8 taps, layers without a feed-forward, a model
without any page).  Where random numbers would hide a fault, the inputs are made so that it shows: single keys stand far
out and lie just inside and just outside the window and the kept tokens, sinks outweigh the keys, recurrences decay so
slowly that what hundreds of tokens back wrote still decides the output.
"""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import helpers as H
from tests import tedisun_helpers as L
from tests.plain import tedisun_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": dict(atol=3e-5, rtol=2e-4), "bfloat16": dict(atol=3e-2, rtol=0.1)}


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def batch_of(lens):
    """(request index of every token, first token row of every request) of a step with these portions."""
    return i32([r for r, n in enumerate(lens) for _ in range(n)]), i32(np.concatenate([[0], np.cumsum(lens)]))


def chunks_of(lens, longer_than=16):
    """The description of a step's long requests for the chunked recurrences."""
    from lgml_b200.engine.batch import ScanChunks

    rows, first, reqs, start = [], [0], [], 0
    for r, n in enumerate(lens):
        if n > longer_than:
            rows += [(start + t, start + min(t + 64, n)) for t in range(0, n, 64)]
            first.append(len(rows))
            reqs.append(r)
        start += n
    if not reqs:
        return None
    return ScanChunks(i32(np.array(rows).reshape(-1)).view(-1, 2), i32(first), i32(reqs), longer_than, len(reqs) < len(lens))


def portions_of(total, cuts):
    out, a, i = [], 0, 0
    while a < total:
        b = min(total, a + cuts[i % len(cuts)])
        out.append((a, b))
        a, i = b, i + 1
    return out


def close_to(got, want, tol, what=""):
    err = np.abs(np.asarray(got, dtype=np.float64) - want)
    assert err.max() < tol * (1 + np.abs(want).max()), f"{what}: {err.max():.3g} at {np.unravel_index(int(err.argmax()), err.shape)}"


# ---------------------------------------------------------------------------------------------
# streams
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("R,E,n", [(1, 36, 5), (2, 64, 7), (2, 2048, 300), (3, 37, 9), (3, 320, 4), (4, 1032, 6), (5, 48, 3), (8, 33, 2)])
def test_streams_gate_and_norm_in_one_kernel(out_dtype, R, E, n):
    from lgml_b200 import ops

    rng = np.random.default_rng(R * 1000 + E)
    eps, tol = 1e-5, 1e-5 if out_dtype == torch.float32 else 1e-2
    start, d, gate = rng.normal(size=(n, E)), rng.normal(size=(n, E)), rng.normal(size=(n, E + 8)) * 2
    w, w_in, w_out, mix = rng.normal(size=E) * 0.3 + 1, rng.normal(size=R), rng.normal(size=R), rng.normal(size=(R, R))
    norm = lambda u: P.rms_unit(u, eps) * w
    new = lambda m: torch.empty((m, E), dtype=out_dtype, device=DEV)
    # the streams start as scaled rows
    x = torch.full((n, R, E), float("nan"), device=DEV)
    out = ops.stream_norm(x, eps, new(n), f32(w), w_in=f32(w_in), start=f32(start), start_scale=1.7)
    X = np.repeat((start * 1.7)[:, None], R, axis=1)
    close_to(x.cpu(), X, 1e-6, "start")
    close_to(out.float().cpu(), norm(P.streams_read(X, w_in)), tol, "start")
    # a gated result (a column slice of a wider product), all streams from the old ones
    X = rng.normal(size=(n, R, E))
    x = f32(X)
    out = ops.stream_norm(x, eps, new(n), f32(w), w_in=f32(w_in), delta=f32(d), gate=f32(gate)[:, 4:4 + E], w_out=f32(w_out), mix=f32(mix))
    X1 = P.streams_write(X, d * P.sigmoid(gate[:, 4:4 + E]), w_out, mix)
    close_to(x.cpu(), X1, 1e-5, "update")
    close_to(out.float().cpu(), norm(P.streams_read(X1, w_in)), tol, "update")
    # a result as partial sums with a bias, no gate, chosen rows, the plain sum of the streams: x stays as it was
    parts, bias = rng.normal(size=(11, n, E)), rng.normal(size=E)
    x, rows = f32(X), [n - 1, 0, n - 1]
    out = ops.stream_norm(x, eps, new(3), f32(w), delta=ops.Partials(f32(parts), f32(bias)), w_out=f32(w_out), mix=f32(mix), rows=i32(rows))
    assert torch.equal(x, f32(X))
    X2 = P.streams_write(X, parts.sum(0) + bias, w_out, mix)
    close_to(out.float().cpu(), norm(X2.sum(axis=1))[rows], tol, "rows")
    # nothing pending; and a result without a norm behind it
    out = ops.stream_norm(x, eps, new(n), f32(w), w_in=f32(w_in))
    close_to(out.float().cpu(), norm(P.streams_read(X, w_in)), tol, "nothing pending")
    assert ops.stream_norm(x, eps, None, None, delta=f32(d), w_out=f32(w_out), mix=f32(mix)) is None
    close_to(x.cpu(), P.streams_write(X, d, w_out, mix), 1e-5, "no norm")


def test_streams_refuse_what_does_not_fit():
    from lgml_b200 import ops

    x, w = torch.zeros((2, 2, 8), device=DEV), torch.ones(8, device=DEV)
    out = torch.empty((2, 8), device=DEV)
    with pytest.raises(ops.KernelError):
        ops.stream_norm(x, 1e-5, out, w, delta=torch.zeros((2, 8), device=DEV))             # no mix matrix
    with pytest.raises(ops.KernelError):
        ops.stream_norm(x, 1e-5, out, w, w_in=torch.zeros(3, device=DEV))
    with pytest.raises(ops.KernelError):
        ops.stream_norm(torch.zeros((2, 9, 8), device=DEV), 1e-5, out, w)


# ---------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------

HEADS = [(4, 2, 64, 64), (2, 1, 128, 128), (6, 2, 32, 24), (3, 3, 48, 80), (2, 2, 10, 7), (1, 1, 160, 96)]
MASKS = [(40, 5), (64, 64), (1, 3), (65, 70), (129, 1), (63, 0), (0, 0), (120, 130)]
# the 32-bit form is one kernel: a mask per head size
WINDOWS = [(torch.bfloat16, h, m) for h in HEADS for m in MASKS] + [(torch.float32, h, m) for h, m in zip(HEADS, (MASKS[0], MASKS[2], MASKS[3], MASKS[6], MASKS[1], MASKS[7]))]


@pytest.mark.parametrize("dtype,heads,mask", WINDOWS)
def test_window_with_kept_tokens_and_sink_in_every_kernel_form(dtype, heads, mask):
    """Norm per head, turn, cache write and attention.  Every query points the same way before the turn, and so do a few keys
    (the rest are random): those stand far out for all queries, so a query just inside and one just outside the window of
    such a key differ by most of its value."""
    from lgml_b200 import ops
    from lgml_b200.engine.runtime import Runtime
    from lgml_b200.engine.batch import CacheView
    from lgml_b200.models.tedisun import rotation_of

    (H_, G, D, Dv), (size, keep) = heads, mask
    rng = np.random.default_rng(H_ * 100 + D + size * 7 + keep)
    n, eps = 290, 1e-5
    rot = {"base": 5000.0, "dims": 2 * (D // 8), "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}}
    scale = 9.0 / D
    base = rng.normal(size=(H_, D))
    q = base[None] + 0.1 * rng.normal(size=(n, H_, D))
    k, v = rng.normal(size=(n, G, D)), rng.normal(size=(n, G, Dv)) * 2
    loud = sorted({0, max(keep - 1, 0), keep, 20, 63, 64, 100, 127, 150, 192})
    for g in range(G):
        k[loud, g] = base[g * (H_ // G)] + 0.05 * rng.normal(size=(len(loud), D))
    qw, kw, sink, v_scale = rng.normal(size=D) * 0.1 + 1, rng.normal(size=D) * 0.1 + 1, rng.normal(size=H_) * 0.3 + 7.5, 1.3
    freq = P.rms_unit
    qn, kn = freq(q, eps) * qw, freq(k, eps) * kw
    turn = lambda x: P.rotate_halves(x, rot, np.arange(n))
    plain = lambda **o: P.sink_window_attention(turn(qn), turn(kn), v * v_scale, scale, o.get("sink", sink), o.get("size", size), o.get("keep", keep))
    want = plain()
    for other in ([dict(size=size + 1), dict(size=size - 1)] if size > 1 else []) + ([dict(keep=keep + 1), dict(keep=keep - 1)] if size and keep else []) \
            + [dict(sink=sink - 50)]:
        assert np.abs(plain(**other) - want).max() > 0.2, f"{other} would not show"
    n_pages, page = 9, 64
    rt = Runtime(DEV, dtype)
    position = rotation_of(D, rot)
    position.bind("", {}, rt)
    pages = [7, 2, 5, 0, 3]
    table = i32(pages).view(1, -1)
    proj = f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], axis=1))
    for form, cuts in (("auto", [290]), ("auto", [7, 2, 1, 60, 3, 129]), ("split", [30, 1, 5])):
        k_pages = torch.full((n_pages, G, page, D), 60.0, dtype=dtype, device=DEV)       # what an earlier request may have left
        v_pages = torch.full((n_pages, G, page, Dv), 60.0, dtype=dtype, device=DEV)
        got = np.zeros_like(want)
        for a, b in portions_of(n, cuts):
            m = b - a
            pos, seq = i32(range(a, b)), i32([0] * m)
            qd = ops.norm_rope_store(proj[a:b], f32(qw), f32(kw), eps, pos, seq, table, position.inv_freq, position.n_rot, k_pages, v_pages, H_, rt.status,
                                     v_scale=v_scale)
            out = torch.zeros((m, H_ * Dv + 8), dtype=dtype, device=DEV)[:, :H_ * Dv]

            class Batch:
                positions, seq_of_token, max_q_len, max_kv_len = pos, seq, m, b

                @staticmethod
                def attention_tiles(tt):
                    return torch.tensor([[0, t0, min(tt, m - t0), 0] for t0 in range(0, m, tt)], dtype=torch.int32, device=DEV)

            view = CacheView(k=k_pages, v=v_pages, block_table=table)
            if form == "split" and dtype == torch.bfloat16:
                ops.sink_decode(qd, pos, seq, table, k_pages, v_pages, out, H_, scale, size, rt.status, 3 if b > 128 else 1, sinks=f32(sink), keep_first=keep)
            else:
                rt.sink_attention(qd, Batch, view, out, H_, scale, size, None, f32(sink), None, keep_first=keep)
            got[a:b] = out.float().cpu().numpy().reshape(m, H_, Dv)
        rt.check_status()
        tol = 3e-5 if dtype == torch.float32 else 4e-2
        err = np.abs(got - want).max(axis=(1, 2))
        assert err.max() < tol * (1 + np.abs(want).max()), f"{form} {cuts}: token {int(err.argmax())}: {err.max():.3g}"


@pytest.mark.parametrize("D,Dv,n_rot", [(16, 8, 16), (10, 7, 4), (64, 64, 0), (128, 256, 32)])
def test_norm_turn_and_store_at_far_positions_and_without_norm(D, Dv, n_rot):
    """Positions of tens of thousands turn as exactly as the first ones; without norm weights q and k only turn; without
    ``write_kv`` the cache stays untouched."""
    from lgml_b200 import ops
    from lgml_b200.engine.runtime import Runtime
    from lgml_b200.models.tedisun import rotation_of

    rng = np.random.default_rng(D)
    H_, G, n = 3, 1, 6
    rt = Runtime(DEV, torch.float32)
    rot = {"base": 900.0, "dims": max(n_rot, 2)}
    position = rotation_of(D, rot)
    position.bind("", {}, rt)
    pos = np.array([0, 1, 63, 20000, 65535, 70000])
    table = torch.full((1, 1100), -1, dtype=torch.int32, device=DEV)
    for p in pos:
        table[0, p // 64] = int(p // 64) % 5
    q, k, v = rng.normal(size=(n, H_, D)), rng.normal(size=(n, G, D)), rng.normal(size=(n, G, Dv))
    proj = f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], axis=1))
    kp, vp = torch.full((5, G, 64, D), 9.0, device=DEV), torch.full((5, G, 64, Dv), 9.0, device=DEV)
    w = rng.normal(size=D)
    for write in (False, True):
        for qw in (w, None):
            qd = ops.norm_rope_store(proj, f32(qw) if qw is not None else None, None, 1e-5, i32(pos), i32([0] * n), table, position.inv_freq, n_rot, kp, vp, H_,
                                     rt.status, write_kv=write)
            qn = q if qw is None else P.rms_unit(q, 1e-5) * qw
            want = P.rotate_halves(qn, rot, pos) if n_rot else qn
            close_to(qd.cpu().numpy().reshape(n, H_, D), want, 2e-6, "q")
            if not write:
                assert bool((kp == 9.0).all()) and bool((vp == 9.0).all())
    want_k = P.rotate_halves(k, rot, pos) if n_rot else k
    for i, p in enumerate(pos):
        close_to(kp[(p // 64) % 5, 0, p % 64].cpu(), want_k[i, 0], 2e-6, "k")
        close_to(vp[(p // 64) % 5, 0, p % 64].cpu(), v[i, 0], 1e-6, "v")
    rt.check_status()
    table[0, 0] = -1            # a position without a page: flagged, not written
    ops.norm_rope_store(proj, None, None, 1e-5, i32(pos), i32([0] * n), table, position.inv_freq, n_rot, kp, vp, H_, rt.status)
    with pytest.raises(Exception):
        rt.check_status()


# ---------------------------------------------------------------------------------------------
# recurrences
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("H_,G,D,Dv", [(4, 2, 16, 24), (3, 1, 10, 7), (2, 2, 64, 128), (6, 3, 128, 64), (1, 1, 100, 33), (2, 1, 200, 16)])
def test_delta_rule_with_one_decay_per_head_in_pieces(H_, G, D, Dv):
    """A head that hardly forgets beside one that forgets at once; a key of the first tokens asked for at the end.  One portion,
    portions down to two tokens, single tokens, two requests side by side in slots that are used again."""
    from lgml_b200 import ops

    rng = np.random.default_rng(D * 10 + H_)
    n = 330
    off = -(-(H_ * D * Dv) // 4) * 4
    C = 2 * G * D + H_ * Dv
    raw = rng.normal(size=(n, C))
    raw[n - 1, :G * D] = raw[2, G * D:2 * G * D]              # the last query is an early key
    raw[n - 40, :G * D] = raw[n - 41, G * D:2 * G * D]
    a, b = rng.normal(size=(n, H_)), rng.normal(size=(n, H_)) + 1.0
    a_log, dt_bias = np.linspace(-9.0, 1.0, H_), rng.normal(size=H_) * 0.2
    rep = np.arange(H_) // (H_ // G)
    q = P.unit(raw[:, :G * D].reshape(n, G, D))[:, rep] * D ** -0.5
    k = P.unit(raw[:, G * D:2 * G * D].reshape(n, G, D))[:, rep]
    g = np.exp(-np.exp(a_log) * P.softplus(a + dt_bias))
    want = P.delta_scan(q, k, raw[:, 2 * G * D:].reshape(n, H_, Dv), P.sigmoid(b), g)
    ab = f32(np.concatenate([a, b], axis=1))
    state = torch.zeros((3, off + 8), device=DEV)
    for chunked, cuts in [(f, c) for f in (False, True) for c in ([330], [64, 2, 130, 3], [1, 2, 70], [33, 31, 65])]:
        state.zero_()
        other = 0
        got = np.zeros_like(want)
        for i, (s, e) in enumerate(portions_of(n, cuts)):
            lens, rows, slots = [e - s], raw[s:e], [1]
            gates = ab[s:e]
            if i % 2 == 0:                                    # another request's tokens ahead of these in the same step
                m = 5 + i % 3
                lens, rows, slots = [m, e - s], np.concatenate([raw[other % 200:other % 200 + m], rows]), [0, 1]
                gates = torch.cat([ab[:m], gates])
                other += m
            _, starts = batch_of(lens)
            qkv = f32(rows)
            gb = ops.delta_head_prepare(qkv, gates[:, :H_], gates[:, H_:], f32(a_log), f32(dt_bias), H_, G, D)
            o = ops.delta_scan(qkv, gb, state, starts, i32(slots), H_, G, D, Dv, chunks=chunks_of(lens) if chunked else None)
            got[s:e] = o[-(e - s):].cpu().numpy().reshape(-1, H_, Dv)
        close_to(got, want, 2e-5, f"{cuts} {'chunks' if chunked else 'token by token'}")
        assert bool((state[:, off:] == 0).all()) and bool((state[2] == 0).all())


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_output_norm_with_the_silu_gate(out_dtype):
    from lgml_b200 import ops

    rng = np.random.default_rng(4)
    n, H_, Dv = 9, 3, 36
    o, w, gate = rng.normal(size=(n, H_ * Dv)), rng.normal(size=Dv), rng.normal(size=(n, H_ * Dv + 5)) * 2
    for act, fn in (("silu", P.silu), ("sigmoid", P.sigmoid)):
        y = ops.delta_output(f32(o), f32(w), f32(gate)[:, 3:3 + H_ * Dv], 1e-5, out_dtype, H_, act=act)
        want = (P.rms_unit(o.reshape(n, H_, Dv), 1e-5) * w * fn(gate[:, 3:3 + H_ * Dv]).reshape(n, H_, Dv)).reshape(n, -1)
        close_to(y.float().cpu(), want, 1e-5 if out_dtype == torch.float32 else 1e-2, act)


@pytest.mark.parametrize("H_,D,Dv", [(2, 16, 24), (1, 5, 9), (3, 64, 64), (2, 128, 130), (4, 40, 257), (4, 33, 7), (1, 300, 20)])
def test_matrix_memory_in_portions_pieces_and_single_tokens(H_, D, Dv):
    """Gates of both signs far into their cap; a head whose input gates are so low that exp(-m) decides the denominator for long;
    a head that never forgets, asked at the end for what the first tokens wrote."""
    from lgml_b200 import ops

    rng = np.random.default_rng(D * 10 + H_)
    n, cap = 400, 7.0
    q, k, v = rng.normal(size=(n, H_, D)), rng.normal(size=(n, H_, D)), rng.normal(size=(n, H_, Dv))
    zi, zf = rng.normal(size=(n, H_)) * 6, rng.normal(size=(n, H_)) * 2 + 4
    zi[:, 0] -= 30.0 * (np.arange(n) < 100)
    zf[:, -1] += 40.0
    q[n - 1, -1], zi[3, -1] = k[3, -1] * 2, 30.0
    i, f = P.soft_capped(zi, cap), P.log_sigmoid(P.soft_capped(zf, cap))
    o = P.matrix_memory_scan(q * D ** -0.5, k, v, i, f)
    w, gate = rng.normal(size=H_ * Dv), rng.normal(size=(n, H_ * Dv))
    want = P.rms_unit(o, 1e-6).reshape(n, -1) * w * P.sigmoid(gate)
    # m from 0, not from minus infinity: the first token of head 0 shows it
    assert np.abs(o[0, 0] * (np.exp(-max(f[0, 0], i[0, 0])) + 1e-6) - np.exp(i[0, 0] - max(f[0, 0], i[0, 0])) * v[0, 0] * (q[0, 0] @ k[0, 0]) * D ** -0.5).max() < 1e-9
    wide = H_ * (Dv + 2 * D)
    proj = f32(np.concatenate([v.reshape(n, -1), k.reshape(n, -1), q.reshape(n, -1), zi, zf, np.zeros((n, -(wide + 2 * H_) % 4))], axis=1))
    m_off = H_ * (Dv + 1) * D
    for chunked, cuts in [(f, c) for f in (False, True) for c in ([400], [150, 2, 248], [1, 2, 3, 90], [64, 65])]:
        state = torch.full((3, m_off + H_ + 3), 5.0, device=DEV)
        state[[0, 2], :m_off + H_] = 0.0
        got = np.zeros_like(want)
        y_all = []
        for s, e in portions_of(n, cuts):
            m = e - s
            lens, slots = [m, 4], [2, 0]                     # a second request of four tokens in every step
            rows = torch.cat([proj[s:e], proj[:4]])
            _, starts = batch_of(lens)
            gates = ops.memory_gates(rows[:, wide:wide + H_], rows[:, wide + H_:wide + 2 * H_], cap, state[:, m_off:m_off + H_], starts, i32(slots))
            pieces = None
            if m > 128:
                cutp = [(t, min(t + 64, m)) for t in range(0, m, 64)] + [(m, m + 4)]
                pieces = (i32(np.array(cutp).reshape(-1)).view(-1, 2), i32([0, len(cutp) - 1, len(cutp)]))
            y = ops.memory_scan(rows[:, :wide], gates, state, starts, i32(slots), H_, D, Dv, pieces=pieces, chunks=chunks_of(lens) if chunked else None)
            out = torch.empty((m + 4, H_ * Dv), device=DEV)
            ops.memory_output(y, gates, D ** -0.5, f32(w), torch.cat([f32(gate[s:e]), f32(gate[:4])]), 1e-6, out)
            got[s:e] = out[:m].cpu().numpy()
        # (an output of all but nothing over its root mean square magnifies rounding: those rows are held to their size before it)
        size = np.sqrt((o ** 2).mean(axis=-1))
        err = np.abs(got - want).reshape(n, H_, Dv).max(axis=-1)
        bound = 3e-4 * (1 + np.abs(want).max()) * np.maximum(1.0, 0.02 / size)
        assert (err < bound).all(), f"{cuts} {chunked}: {np.unravel_index(int((err / bound).argmax()), err.shape)} {(err / bound).max():.3g}"
        assert bool((state[1] == 5.0).all()) and bool((state[:, m_off + H_:] == 5.0).all())


def test_gates_of_a_long_portion_are_those_of_single_tokens():
    from lgml_b200 import ops

    rng = np.random.default_rng(8)
    n, H_, cap = 1000, 3, 12.0
    z = f32(rng.normal(size=(n, 2 * H_)) * 5 + np.repeat([0.0, 3.0], H_))
    one, many = torch.zeros((1, H_), device=DEV), torch.zeros((1, H_), device=DEV)
    whole = ops.memory_gates(z[:, :H_], z[:, H_:], cap, many, i32([0, n]), i32([0]))
    steps = torch.cat([ops.memory_gates(z[t:t + 1, :H_], z[t:t + 1, H_:], cap, one, i32([0, 1]), i32([0])) for t in range(n)])
    assert float((whole - steps).abs().max()) < 1e-5 * float(steps.abs().max()) and float((one - many).abs().max()) < 1e-5
    zi, zf = z[:, :H_].double().cpu().numpy(), z[:, H_:].double().cpu().numpy()
    i, f, m = P.soft_capped(zi, cap), P.log_sigmoid(P.soft_capped(zf, cap)), np.zeros(H_)
    for t in range(n):
        before, m = m, np.maximum(f[t] + m, i[t])
        close_to(whole[t].cpu(), np.concatenate([np.exp(f[t] + before - m), np.exp(i[t] - m), np.exp(-m), f[t] + before - m]), 2e-5, str(t))


# ---------------------------------------------------------------------------------------------
# experts
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("X,I,top,E,F,n", [(5, 2, 2, 64, 48, 3), (16, 3, 4, 128, 64, 200), (1, 0, 1, 24, 16, 5), (3, 5, 8, 64, 40, 60), (40, 1, 3, 72, 520, 90),
                                           (6, 2, 2, 35, 21, 11), (2, 30, 3, 64, 32, 150)])
def test_router_and_experts_some_of_which_return_their_input(dtype, X, I, top, E, F, n):
    from lgml_b200 import ops
    from lgml_b200.engine.runtime import Runtime

    rng = np.random.default_rng(X * 100 + E)
    bf = lambda a: torch.tensor(a, dtype=torch.float32).to(torch.bfloat16).double().numpy()
    W = {"p.router": bf(rng.normal(size=(X + I, E)) * 2 / E ** 0.5), "p.correction": rng.permutation(X + I) * 0.05}
    for e in range(X):
        for name, shape, fan in (("gate", (F, E), E), ("up", (F, E), E), ("down", (E, F), F)):
            W[f"p.e{e}.{name}"] = bf(rng.normal(size=shape) * 1.5 / fan ** 0.5)
    h = bf(rng.normal(size=(n, E)))
    rt = Runtime(DEV, dtype)
    dev = lambda a: torch.tensor(a, dtype=dtype, device=DEV)
    ids, wts = P.route(h, W, "p", top)
    got = ops.moe_router(dev(h), f32(W["p.router"]), f32(W["p.correction"]), top, "softmax_all", n_identity=I)
    z = torch.zeros((n, X + I + 3), device=DEV)
    z[:, 1:1 + X + I] = f32(h @ W["p.router"].T)
    ready = ops.moe_select(z[:, 1:1 + X + I], f32(W["p.correction"]), top, n_identity=I)       # the same choice from ready logits
    margin = P.choice_margin(h, W, "p", top) > 1e-5
    for a, b in zip(got, ready):
        assert np.allclose(np.sort(a.cpu().numpy().reshape(n, -1)[margin], axis=1), np.sort(b.cpu().numpy().reshape(n, -1)[margin], axis=1), atol=1e-5)
    want_ids = np.where(ids >= X, -1, ids)
    # (the order of the chosen is by falling choice score, but two of them may lie as close as rounding)
    assert np.array_equal(np.sort(got[0].cpu().numpy()[margin], axis=1), np.sort(want_ids[margin], axis=1))
    assert np.allclose(np.sort(got[1].cpu().numpy()[margin], axis=1), np.sort(wts[margin], axis=1), atol=1e-5)
    if I:
        assert np.allclose(got[2].cpu().numpy()[margin], np.where(ids >= X, wts, 0.0).sum(axis=1)[margin], atol=1e-5)
    w_gu = torch.stack([torch.stack([dev(W[f"p.e{e}.gate"]), dev(W[f"p.e{e}.up"])], dim=1).reshape(2 * F, E) for e in range(X)]).contiguous()
    wd = torch.stack([dev(W[f"p.e{e}.down"]) for e in range(X)]).contiguous()
    want = P.experts(h, W, "p", {"router": {"experts": X, "identity": I, "top": top}})
    also = dict(also=dev(h), also_w=got[2]) if I else {}
    forms = {"rows": lambda: ops.moe_experts_rows(dev(h), got[0], got[1], w_gu, wd, **also), "chosen": lambda: rt.moe_experts(dev(h), got[0], got[1], w_gu, wd, **also)}
    if dtype == torch.bfloat16 and E % 8 == 0 and F % 8 == 0:
        forms["grouped"] = lambda: ops.moe_experts_tcgen05(dev(h), got[0], got[1], w_gu, wd, rt.status, **also)
    for name, run in forms.items():
        y = run().float().cpu().numpy()
        rt.check_status()
        close_to(y[margin], want[margin], 2e-5 if dtype == torch.float32 else 2e-2, name)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_slot_an_identity_expert(dtype):
    """No token chooses an expert with matrices: the output is the input times the chosen scores' sum, in every form."""
    from lgml_b200 import ops
    from lgml_b200.engine.runtime import Runtime

    rng = np.random.default_rng(3)
    n, E, F, X, I, top = 40, 64, 32, 4, 3, 2
    rt = Runtime(DEV, dtype)
    h = torch.tensor(rng.normal(size=(n, E)), dtype=dtype, device=DEV)
    corr = f32([0.0] * X + [5.0] * I)
    ids, wts, own = ops.moe_router(h, f32(rng.normal(size=(X + I, E)) * 0.1), corr, top, "softmax_all", n_identity=I)
    assert bool((ids == -1).all())
    w_gu, wd = torch.full((X, 2 * F, E), float("nan"), dtype=dtype, device=DEV), torch.full((X, E, F), float("nan"), dtype=dtype, device=DEV)
    want = h.float() * wts.sum(dim=1, keepdim=True)
    runs = [ops.moe_experts_rows(h, ids, wts, w_gu, wd, also=h, also_w=own)]
    if dtype == torch.bfloat16:
        runs.append(ops.moe_experts_tcgen05(h, ids, wts, w_gu, wd, rt.status, also=h, also_w=own))
    for y in runs:
        assert float((y - want).abs().max()) < 1e-5
    rt.check_status()


# ---------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------

def make_runner(folder, dtype, n_pages, slots=4, **kw):
    from lgml_b200.engine.engine import parse_dtype
    from lgml_b200.engine.runner import ModelRunner

    return ModelRunner.from_folder(folder, parse_dtype(dtype), DEV, n_pages=n_pages, max_slots=slots, max_step_tokens=n_pages * 64, **kw)


_clear = {}


def sequences(cfg, weights, dtype, lens, seed=50):
    """Token ids of these lengths; for bfloat16 such that no router decides by a close call."""
    if dtype == "float32":
        return {f"r{i}": H.random_ids(n, cfg["vocab"], seed + i) for i, n in enumerate(lens)}
    out = {}
    for i, n in enumerate(lens):
        key = (id(weights), n, seed + i)
        if key not in _clear:
            _clear[key] = L.clear_ids(cfg, weights, n, seed + i)
        out[f"r{i}"] = _clear[key]
    return out


# one mechanism at a time: a model of one or two layers that has as little else as the design allows
SMALL = dict(size=9, keep_first=2)
ALONE = {
    "delta": L.config(53, 40, 1, [L.delta(2, 1, 12, 8, 3)]),
    "attention_far": L.config(53, 40, 1, [L.parallel(L.left(2, 2, 16, 16, 0.4, base=9000.0, dims=6, scaling=(16.0, 1.0, 8.0, 48)), L.right(1, 4, 4, 5.0), (1.0, 0.0))]),
    "window_and_first_tokens": L.config(53, 40, 1, [L.parallel(L.left(2, 1, 16, 8, 0.4, dims=4, **SMALL), L.right(1, 4, 4, 5.0), (1.2, 0.0))]),
    "memory": L.config(53, 40, 1, [L.parallel(L.left(1, 1, 8, 8, 0.3, dims=4, size=1), L.right(3, 24, 40, 10.0), (0.0, 1.4))]),
    "five_streams": L.config(53, 40, 5, [L.delta(1, 1, 8, 8, 2, L.moe(24, 3, 1)), L.delta(2, 2, 8, 4, 1)], scale=2.0),
    "experts": L.config(53, 40, 1, [L.delta(1, 1, 8, 8, 1, L.moe(56, 9, 3, 2))], softcap=3.0),
    "identity_only_sometimes": L.config(53, 40, 2, [L.delta(1, 1, 8, 8, 2, L.moe(16, 1, 2, 6))]),
    "odd_width": L.config(51, 35, 3, [L.parallel(L.left(3, 1, 10, 7, 0.3, dims=6, size=20, keep_first=1), L.right(3, 5, 9, 4.0), (0.9, 1.1), L.moe(19, 3, 2, 1)),
                                      L.delta(3, 3, 7, 5, 4, L.moe(33, 2, 1, 1))], scale=1.5, softcap=10.0),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_at_a_time(name, tmp_path):
    """Models of one or two layers, in float32: whole, in portions down to two tokens, token by token."""
    cfg = ALONE[name]
    weights = L.random_weights(cfg, seed=21, sharpen=1.5)
    folder = L.write_folder(tmp_path / name, cfg, weights)
    seqs = sequences(cfg, weights, "float32", [1, 2, 70, 150], seed=30)
    for trace in (H.trace_whole(seqs), H.trace_portions(seqs), H.trace_tail(seqs, tail=40)):
        runner = make_runner(folder, "float32", n_pages=4)
        L.compare(H.run_trace(runner, trace), cfg, weights, seqs, **TOL["float32"])
    if name == "odd_width":
        # bfloat16 at a width no 16-byte access or tensor-memory copy takes: the products fall to the library, the rest to scalar accesses
        cfg = L.calm(cfg)
        weights = L.random_weights(cfg, seed=21, calm=True)
        folder = L.write_folder(tmp_path / (name + "_bf16"), cfg, weights)
        seqs = sequences(cfg, weights, "bfloat16", [1, 2, 70, 150], seed=30)
        runner = make_runner(folder, "bfloat16", n_pages=4)
        L.compare(H.run_trace(runner, H.trace_portions(seqs)), cfg, weights, seqs, **TOL["bfloat16"])


@pytest.fixture(scope="module", params=sorted(L.CONFIGS))
def model(request, tmp_path_factory):
    cfg = L.CONFIGS[request.param]
    made = {}
    # float32 runs see attention sharpened (a wrong key moves the logits far past the tolerance) and close router calls;
    # bfloat16's own rounding of q and k would be amplified alike, so its models are left as drawn
    for dtype, c, kw in (("float32", cfg, dict(sharpen=1.5)), ("bfloat16", L.calm(cfg), dict(calm=True))):
        weights = L.random_weights(c, seed=11, **kw)
        made[dtype] = (weights, L.write_folder(tmp_path_factory.mktemp(f"{request.param}_{dtype}"), c, weights), c)
    return request.param, made


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_all_cuttings_match_the_plain_model(model, dtype):
    """Whole; the last 32 tokens one by one; portions down to two tokens; and up to three live requests with so few
    pages and slots that both are used again."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, weights, dtype, [1, 5, 23, 64, 65, 97, 150, 201])
    results = {}
    for kind, trace in (("whole", H.trace_whole(seqs)), ("tail", H.trace_tail(seqs)), ("portions", H.trace_portions(seqs))):
        runner = make_runner(folder, dtype, n_pages=4)
        results[kind] = H.run_trace(runner, trace)
        assert all(g.pool.n_held == 0 for g in runner.cache.groups)
    trace = H.trace_mixed(seqs, max_tokens=64 * 7, seed=5, max_live=3)
    assert max(len(st["entries"]) for st in trace) >= 3
    runner = make_runner(folder, dtype, n_pages=7, slots=3)
    results["mixed"] = H.run_trace(runner, trace)
    assert all(g.pool.taken_total > g.pool.n_pages for g in runner.cache.groups), "no page was used twice"
    for kind, got in results.items():
        worst = L.compare(got, cfg, weights, seqs, **TOL[dtype])
        print(f"{name} {dtype} {kind}: max |diff| {worst:.3g}")
    if dtype == "float32":
        for kind in ("tail", "portions", "mixed"):
            for key, row in results["whole"].items():
                assert float((row - results[kind][key]).abs().max()) < 5e-5 * (1.0 + float(row.abs().max())), f"float32 {kind} differs from whole at {key}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_then_long_decoding(model, dtype):
    """Three tokens of prompt, then 230 tokens one by one (through captured steps): the states are carried 230 times,
    every convolution starts inside its first taps, and every window passes over decoded tokens."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, weights, dtype, [233], seed=70)
    runner = make_runner(folder, dtype, n_pages=4)
    got = H.run_trace(runner, H.trace_tail(seqs, tail=230))
    assert runner.graph_replays > 100
    L.compare(got, cfg, weights, seqs, **TOL[dtype])


def test_a_slot_that_is_used_again_starts_from_nothing(model):
    name, made = model
    weights, folder, cfg = made["float32"]
    seqs = sequences(cfg, weights, "float32", [130, 75], seed=90)
    fresh = make_runner(folder, "float32", n_pages=3, slots=1)
    want = H.run_trace(fresh, H.trace_portions({"r1": seqs["r1"]}))
    used = make_runner(folder, "float32", n_pages=3, slots=1)
    H.run_trace(used, H.trace_portions({"r0": seqs["r0"]}))
    got = H.run_trace(used, H.trace_portions({"r1": seqs["r1"]}))
    for key, row in want.items():
        assert torch.equal(row, got[key]), f"position {key[1]} differs after the slot was used before"
    L.compare(got, cfg, weights, {"r1": seqs["r1"]}, **TOL["float32"])


def test_batch_of_unequal_requests_equals_each_alone(model):
    name, made = model
    weights, folder, cfg = made["float32"]
    seqs = sequences(cfg, weights, "float32", [90, 3, 41, 1], seed=120)
    runner = make_runner(folder, "float32", n_pages=8)
    alone = H.run_trace(runner, H.trace_whole(seqs))
    together = H.run_trace(runner, [{"step": 0, "entries": [{"id": r, "tokens": ids, "want": list(range(len(ids)))} for r, ids in seqs.items()],
                                     "end": list(seqs)}])
    for key, row in alone.items():
        assert float((row - together[key]).abs().max()) < 1e-5 * (1.0 + float(row.abs().max())), f"{key} differs beside other requests"
    L.compare(together, cfg, weights, seqs, **TOL["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_tokens_in_a_step_beside_decoded_ones(model, dtype):
    """A portion of 290 tokens beside a decoded token (recurrences in pieces side by side; attention and experts on tensor cores
    where the sizes allow, in bfloat16); then the same request goes on token by token from the states and pages that step left."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, weights, dtype, [320, 80], seed=140)
    runner = make_runner(folder, dtype, n_pages=16)
    a, b = runner.open("r0"), runner.open("r1")
    got = {}
    rows = runner.step([(b, seqs["r1"][:70], [69])]).float().cpu()
    got[("r1", 69)] = rows[0]
    rows = runner.step([(a, seqs["r0"][:290], list(range(0, 290, 7))), (b, seqs["r1"][70:71], [0])]).float().cpu()
    for i, p in enumerate(range(0, 290, 7)):
        got[("r0", p)] = rows[i]
    got[("r1", 70)] = rows[-1]
    for p in range(290, 320):
        q = 71 + p - 290
        entries = [(a, [seqs["r0"][p]], [0])] + ([(b, [seqs["r1"][q]], [0])] if q < 80 else [])
        rows = runner.step(entries).float().cpu()
        got[("r0", p)] = rows[0]
        if len(entries) > 1:
            got[("r1", q)] = rows[1]
    runner.rt.check_status()
    L.compare(got, cfg, weights, seqs, **TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(model, dtype):
    """Engine.generate (scheduler, portions of 16 prompt tokens, sampling on the device, steps run ahead) and
    Engine.greedy against greedy decoding with the plain model."""
    import lgml_b200

    name, made = model
    weights, folder, cfg = made[dtype]
    prompts = [H.random_ids(n, cfg["vocab"], 200 + n) for n in (37, 5, 70)]
    eng = lgml_b200.Engine(str(folder), dtype=dtype, n_ctx=256, slots=2, ubatch=16)
    outs = eng.generate(prompts, max_tokens=10, temperature=0.0, stop=[])
    solo, _ = eng.greedy(prompts[0], 10)
    for prompt, got in zip(prompts, outs):
        assert len(got) == 10
        for i, tok in enumerate(got):
            margins: list = []
            row = torch.from_numpy(P.forward(cfg, L.numpy_of(weights), prompt + got[:i], margins=margins)[-1])
            if dtype == "bfloat16" and min((float(m.min()) for m in margins), default=1.0) < 0.01:
                break           # from here on a router's close call may have gone the other way
            gap = float(row.max() - row[tok])
            bound = 1e-4 if dtype == "float32" else 5e-2 * float(row.abs().max())
            assert gap <= bound, f"{dtype}: token {i} is {tok}, the plain model prefers {int(row.argmax())} by {gap:.3g}"
    if dtype == "float32":
        assert solo == outs[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_as_a_process(model, tmp_path, dtype):
    """bin/trace_run as a process on a mixed trace with two live requests and four pages."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, weights, dtype, [70, 20, 131], seed=310)
    trace = H.trace_mixed(seqs, max_tokens=64 * 4, seed=2, max_live=2)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                           "--max-tokens", str(64 * 4)], input="\n".join(json.dumps(s) for s in trace) + "\n", text=True,
                          capture_output=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    done = [ln for ln in proc.stdout.splitlines() if ln.startswith("done ")]
    assert done == [f"done {s['step']}" for s in trace]
    got, fed = {}, {r: 0 for r in seqs}
    for st in trace:
        wanted = sum(len(e["want"]) for e in st["entries"])
        rows = np.fromfile(out / f"{st['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) if wanted else np.zeros((0, cfg["vocab"]))
        assert rows.shape[0] == wanted
        r = 0
        for e in st["entries"]:
            for i in e["want"]:
                got[(e["id"], fed[e["id"]] + i)] = torch.from_numpy(rows[r].copy())
                r += 1
            fed[e["id"]] += len(e["tokens"])
    assert sum(fed.values()) == 221
    L.compare(got, cfg, weights, seqs, **TOL[dtype])


def test_command_line_generates_with_the_folders_architecture(model):
    name, made = model
    weights, folder, cfg = made["float32"]
    prompt = H.random_ids(19, cfg["vocab"], 400)
    proc = subprocess.run([sys.executable, "-m", "lgml_b200", "-m", str(folder), "--dtype", "float32", "-c", "128", "--prompt-ids", ",".join(map(str, prompt)),
                           "-n", "5", "--temperature", "0", "--repeat-stop", "0"], capture_output=True, text=True, timeout=600, cwd=str(ROOT))
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = [int(t) for t in proc.stdout.strip().splitlines()[-1].split(",")]
    assert len(got) == 5
    for i, tok in enumerate(got):
        row = L.oracle_logits(cfg, weights, prompt + got[:i])[-1]
        assert float(row.max() - row[tok]) <= 1e-4


def test_random_weights_mode_runs_the_design():
    """A configuration alone is enough: the engine draws weights of the shapes and kinds the parts ask for."""
    from lgml_b200.config import config_from_dict
    from lgml_b200.engine.runner import ModelRunner

    runner = ModelRunner.from_config(config_from_dict(L.MIXED), seed=3, dtype=torch.bfloat16, n_pages=4, max_slots=2)
    req = runner.open("a")
    rows = runner.step([(req, H.random_ids(70, 97, 1), [0, 69])])
    runner.rt.check_status()
    assert rows.shape == (2, 97) and bool(torch.isfinite(rows).all())
