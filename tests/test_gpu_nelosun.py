"""Nelosun in the engine against the plain implementation: every mechanism alone, then whole models under every way of
cutting the work.

The models are small and differ from each other in every size and option (loops in the middle, over everything, of one layer and
that run once; one to eight heads of 5 to 128 entries; latent cells of 12 to 544 numbers; one to seven taps; recurrences narrower
and wider than the model in parts of 7 to 96 channels; one to forty experts of which one to all are a token's; layers without a
feed-forward).  Where random numbers would hide a fault, the inputs are made so that it shows: single keys stand far out, scores
so low that the one in the denominator is all there is, recurrences that still hold what hundreds of tokens back wrote, gate
logits whose products would not survive sixteen bits.
"""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import helpers as H
from tests import nelosun_helpers as L
from tests.plain import nelosun_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": dict(atol=3e-5, rtol=2e-4), "bfloat16": dict(atol=3e-2, rtol=0.06)}


def i32(values):
    return torch.tensor(np.asarray(list(values)), dtype=torch.int32, device=DEV)


def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def bf(a):
    """The nearest bfloat16 numbers, as float64."""
    return torch.tensor(np.asarray(a)).to(torch.bfloat16).double().numpy()


def dev(a, dtype):
    return torch.tensor(np.asarray(a), dtype=torch.float64).to(dtype).to(DEV)


def portions_of(total, cuts):
    out, a, i = [], 0, 0
    while a < total:
        n = min(cuts[i % len(cuts)], total - a)
        out.append((a, a + n))
        a, i = a + n, i + 1
    return out


def runtime(dtype):
    from lgml_b200.engine.runtime import Runtime

    return Runtime(DEV, dtype)


def worst(got, want):
    return float(np.abs(np.asarray(got.detach().double().cpu() if torch.is_tensor(got) else got) - want).max())


# ---------------------------------------------------------------------------------------------
# the norm with channel scales
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,n", [(33, 5), (36, 7), (64, 130), (1030, 3), (2048, 70), (4100, 4), (9000, 3)])
def test_scaled_terms_and_norm_in_one_kernel(out_dtype, E, n):
    """x += s_a (product in parts + bias) + s_b (tensor, or a token's experts); then the norm, also into the experts' tiles; chosen rows; x replaced;
    a product over x in two pieces; x in two pieces."""
    from lgml_b200 import ops

    rng = np.random.default_rng(E + n)
    x, w, bias, sa, sb = rng.normal(size=(n, E)), *(rng.normal(size=E) for _ in range(4))
    eps = 1e-4
    norm = lambda v: P.rms_norm(v, w, eps)
    tol = 2e-6 if out_dtype == torch.float32 else 2e-2
    run = lambda xd, terms, **kw: ops.scaled_norm(xd, terms, eps, f32(w), torch.empty((n, E), dtype=out_dtype, device=DEV), **kw)
    for n_parts in (1, 2, 9, 11):
        parts = rng.normal(size=(n_parts, n, E))
        a = parts.sum(axis=0) + bias
        for top in (0, 1, 2, 3):
            if top:
                y = rng.normal(size=(4 * n * top, E))
                places = np.stack([rng.permutation(4 * n * top)[:top] for _ in range(n)])
                b, term = y[places].sum(axis=1) * 0.7, ops.Term(ops.ExpertRows(f32(y), i32(places.reshape(-1)).view(n, top), 0.7), f32(sb))
            else:
                b = rng.normal(size=(n, E))
                term = ops.Term(f32(b), f32(sb), mul=1.0)
            want = x + sa * a + sb * b
            xd = f32(x)
            tiles, at = None, None
            if out_dtype == torch.bfloat16:
                tiles = torch.zeros((5 * n, E), dtype=torch.bfloat16, device=DEV)
                at = i32(np.stack([rng.permutation(n) * 2, rng.permutation(n) * 2 + 1], axis=1).reshape(-1)).view(n, 2)
            out = run(xd, (ops.Term(ops.Partials(f32(parts), f32(bias)), f32(sa)), term), tiles=tiles, places=at)
            assert worst(xd, want) < 2e-5 and worst(out, norm(want)) < tol * (1 + np.abs(norm(want)).max())
            if tiles is not None:
                assert torch.equal(tiles[at[:, 0].long()], out) and torch.equal(tiles[at[:, 1].long()], out)
            # chosen rows: x stays as it is
            xd, rows = f32(x), np.array([n - 1, 0, n // 2])
            out = ops.scaled_norm(xd, (ops.Term(ops.Partials(f32(parts), f32(bias)), f32(sa)), term), eps, f32(w), torch.empty((3, E), dtype=out_dtype, device=DEV),
                                  rows=i32(rows))
            assert torch.equal(xd, f32(x)) and worst(out, norm(want)[rows]) < tol * (1 + np.abs(norm(want)).max())
    # nothing pending, nothing wanted
    xd = f32(x)
    assert worst(run(xd, ()), norm(x)) < tol * (1 + np.abs(norm(x)).max()) and torch.equal(xd, f32(x))
    ops.scaled_norm(xd, (), eps, f32(w), torch.empty((0, E), dtype=out_dtype, device=DEV), rows=i32([]))
    # x replaced: a product over x in two pieces, and column slices of a wider product, each with a factor
    for n_parts in (1, 3):
        two, wide = rng.normal(size=(n_parts, 2 * n, E)), rng.normal(size=(n, 2 * E))
        want = two[:, :n].sum(axis=0) + two[:, n:].sum(axis=0) + 2.5 * wide[:, E:]
        xd = torch.full((n, E), float("nan"), device=DEV)
        value = ops.Partials(f32(two)) if n_parts > 1 else f32(two[0])
        out = run(xd, (ops.Term(value, stacked=True), ops.Term(f32(wide)[:, E:], mul=2.5)), keep=False)
        assert worst(xd, want) < 2e-5 and worst(out, norm(want)) < tol * (1 + np.abs(norm(want)).max())
    want = 0.5 * wide[:, :E] + 0.5 * wide[:, E:]
    xd = torch.full((n, E), float("nan"), device=DEV)
    wd = f32(wide)
    run(xd, (ops.Term(wd[:, :E], mul=0.5), ops.Term(wd[:, E:], mul=0.5)), keep=False)
    assert worst(xd, want) < 2e-5
    # no norm: x in two bfloat16 pieces that hold sixteen of its bits
    xd, split = f32(x), torch.empty((2 * n, E), dtype=torch.bfloat16, device=DEV)
    ops.scaled_norm(xd, (ops.Term(f32(wide)[:, :E], f32(sa)),), split=split)
    want = x + sa * wide[:, :E]
    assert worst(xd, want) < 2e-5 and torch.equal(split[:n], xd.to(torch.bfloat16))
    assert bool(((split[:n].float() + split[n:].float() - xd).abs() <= xd.abs() * 2.0 ** -16 + 1e-30).all())


def test_scaled_terms_refuse_what_does_not_fit():
    from lgml_b200 import ops

    x, w, out = torch.zeros((3, 8), device=DEV), torch.ones(8, device=DEV), torch.empty((3, 8), device=DEV)
    part = lambda *shape: ops.Partials(torch.zeros(shape, device=DEV))
    for terms in ((ops.Term(part(2, 3, 8)), ops.Term(part(2, 3, 8))), (ops.Term(part(2, 4, 8)),), (ops.Term(torch.zeros((3, 7), device=DEV)),),
                  (ops.Term(torch.zeros((3, 8), device=DEV), torch.ones(7, device=DEV)),), (ops.Term(torch.zeros((3, 8), device=DEV), stacked=True),)):
        with pytest.raises(ops.KernelError):
            ops.scaled_norm(x, terms, 1e-5, w, out)
    with pytest.raises(ops.KernelError):
        ops.scaled_norm(x, (), 1e-5, w)                    # a weight without an output
    with pytest.raises(ops.KernelError):
        ops.scaled_norm(x, (), 1e-5, w, out, rows=i32([0, 1, 2]), split=torch.empty((6, 8), dtype=torch.bfloat16, device=DEV))


# ---------------------------------------------------------------------------------------------
# experts that stand in a table
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("n", [1, 7, 8, 20, 64, 150, 700])
def test_routing_of_several_tables_in_one_launch(n):
    """Every row has a place of its own in a tile of its expert, and the tiles hold nothing else."""
    from lgml_b200 import ops

    rng = np.random.default_rng(n)
    vocab, shapes = 53, [(5, 2), (1, 1), (40, 3), (7, 7), (3, 1)]
    tables = [np.stack([rng.permutation(X)[:top] for _ in range(vocab)]) for X, top in shapes]
    at, desc = 0, []
    for t, (X, top) in zip(tables, shapes):
        desc.append((X, top, at))
        at += t.size
    ids = rng.integers(0, vocab, size=n)
    routes = ops.table_route(i32(ids), vocab, i32(np.concatenate([t.reshape(-1) for t in tables])), i32(np.array(desc).reshape(-1)).view(-1, 3), shapes)
    for table, (X, top), r in zip(tables, shapes, routes):
        assert np.array_equal(r.ids.cpu().numpy(), table[ids])
        tiles, places = r.tiles.cpu().numpy(), r.places.cpu().numpy().reshape(-1)
        count, list_ = int(tiles[-1]), tiles[:-1].reshape(-1, 3)
        assert count <= len(list_) and len(set(places)) == n * top and r.tile_rows in (16, 32, 64, 128)
        assert np.array_equal(list_[places // r.tile_rows, 0], table[ids].reshape(-1)) and places.max() < count * r.tile_rows
        for k in range(count):
            inside = places[places // r.tile_rows == k] - k * r.tile_rows
            assert sorted(inside) == list(range(list_[k, 2])) and list_[k, 2] > 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("X,top,E,F,n", [(5, 2, 64, 48, 3), (16, 4, 128, 64, 200), (1, 1, 24, 16, 5), (40, 3, 72, 520, 9), (8, 8, 64, 40, 60), (3, 1, 37, 19, 11),
                                         (8, 2, 256, 136, 8), (6, 2, 64, 48, 33), (4, 2, 64, 264, 90), (12, 1, 520, 24, 500)])
def test_clamped_experts_in_every_form(dtype, X, top, E, F, n):
    """The row form and the grouped products (tiles of 16 to 128 rows), each token's experts counting the same; the branches reach the clamps."""
    from lgml_b200 import ops

    rng = np.random.default_rng(X * 100 + n)
    limit, alpha = 0.8, 1.702
    wg, wu, wd = (bf(rng.normal(size=s) * g / s[2] ** 0.5) for s, g in (((X, F, E), 1.5), ((X, F, E), 1.5), ((X, E, F), 1.0)))
    h = bf(rng.normal(size=(n, E)))
    table = np.stack([rng.permutation(X)[:top] for _ in range(31)])
    ids = rng.integers(0, 31, size=n)
    W = {"t.table": table}
    for e in range(X):
        W[f"t.e{e}.gate"], W[f"t.e{e}.up"], W[f"t.e{e}.down"] = wg[e], wu[e], wd[e]
    f = {"expert": {"limit": limit}, "router": {"top": top}}
    want = P.table_experts(h, ids, W, "t", f)
    for other in (dict(limit=limit * 1.1), dict(limit=1e9)):
        assert np.abs(P.table_experts(h, ids, W, "t", {"expert": other, "router": {"top": top}}) - want).max() > 0.02, "the clamp would not show"
    rt = runtime(dtype)
    w_gu = dev(np.stack([wg, wu], axis=2).reshape(X, 2 * F, E), dtype)
    wdd, hd = dev(wd, dtype), dev(h, dtype)
    route = ops.table_route(i32(ids), 31, i32(table.reshape(-1)), i32([X, top, 0]).view(1, 3), [(X, top)])[0]
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    got = ops.moe_experts_rows(hd, route.ids, None, w_gu, wdd, clamp=(alpha, limit))
    assert worst(got, want) < tol * (1 + np.abs(want).max())
    wts = torch.full((n, top), 1.0 / top, device=DEV)
    assert worst(ops.moe_experts_rows(hd, route.ids, wts, w_gu, wdd, clamp=(alpha, limit)), want) < tol * (1 + np.abs(want).max())
    if dtype == torch.bfloat16 and w_gu.shape[1] % 16 == 0 and E % 8 == 0:
        a = torch.full((route.max_tiles * route.tile_rows, E), float("nan"), dtype=dtype, device=DEV)       # rows without a token hold anything
        a[route.places.reshape(-1).long()] = hd.repeat_interleave(top, dim=0)
        y = ops.moe_tile_products(a, route.tiles, w_gu, wdd, rt.status, clamp=(alpha, limit))
        rt.check_status()
        got = y[route.places.long()].sum(dim=1) / top
        assert worst(got, want) < tol * (1 + np.abs(want).max())


# ---------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------

HEADS = [(4, 2, 64, 64), (2, 1, 128, 128), (6, 2, 32, 24), (3, 3, 48, 80), (2, 2, 10, 7), (1, 1, 160, 96), (12, 1, 64, 64), (2, 1, 600, 520)]


class Step:
    """A step of one request's tokens a .. b - 1."""

    def __init__(self, a, b):
        self.positions, self.seq_of_token, self.max_q_len, self.max_kv_len = i32(range(a, b)), i32([0] * (b - a)), b - a, b

    def attention_tiles(self, tt):
        m = self.max_q_len
        return torch.tensor([[0, t0, min(tt, m - t0), 0] for t0 in range(0, m, tt)], dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("dtype,heads", [(d, h) for d in (torch.float32, torch.bfloat16) for h in HEADS])
def test_one_in_the_denominator_and_a_gate_per_head_in_every_kernel_form(dtype, heads):
    """Queries and keys are made so that for the tokens of one half all scores are far below zero (the one in the denominator takes nearly
    everything) and for the others a few keys stand far out, at the borders of pages and at the query itself."""
    from lgml_b200 import ops
    from lgml_b200.engine.batch import CacheView

    H_, G, D, Dv = heads
    rng = np.random.default_rng(H_ * 100 + D)
    n, scale, coef, every = 200, 4.0 / D, 0.8, 50
    base = rng.normal(size=(H_, D))
    temp = P.query_temperature(n, coef, every)
    sign = np.where(np.arange(n) % 3 == 1, -1.0, 1.0)
    q = sign[:, None, None] * base[None] + 0.1 * rng.normal(size=(n, H_, D))
    k, v = 0.3 * rng.normal(size=(n, G, D)), rng.normal(size=(n, G, Dv)) * 2
    loud = [0, 3, 63, 64, 100, 127, 128, 191]
    for g in range(G):
        k[:, g] += 0.2 * base[g * (H_ // G)]
        k[loud, g] = base[g * (H_ // G)] + 0.05 * rng.normal(size=(len(loud), D))
    gate = rng.normal(size=(n, H_)) * 2

    def plain(sink=True, floor=True, gated=True, seen=None):
        t = temp if floor else np.array([1.0 + coef * np.log((p + 1) / every + 1.0) for p in range(n)])
        out = np.zeros((n, H_, Dv))
        see = P.causal(n) if seen is None else seen
        for h in range(H_):
            s = (q[:, h] * t[:, None]) @ k[:, h // (H_ // G)].T * scale
            w = (P.softmax_plus_one if sink else P.softmax_rows)(s, see)
            out[:, h] = w @ v[:, h // (H_ // G)] * (P.sigmoid(gate[:, h:h + 1]) if gated else 1.0)
        return out

    want = plain()
    strict = P.causal(n) & ~np.eye(n, dtype=bool)
    strict[0, 0] = True
    for what, other in (("no one", plain(sink=False)), ("no floor", plain(floor=False)), ("no gate", plain(gated=False)), ("not itself", plain(seen=strict))):
        assert np.abs(other - want).max() > (0.1 if what != "no floor" else 0.02), f"{what} would not show"
    rt = runtime(dtype)
    n_pages, pages = 7, [5, 2, 6, 0]
    table = i32(pages).view(1, -1)
    proj = f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), gate], axis=1))
    lo = H_ * D + G * (D + Dv)
    sinks = torch.zeros(H_, device=DEV)
    for form, cuts in (("auto", [n]), ("auto", [7, 2, 1, 60, 3, 129]), ("split", [30, 1, 5]), ("mma", [n]), ("general", [65])):
        if form != "auto" and dtype == torch.float32 or form == "split" and max(D, Dv) > 256 or form == "mma" and max(D, Dv) > 128:
            continue
        kp = torch.full((n_pages, G, 64, D), 60.0, dtype=dtype, device=DEV)       # what an earlier request may have left
        vp = torch.full((n_pages, G, 64, Dv), 60.0, dtype=dtype, device=DEV)
        got = np.zeros_like(want)
        for a, b in portions_of(n, cuts):
            step = Step(a, b)
            qd = ops.sink_qkv_store(proj[a:b], step.positions, step.seq_of_token, table, kp, vp, H_, rt.status, temp_coef=coef, temp_every=every)
            out = torch.zeros((b - a, H_ * Dv + 8), dtype=dtype, device=DEV)[:, :H_ * Dv]
            kw = dict(sinks=sinks, gate=proj[a:b, lo:])
            if form == "split":
                ops.sink_decode(qd, step.positions, step.seq_of_token, table, kp, vp, out, H_, scale, 0, rt.status, 3 if b > 128 else 1, **kw)
            elif form == "mma":
                ops.sink_attention_mma(qd, step.positions, step.attention_tiles(64), table, kp, vp, out, H_, scale, 0, rt.status, **kw)
            elif form == "general":
                ops.sink_attention(qd, step.positions, step.seq_of_token, table, kp, vp, out, H_, scale, 0, rt.status, **kw)
            else:
                rt.sink_attention(qd, step, CacheView(k=kp, v=vp, block_table=table), out, H_, scale, 0, None, sinks, proj[a:b, lo:])
            got[a:b] = out.float().cpu().numpy().reshape(b - a, H_, Dv)
        rt.check_status()
        tol = 3e-5 if dtype == torch.float32 else 3e-2
        err = np.abs(got - want).max(axis=(1, 2))
        assert err.max() < tol * (1 + np.abs(want).max()), f"{form} {cuts}: token {int(err.argmax())}: {err.max():.3g}"


def test_a_gate_of_another_width_is_refused():
    from lgml_b200 import ops

    q, kp, vp = torch.zeros((2, 16), device=DEV), torch.zeros((1, 1, 64, 8), device=DEV), torch.zeros((1, 1, 64, 4), device=DEV)
    out, table, status = torch.zeros((2, 8), device=DEV), i32([0]).view(1, 1), torch.zeros(1, dtype=torch.int32, device=DEV)
    for cols in (3, 7, 9):
        with pytest.raises(ops.KernelError):
            ops.sink_attention(q, i32([0, 1]), i32([0, 0]), table, kp, vp, out, 2, 0.3, 0, status, gate=torch.zeros((2, cols), device=DEV))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads", [(4, 32, 32, 40, 48, 96), (2, 16, 48, 24, 16, 16), (3, 10, 6, 7, 11, 14), (1, 5, 2, 9, 7, 33), (5, 64, 32, 64, 40, 160), (2, 24, 32, 16, 20, 520)])
def test_latent_attention_with_a_query_latent_whole_and_in_portions(dtype, heads):
    """The mixer between its first projection's input and the output projection's result against the form that builds every head's keys, with a
    key far back that stands out; pairs (i, i + half) turn."""
    from lgml_b200.engine.batch import CacheView
    from lgml_b200.parts import make_part

    H_, D, Dr, Dv, Rq, R = heads
    rng = np.random.default_rng(R + H_)
    E, n = 40, 150
    m = {"heads": H_, "dim": D, "rot_dim": Dr, "vdim": Dv, "q_rank": Rq, "kv_rank": R, "scale": 2.5 / (D + Dr) ** 0.5, "rot": {"base": 300.0, "dims": Dr}}
    mat = lambda o, i, g=1.0: bf(rng.normal(size=(o, i)) * g / i ** 0.5)
    W = {"m.dq": mat(Rq, E), "m.dq.norm": bf(rng.normal(size=Rq) * 0.2 + 1), "m.uq": mat(H_ * (D + Dr), Rq, 1.5), "m.dkv": mat(R + Dr, E, 1.2),
         "m.dkv.norm": bf(rng.normal(size=R) * 0.2 + 1), "m.uk": mat(H_ * D, R, 1.3), "m.uv": mat(H_ * Dv, R, 1.3), "m.o": mat(E, H_ * Dv)}
    h = bf(rng.normal(size=(n, E)))
    want = P.latent_attention(h, W, "m", m, 1e-5)
    assert np.abs(P.latent_attention(h, W, "m", {**m, "rot": {"base": 310.0, "dims": Dr}}, 1e-5) - want).max() > (0.05 if Dr > 2 else -1), "the turn would not show"
    rt = runtime(dtype)
    part = make_part("mixer", "latent_attention", width=E, n_heads=H_, head_dim=D, rot_dim=Dr, v_head_dim=Dv, rank=R, scale=m["scale"], eps=1e-5, rope_base=300.0,
                     rope_dims=Dr, q_rank=Rq, halves=True)
    part.bind("m", {k: dev(v, torch.float32 if v.ndim == 1 else dtype) for k, v in W.items()}, rt)
    table = i32([3, 0, 2]).view(1, -1)
    for cuts in ([n], [3, 2, 70, 1], [40, 9]):
        cells = torch.full((5, 1, 64, R + Dr), 7.0, dtype=dtype, device=DEV)
        got = np.zeros((n, E))
        for a, b in portions_of(n, cuts):
            step = Step(a, b)
            step.n_tokens, step.decode_splits, step.n_seqs, step.seq_lens = b - a, None, 1, [b - a]
            y = part.forward(rt, dev(h[a:b], dtype), step, CacheView(k=cells, v=cells[..., :R], block_table=table))
            got[a:b] = (y.sum() if hasattr(y, "data") and not torch.is_tensor(y) else y).float().cpu().numpy()
        rt.check_status()
        tol = 3e-5 if dtype == torch.float32 else 4e-2
        err = np.abs(got - want).max(axis=1)
        assert err.max() < tol * (1 + np.abs(want).max()), f"{cuts}: token {int(err.argmax())}: {err.max():.3g}"


def test_latent_angles_at_far_positions_and_a_missing_page():
    """Positions of tens of thousands turn as exactly as the first ones, in cells and queries; a position without a page is flagged, not written."""
    from lgml_b200 import ops

    rng = np.random.default_rng(4)
    H_, D, Dr, Rq, R, base = 2, 12, 10, 9, 14, 900.0
    rt = runtime(torch.float32)
    pos = np.array([0, 1, 63, 20000, 65535, 70000])
    n = len(pos)
    table = torch.full((1, 1100), -1, dtype=torch.int32, device=DEV)
    for p in pos:
        table[0, p // 64] = int(p // 64) % 5
    f = np.array([base ** (-2.0 * i / Dr) for i in range(Dr // 2)])
    hi = f.astype(np.float32)
    freq = torch.stack([f32(hi), f32(f - hi.astype(np.float64))]).contiguous()
    down, wq, w = rng.normal(size=(n, Rq + R + Dr)), rng.normal(size=Rq), rng.normal(size=R)
    cells = torch.full((5, 1, 64, R + Dr), 9.0, device=DEV)
    cq, cs = ops.latent_down(f32(down), f32(wq), f32(w), 1e-5, freq, Dr, i32(pos), i32([0] * n), table, cells, Rq, R, Dr, rt.status, halves=True)
    rt.check_status()
    assert worst(cq, P.rms_norm(down[:, :Rq], wq, 1e-5)) < 2e-6
    c, r = P.rms_norm(down[:, Rq:Rq + R], w, 1e-5), P.rotate_half(down[:, Rq + R:], base, Dr, pos)
    for i, p in enumerate(pos):
        assert worst(cells[(p // 64) % 5, 0, p % 64], np.concatenate([c[i], r[i]])) < 3e-6
    q, wuk = rng.normal(size=(n, H_ * (D + Dr))), rng.normal(size=(H_, R, D))
    full = ops.latent_query(f32(q), f32(wuk), cs, Dr, Dr, halves=True)
    qh = q.reshape(n, H_, D + Dr)
    want = np.concatenate([np.einsum("thd,hrd->thr", qh[:, :, :D], wuk), P.rotate_half(qh[:, :, D:], base, Dr, pos)], axis=2)
    assert worst(full.view(n, H_, R + Dr), want) < 1e-5
    table[0, 0] = -1
    ops.latent_down(f32(down), f32(wq), f32(w), 1e-5, freq, Dr, i32(pos), i32([0] * n), table, cells, Rq, R, Dr, rt.status, halves=True)
    with pytest.raises(Exception):
        rt.check_status()


# ---------------------------------------------------------------------------------------------
# the recurrence
# ---------------------------------------------------------------------------------------------

RECURRENCES = [(48, 3, 4), (128, 2, 3), (21, 3, 7), (64, 1, 1), (96, 2, 2), (40, 5, 5), (512, 2, 4), (36, 1, 4), (24, 3, 4)]


def recurrence(C, B, taps, seed):
    rng = np.random.default_rng(seed)
    P_ = C // B
    W = {"conv": bf(rng.normal(size=(C, taps)) * 0.6), "conv.b": rng.normal(size=C) * 0.3, "ra": bf(rng.normal(size=(B, P_, P_)) * 2 / P_ ** 0.5),
         "ri": bf(rng.normal(size=(B, P_, P_)) * 2 / P_ ** 0.5), "ra.b": rng.normal(size=(B, P_)) * 0.5, "ri.b": rng.normal(size=(B, P_)) * 0.5,
         # from decays that still hold a tenth after 2,000 tokens to none at all
         "lam": rng.uniform(-10.0, 1.0, size=C)}
    return rng, {k: np.float32(v).astype(np.float64) for k, v in W.items()}


def plain_recurrence(x, y, W):
    u = P.causal_conv(x, W["conv"], W["conv.b"])
    r, i = P.sigmoid(P.block_linear(u, W["ra"], W["ra.b"])), P.sigmoid(P.block_linear(u, W["ri"], W["ri.b"]))
    return u, r, i, P.rglru_scan(u, r, i, W["lam"]) * P.gelu_tanh(y)


def bound_weights(W, dtype):
    sp8 = 8.0 * np.logaddexp(0.0, W["lam"])
    return (f32(W["conv"].T.copy()), f32(W["conv.b"])), (dev(W["ra"], dtype), f32(W["ra.b"].reshape(-1)), dev(W["ri"], dtype), f32(W["ri.b"].reshape(-1)), f32(sp8))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,B,taps", RECURRENCES)
def test_gates_are_32_bit_sums_in_every_form(dtype, C, B, taps):
    """Decays and pushed terms from float32 inputs to 32-bit accuracy, with matrices in either type: sixteen bits of the inputs would not do (checked
    first).  The pieces of an input add up to it."""
    from lgml_b200 import ops

    rng, W = recurrence(C, B, taps, C + taps)
    n = 150
    x = np.float32(rng.normal(size=(n, C)) * 3).astype(np.float64)
    proj = f32(np.concatenate([x, x], axis=1))
    conv, gates = bound_weights(W, dtype)
    state = torch.zeros((2, ops.rglru_state_floats(C, taps)), device=DEV)
    args = (proj, *conv, state, i32([0] * n), i32([0, n]), i32([1]), i32(range(n)))
    u = ops.rglru_conv(*args)
    want_u = P.causal_conv(x, W["conv"], W["conv.b"])
    assert worst(u, want_u) < 1e-5
    ud = u.double().cpu().numpy()
    r, i = P.sigmoid(P.block_linear(ud, W["ra"], W["ra.b"])), P.sigmoid(P.block_linear(ud, W["ri"], W["ri.b"]))
    log_a = -8.0 * r * P.softplus(W["lam"])
    a, push = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * ud
    rough = P.sigmoid(P.block_linear(bf(ud), W["ri"], W["ri.b"]))
    assert np.abs(np.sqrt(-np.expm1(2.0 * log_a)) * rough * ud - push).max() > 1e-3, "rounded inputs would not show"
    ab = ops.rglru_gates(u, *gates)
    assert worst(ab[0], a) < 2e-6 and worst(ab[1], push) < 1e-5 * (1 + np.abs(push).max())
    if dtype == torch.bfloat16 and (C // B) % 8 == 0:
        rt = runtime(dtype)
        for m in (150, 60, 32, 5):          # tiles of 128, 64 and 32 rows, whole and partly filled
            P_ = C // B
            few = (proj[:m], *conv, torch.zeros_like(state), i32([0] * m), i32([0, m]), i32([1]), i32(range(m)))
            pieces = ops.rglru_conv(*few, part=P_)
            rows, tile = ops.rglru_pieces_rows(m)
            assert tuple(pieces.shape) == (B, rows, 3, P_)
            assert worst(pieces[:, :m].double().sum(dim=2).permute(1, 0, 2).reshape(m, C), ud[:m]) < 1e-6
            tiles = i32([v for b in range(B) for _ in range(rows // tile) for v in (b, 0, 0)] + [B * (rows // tile)])
            chunks = i32([0, min(7, m), min(7, m), m]).view(2, 2)
            for ch in (None, chunks):
                ab, ends = ops.rglru_gates_pieces(pieces, m, ops.rglru_pieces_matrices(gates[0], gates[2]), tiles, gates[1], gates[3], gates[4], rt.status, chunks=ch)
                rt.check_status()
                assert worst(ab[0], a[:m]) < 1e-5 and worst(ab[1], push[:m]) < 1e-5 * (1 + np.abs(push).max())
            for k, (lo, hi) in enumerate(chunks.tolist()):
                S = np.zeros(C)
                for t in range(lo, hi):
                    S = a[t] * S + push[t]
                assert worst(ends[0, k], np.prod(a[lo:hi], axis=0)) < 3e-5 and worst(ends[1, k], S) < 1e-4 * (1 + np.abs(S).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,B,taps", RECURRENCES)
def test_recurrence_whole_in_pieces_and_token_by_token(dtype, C, B, taps):
    """Three requests in steps of every kind: one-token steps (one kernel), portions, long portions in pieces side by side, a request that sits a
    step out; the slots are not the first ones and hold what an earlier request left until they are cleared."""
    from lgml_b200 import ops

    rng, W = recurrence(C, B, taps, 7 * C + taps)
    lens = [330, 200, 75]
    xs = [np.float32(rng.normal(size=(n, C))).astype(np.float64) for n in lens]
    ys = [np.float32(rng.normal(size=(n, C))).astype(np.float64) for n in lens]
    want = [plain_recurrence(x, y, W)[3] for x, y in zip(xs, ys)]
    flip = [v.copy() for v in xs]
    flip[0][0] *= -1
    assert np.abs(plain_recurrence(flip[0], ys[0], W)[3][-1] - want[0][-1]).max() > 1e-3, "the first token would not show at the end"
    conv, gates = bound_weights(W, dtype)
    rt = runtime(dtype)
    slots = [3, 0, 2]
    plans = {"whole": [[330, 200, 75]], "single": [[1, 1, 1]] * 330, "mixed": [[1, 7, 75], [2, 1, 0], [64, 0, 0], [65, 3, 0], [1, 1, 0], [1, 1, 0], [129, 180, 0], [67, 7, 0]]}
    for name, plan in plans.items():
        state = torch.full((4, ops.rglru_state_floats(C, taps) + 3), 5.0, device=DEV)
        for s in slots:
            state[s].zero_()
        at, got = [0, 0, 0], [np.zeros_like(w) for w in want]
        for portion in plan:
            here = [(r, min(n, lens[r] - at[r])) for r, n in enumerate(portion) if n and at[r] < lens[r]]
            if not here:
                continue
            cat = lambda seqs: np.concatenate([seqs[r][at[r]:at[r] + n] for r, n in here])
            proj = f32(np.concatenate([cat(xs), cat(ys)], axis=1))
            pos = i32(np.concatenate([np.arange(at[r], at[r] + n) for r, n in here]))
            seq, start = i32([k for k, (_, n) in enumerate(here) for _ in range(n)]), i32(np.concatenate([[0], np.cumsum([n for _, n in here])]))
            sl = i32([slots[r] for r, _ in here])
            total = proj.shape[0]
            if max(n for _, n in here) == 1:
                out = ops.rglru_step(proj, *conv, state, sl, pos, *gates)
            else:
                out = torch.empty((total, C), dtype=dtype, device=DEV)
                pieces, ends = (None, None), None
                if max(n for _, n in here) > 64:
                    rows, first, t = [], [0], 0
                    for _, n in here:
                        rows += [(t + k, t + min(k + ops.rglru_chunk_tokens(), n)) for k in range(0, n, ops.rglru_chunk_tokens())]
                        first.append(len(rows))
                        t += n
                    pieces = (i32(np.array(rows).reshape(-1)).view(-1, 2), i32(first))
                P_ = C // B
                if dtype == torch.bfloat16 and P_ % 8 == 0 and total >= 32:
                    u = ops.rglru_conv(proj, *conv, state, seq, start, sl, pos, part=P_)
                    r_, tile = ops.rglru_pieces_rows(total)
                    tiles = i32([v for b in range(B) for _ in range(r_ // tile) for v in (b, 0, 0)] + [B * (r_ // tile)])
                    ab, ends = ops.rglru_gates_pieces(u, total, ops.rglru_pieces_matrices(gates[0], gates[2]), tiles, gates[1], gates[3], gates[4], rt.status,
                                                      chunks=pieces[0])
                    rt.check_status()
                else:
                    ab = ops.rglru_gates(ops.rglru_conv(proj, *conv, state, seq, start, sl, pos), *gates)
                ops.rglru_scan(ab, proj, state, start, sl, out, *pieces, ends=ends)
            t = 0
            for r, n in here:
                got[r][at[r]:at[r] + n] = out[t:t + n].float().cpu().numpy()
                at[r] += n
                t += n
        if name != "mixed":
            assert at == lens
        assert bool((state[1] == 5.0).all()), "a slot that no request holds was written"
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        for r in range(3):
            err = np.abs(got[r][:at[r]] - want[r][:at[r]]).max(axis=1)
            assert err.max() < tol * (1 + np.abs(want[r]).max()), f"{name}, request {r}, token {int(err.argmax())}: {err.max():.3g}"


# ---------------------------------------------------------------------------------------------
# the start of a pass
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,n", [(64, 3), (37, 5), (136, 90), (1024, 9)])
def test_a_pass_makes_x_anew_without_rounding_it(dtype, E, n):
    """First and later passes, at the start of the model and behind a layer: to 32-bit accuracy in both compute types (the matrix holds bfloat16
    numbers); rounding x on its way into the product would cost a hundred times as much."""
    from lgml_b200 import ops
    from lgml_b200.parts import PassInput, RMSNorm, ScaledTerms, TokenEmbedding

    rng = np.random.default_rng(E)
    vocab, scale = 29, 2.7
    table, w = bf(rng.normal(size=(vocab, E))), bf(rng.normal(size=(E, 2 * E)) / E ** 0.5)
    ids = rng.integers(0, vocab, size=n)
    rt = runtime(dtype)
    emb = TokenEmbedding(vocab, E, name="embed")
    emb.bind("", {"embed": dev(table, dtype)}, rt)
    part, norm = PassInput(E, emb, scale), RMSNorm(E, 1e-5, suffix="")
    part.bind("", {"loop.in": dev(w, dtype)}, rt)
    norm.bind("n", {"n": torch.ones(E, device=DEV)}, rt)
    rt.delta_dtype = torch.float32

    class Batch:
        token_ids, shared = i32(ids), {}

    x0 = table[ids] * scale
    tol = 1e-4
    # the model starts with the pass: x is not read
    xd = torch.full((n, E), float("nan"), device=DEV)
    norm.forward(rt, xd, rt.dtype, delta=part.forward(rt, xd, None, Batch, 0, starts_model=True))
    x1 = np.concatenate([x0, x0], axis=1) @ w.T
    assert worst(xd, x1) < tol
    # a later pass, with something pending
    d, s = rng.normal(size=(n, E)), rng.normal(size=E)
    norm.forward(rt, xd, rt.dtype, delta=part.forward(rt, xd, ScaledTerms((ops.Term(f32(d), f32(s)),)), Batch, 1, starts_model=False))
    x2 = np.concatenate([x1 + d * s, x0], axis=1) @ w.T
    assert worst(xd, x2) < tol
    if dtype == torch.bfloat16:
        assert np.abs(np.concatenate([bf(x1 + d * s), x0], axis=1) @ w.T - x2).max() > 10 * tol, "rounding would not show"
    # a first pass behind other layers, with and without something pending
    for pending, plus in ((None, 0.0), (f32(d), d)):
        Batch.shared = {}
        x = rng.normal(size=(n, E))
        xd = f32(x)
        norm.forward(rt, xd, rt.dtype, delta=part.forward(rt, xd, pending, Batch, 0, starts_model=False))
        assert worst(xd, np.concatenate([x + plus, x0], axis=1) @ w.T) < tol
    rt.check_status()


# ---------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------

def make_runner(folder, dtype, n_pages, slots=4, **kw):
    from lgml_b200.engine.engine import parse_dtype
    from lgml_b200.engine.runner import ModelRunner

    return ModelRunner.from_folder(folder, parse_dtype(dtype), DEV, n_pages=n_pages, max_slots=slots, max_step_tokens=n_pages * 64, **kw)


def sequences(cfg, lens, seed=50):
    return {f"r{i}": H.random_ids(n, cfg["vocab"], seed + i) for i, n in enumerate(lens)}


# one mechanism at a time: a model of one or two layers that has as little else as the design allows
ALONE = {
    "attention": L.config(53, 40, [L.attention(4, 2, 16, 8, 0.4)]),
    "temperature_of_one_step": L.config(53, 40, [L.attention(2, 1, 16, 16, 0.3, temp=(0.9, 1))]),
    "latent": L.config(53, 40, [L.latent(2, 12, 8, 20, 16, 24, 0.4)]),
    "recurrence": L.config(53, 40, [L.rglru(56, 7, 4)]),
    "recurrence_without_taps": L.config(53, 40, [L.rglru(24, 2, 1)]),
    "experts": L.config(53, 40, [L.rglru(8, 1, 2, mlp=L.moe(56, 9, 4, 0.5))]),
    "one_expert": L.config(53, 40, [L.attention(1, 1, 8, 8, 0.3, mlp=L.moe(16, 1, 1, 0.4))]),
    "a_loop_of_one_layer": L.config(53, 40, [L.rglru(24, 2, 3, mlp=L.moe(16, 3, 2, 1.0))], loop=(0, 1, 5), scale=4.0),
    "a_loop_behind_a_layer": L.config(53, 40, [L.attention(2, 2, 8, 8, 0.4), L.rglru(24, 2, 3)], loop=(1, 2, 2), scale=0.3),
    "odd_width": L.config(51, 35, [L.attention(3, 1, 10, 7, 0.3, mlp=L.moe(19, 3, 2, 1.0)), L.rglru(33, 3, 4, mlp=L.moe(33, 2, 1, 0.7)), L.latent(2, 6, 4, 5, 9, 11, 0.4)],
                          scale=1.5, loop=(0, 2, 2)),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_at_a_time(name, tmp_path):
    """Models of one to three layers, whole, in portions down to two tokens, and the last 40 tokens one by one."""
    cfg = ALONE[name]
    for dtype, sharpen in (("float32", 1.5), ("bfloat16", 1.0)):
        weights = L.random_weights(cfg, seed=21, sharpen=sharpen)
        folder = L.write_folder(tmp_path / (name + dtype), cfg, weights)
        seqs = sequences(cfg, [1, 2, 70, 150], seed=30)
        for trace in (H.trace_whole(seqs), H.trace_portions(seqs), H.trace_tail(seqs, tail=40)):
            runner = make_runner(folder, dtype, n_pages=4)
            L.compare(H.run_trace(runner, trace), cfg, weights, seqs, **TOL[dtype])


@pytest.fixture(scope="module", params=sorted(L.CONFIGS))
def model(request, tmp_path_factory):
    cfg = L.CONFIGS[request.param]
    made = {}
    # float32 runs see attention sharpened (a wrong key moves the logits far past the tolerance); bfloat16's own rounding of q and k would
    # be amplified alike, so its models are left as drawn
    for dtype, kw in (("float32", dict(sharpen=1.5)), ("bfloat16", {})):
        weights = L.random_weights(cfg, seed=11, **kw)
        made[dtype] = (weights, L.write_folder(tmp_path_factory.mktemp(f"{request.param}_{dtype}"), cfg, weights), cfg)
    return request.param, made


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_all_cuttings_match_the_plain_model(model, dtype):
    """Whole; the last 32 tokens one by one; portions down to two tokens; and up to three live requests with so few
    pages and slots that both are used again."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, [1, 5, 23, 64, 65, 97, 150, 201])
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
        worst_ = L.compare(got, cfg, weights, seqs, **TOL[dtype])
        print(f"{name} {dtype} {kind}: max |diff| {worst_:.3g}")
    if dtype == "float32":
        for kind in ("tail", "portions", "mixed"):
            for key, row in results["whole"].items():
                assert float((row - results[kind][key]).abs().max()) < 5e-5 * (1.0 + float(row.abs().max())), f"float32 {kind} differs from whole at {key}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_then_long_decoding(model, dtype):
    """Three tokens of prompt, then 230 tokens one by one (through captured steps): the states are carried 230 times,
    every convolution starts inside its first taps, and the temperature steps under decoded tokens."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, [233], seed=70)
    runner = make_runner(folder, dtype, n_pages=4)
    got = H.run_trace(runner, H.trace_tail(seqs, tail=230))
    assert runner.graph_replays > 100
    L.compare(got, cfg, weights, seqs, **TOL[dtype])


def test_a_slot_that_is_used_again_starts_from_nothing(model):
    name, made = model
    weights, folder, cfg = made["float32"]
    seqs = sequences(cfg, [130, 75], seed=90)
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
    seqs = sequences(cfg, [60, 3, 41, 1], seed=120)
    runner = make_runner(folder, "float32", n_pages=8)
    alone = H.run_trace(runner, H.trace_whole(seqs))
    together = H.run_trace(runner, [{"step": 0, "entries": [{"id": r, "tokens": ids, "want": list(range(len(ids)))} for r, ids in seqs.items()],
                                     "end": list(seqs)}])
    for key, row in alone.items():
        assert float((row - together[key]).abs().max()) < 1e-5 * (1.0 + float(row.abs().max())), f"{key} differs beside other requests"
    L.compare(together, cfg, weights, seqs, **TOL["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_tokens_in_a_step_beside_decoded_ones(model, dtype):
    """A portion of 290 tokens beside a decoded token (the recurrence in pieces side by side; attention, gates and experts on tensor cores
    where the sizes allow, in bfloat16); then the same request goes on token by token from the states and pages that step left."""
    name, made = model
    weights, folder, cfg = made[dtype]
    seqs = sequences(cfg, [320, 80], seed=140)
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


def test_a_dozen_requests_decoding_at_once(model):
    """More than eight tokens in a one-token step (the recurrence's kernel takes eight a block; experts in tiles), in a captured step and
    beside each other, in both types."""
    name, made = model
    for dtype in ("float32", "bfloat16"):
        weights, folder, cfg = made[dtype]
        seqs = sequences(cfg, [9 + i for i in range(12)], seed=160)
        runner = make_runner(folder, dtype, n_pages=12, slots=12)
        reqs = {r: runner.open(r) for r in seqs}
        got, at = {}, {}
        for r, ids in seqs.items():
            runner.step([(reqs[r], ids[:-6], [])])
            at[r] = len(ids) - 6
        for _ in range(6):
            rows = runner.step([(reqs[r], [ids[at[r]]], [0]) for r, ids in seqs.items()]).float().cpu()
            for i, r in enumerate(seqs):
                got[(r, at[r])] = rows[i]
                at[r] += 1
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
            row = L.oracle_logits(cfg, weights, prompt + got[:i])[-1]
            gap = float(row.max() - row[tok])
            bound = 1e-4 if dtype == "float32" else 5e-2 * float(row.abs().max())
            assert gap <= bound, f"{dtype}: token {i} is {tok}, the plain model prefers {int(row.argmax())} by {gap:.3g}"
    if dtype == "float32":
        assert solo == outs[0]


@pytest.mark.parametrize("name,dtype", [("looped", "float32"), ("looped", "bfloat16"), ("odd", "bfloat16"), ("wide_heads", "bfloat16"), ("big_cells", "float32")])
def test_trace_run_as_a_process(name, tmp_path, dtype):
    """bin/trace_run as a process on a mixed trace with two live requests and four pages; a step that wants nothing writes no file."""
    cfg = L.CONFIGS[name]
    weights = L.random_weights(cfg, seed=13)
    folder = L.write_folder(tmp_path / "m", cfg, weights)
    seqs = sequences(cfg, [70, 20, 131], seed=310)
    trace = H.trace_mixed(seqs, max_tokens=64 * 4, seed=2, max_live=2)
    for e in trace[1]["entries"]:
        e["want"] = []
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
        assert (out / f"{st['step']}.f32").exists() == (wanted > 0)
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


def test_command_line_generates_with_the_folders_architecture(tmp_path):
    cfg = L.LOOPED
    weights = L.random_weights(cfg, seed=13)
    folder = L.write_folder(tmp_path / "m", cfg, weights)
    prompt = H.random_ids(19, cfg["vocab"], 400)
    proc = subprocess.run([sys.executable, "-m", "lgml_b200", "-m", str(folder), "--dtype", "float32", "-c", "128", "--prompt-ids", ",".join(map(str, prompt)),
                           "-n", "5", "--temperature", "0", "--repeat-stop", "0"], capture_output=True, text=True, timeout=600, cwd=str(ROOT))
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = [int(t) for t in proc.stdout.strip().splitlines()[-1].split(",")]
    assert len(got) == 5
    for i, tok in enumerate(got):
        row = L.oracle_logits(cfg, weights, prompt + got[:i])[-1]
        assert float(row.max() - row[tok]) <= 1e-4


def test_random_weights_mode_draws_the_written_folder(tmp_path):
    """A configuration alone is enough: the engine draws weights of the shapes and kinds the parts ask for, the integer tables too, and they are
    those of the folder that the same seed writes."""
    from lgml_b200.config import config_from_dict
    from lgml_b200.engine.runner import ModelRunner
    from lgml_b200.weights import write_random_model

    cfg = config_from_dict(L.LOOPED)
    folder = write_random_model(tmp_path / "m", cfg, seed=3, dtype="bfloat16")
    ids = H.random_ids(70, 97, 1)
    rows = []
    for runner in (ModelRunner.from_config(cfg, seed=3, dtype=torch.bfloat16, n_pages=4, max_slots=2), make_runner(folder, "bfloat16", 4, slots=2)):
        rows.append(runner.step([(runner.open("a"), ids, [0, 69])]))
        runner.rt.check_status()
    assert rows[0].shape == (2, 97) and bool(torch.isfinite(rows[0]).all()) and torch.equal(rows[0], rows[1])


def test_parts_of_the_design_in_another_arrangement(tmp_path):
    """The mechanisms as parts of a block that is not this design's: a pre-norm layer with a learned sink and a gate per head; a parallel block
    whose feed-forward is a dense one."""
    from lgml_b200.cache import PagedKV
    from lgml_b200.parts import make_part

    att = make_part("mixer", "sink_attention", width=32, n_heads=2, n_kv_heads=1, head_dim=16, v_head_dim=16, scale=0.25, gate="head", slope_base=8.0)
    assert att.cache_spec() == PagedKV(1, 16, None, 16) and {s.name for s in att.tensor_specs("m")} >= {"m.sink", "m.g"} and att.gate_cols == 2
    rt = runtime(torch.float32)
    dense = make_part("feed_forward", "clamped_glu", width=32, inner=24, limit=1.0)
    block = make_part("block", "parallel", norm=make_part("norm", "rmsnorm", width=32, eps=1e-5, suffix=""), mixer=make_part("mixer", "rglru", width=32, inner=16, blocks=2, taps=2),
                      ffn=dense, width=32, names={"scale1": "s1", "scale2": "s2"})
    specs = {s.name: s for s in block.tensor_specs("b")}
    assert {"b.s1", "b.s2", "b.mlp.gate", "b.mix.lam"} <= set(specs)
    from lgml_b200.weights import random_tensors

    tensors = {n: t.to(DEV) for n, t in random_tensors(specs.values(), seed=5, std=0.3).items()}
    host = {n: t.double().cpu().numpy() for n, t in tensors.items()}
    block.bind("b", tensors, rt)
    from lgml_b200 import ops
    from lgml_b200.engine.batch import CacheView

    rng = np.random.default_rng(1)
    x = np.float32(rng.normal(size=(9, 32))).astype(np.float64)
    step = Step(0, 9)
    step.seq_start, step.slots = i32([0, 9]), i32([0])
    xd = f32(x)
    state = torch.zeros((1, *block.cache_spec().shape), device=DEV)
    _, pending = block.forward(rt, xd, None, step, CacheView(state=state))
    ops.scaled_norm(xd, pending.terms)
    h = P.rms_norm(x, host["b.norm1"], 1e-5)
    want = x + host["b.s1"] * P.rglru(h, {k[2:]: v for k, v in host.items()}, "mix", None) + host["b.s2"] * P.clamped_expert(h, host, "b.mlp", 1.0)
    assert worst(xd, want) < 3e-5
