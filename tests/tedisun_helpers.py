"""Test material for the Tedisun design: small configurations that differ from each other in every size and
option, random weights made so that the mechanisms show, and the oracle."""
from __future__ import annotations

import json
import random
from pathlib import Path
from typing import Dict, List, Tuple

import numpy as np
import torch

from tests.plain import tedisun_plain as P


def moe(ff, experts, top, identity=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, scale, base=10000.0, dims=None, scaling=None, size=None, keep_first=0):
    rot = {"base": base, "dims": dim if dims is None else dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep_first}
    return m


def right(heads, dim, vdim, gate_cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def parallel(l, r, scales=(1.0, 1.0), mlp=None):
    return {"type": "parallel", "mixer": {"left": l, "right": r, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def config(vocab, width, streams, layers, eps=1e-5, scale=None, softcap=None):
    cfg = {"architecture": "Tedisun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    return cfg


# Three streams, layers that differ in every size, values longer and shorter than keys, windows of 29 and 64 with 0 and 3
# kept first tokens, a layer without a feed-forward, more experts than a token's row of a warp, convolutions of 2 and 3 taps.
MIXED = config(97, 72, 3, [
    delta(4, 2, 24, 20, 3, moe(40, 5, 2, 1)),
    parallel(left(6, 2, 32, 24, 0.2, base=5000.0, dims=8, scaling=(4.0, 1.0, 4.0, 64), size=29, keep_first=3), right(3, 16, 28, 8.0), (0.7, 1.6), None),
    delta(2, 2, 48, 64, 2, moe(24, 37, 4, 3)),
    parallel(left(2, 1, 48, 80, 0.15, base=300.0, dims=48, size=64), right(2, 40, 8, 20.0), (-1.1, 0.9), moe(72, 3, 3, 2)),
], eps=1e-5, scale=3.0, softcap=20.0)

# One stream, sizes that are no multiple of 8 or of 4, one head, one expert, no identity experts, one tap, a window of one
# token, no cap and no embedding scale.
ODD = config(61, 37, 1, [
    parallel(left(3, 3, 10, 7, 0.35, base=77.0, dims=6, size=1, keep_first=2), right(1, 5, 9, 5.0), (1.3, 0.4), moe(21, 1, 1)),
    delta(3, 1, 9, 13, 1, moe(30, 4, 1, 0)),
    parallel(left(5, 1, 12, 12, 0.3, base=900.0, dims=2, scaling=(2.0, 0.5, 2.0, 40)), right(4, 12, 6, 9.0), (1.0, 1.0), moe(18, 6, 5)),
], eps=3e-6)

# Heads of 64 and 128 entries (the tcgen05 prompt attention in bfloat16), windows across pages with kept first tokens that
# end inside a page and behind one, four streams, experts wide enough for grouped tiles.
WIDE_HEADS = config(103, 96, 4, [
    parallel(left(4, 2, 64, 64, 0.11, base=150000.0, dims=24, scaling=(6.0, 1.0, 4.0, 128), size=70, keep_first=5), right(2, 64, 64, 15.0), (1.5, 0.6),
             moe(64, 8, 2, 1)),
    delta(3, 3, 64, 128, 4, moe(48, 12, 3, 4)),
    parallel(left(2, 1, 128, 128, 0.09, base=20000.0, dims=64, size=33, keep_first=67), right(1, 128, 96, 6.0), (0.8, 0.8), moe(80, 6, 2, 2)),
], eps=1e-6, scale=5.0, softcap=50.0)

# No paged layer at all: every layer is a recurrence; two streams; convolutions of 4, 5 and 8 taps.
ALL_DELTA = config(83, 96, 2, [
    delta(6, 3, 16, 32, 5, moe(32, 7, 2, 1)), delta(1, 1, 100, 44, 8), delta(8, 2, 24, 8, 4, moe(16, 4, 4)),
], eps=1e-5, scale=4.0, softcap=9.0)

CONFIGS = {"mixed": MIXED, "odd": ODD, "wide_heads": WIDE_HEADS, "all_delta": ALL_DELTA}


def random_weights(cfg: dict, seed: int, sharpen: float = 1.0, calm: bool = False) -> Dict[str, torch.Tensor]:
    """Weights as bfloat16-representable float32 tensors, scaled so that no mechanism is lost in the noise: attention far from
    uniform, sinks that weigh as much as a key, decays so slow that a state from hundreds of tokens back still counts,
    input gates of both signs, streams that differ.  ``calm`` (for runs in bfloat16): the routers' corrections lie evenly
    apart, which makes close choices rare, and the input gates stay so low that a normaliser near zero is rare too."""
    g = torch.Generator().manual_seed(seed)
    E, R = cfg["width"], cfg["streams"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def vec(n, sd, mean=0.0):
        return torch.randn(n, generator=g) * sd + mean

    def conv(c, taps):
        return torch.randn(c, taps, generator=g) * 0.5 + torch.eye(taps)[-1] * 0.7

    w = {"embed": torch.randn(cfg["vocab"], E, generator=g) * 0.5, "head": mat(cfg["vocab"], E, 2.0), "final.norm": vec(E, 0.2)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer.get("mlp") else (1,):
            w[f"{p}norm{q}"] = vec(E, 0.2)
            w[f"{p}rg{q}"], w[f"{p}rg{q}.b"] = mat(E, E), vec(E, 0.5, 1.0)
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = vec(R, 0.4, 1.0 / R ** 0.5), vec(R, 0.4, 1.0)
            w[f"{p}hc{q}.mix"] = torch.eye(R) * 0.8 + torch.randn(R, R, generator=g) * 0.25
        q = p + "mix."
        if layer["type"] == "delta":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                w[q + n], w[q + n + ".conv"] = mat(rows, E, 1.2), conv(rows, m["conv"])
            w[q + "b"], w[q + "a"] = mat(H, E, 1.5), mat(H, E)
            w[q + "A_log"], w[q + "dt_bias"] = vec(H, 1.0, -2.5), vec(H, 1.0, -2.0)
            w[q + "norm"], w[q + "g"], w[q + "o"] = vec(Dv, 0.2, 1.0), mat(H * Dv, E), mat(E, H * Dv)
        else:
            l, r = m["left"], m["right"]
            H, G, D, Dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                w[q + "left." + n], w[q + "left." + n + ".b"] = mat(rows, E), vec(rows, 0.3)
            w[q + "left.q.norm"], w[q + "left.k.norm"] = vec(D, 0.2, 1.1 * sharpen), vec(D, 0.2, 1.1 * sharpen)
            w[q + "left.sink"] = vec(H, 1.5)
            w[q + "left.o"], w[q + "left.o.b"] = mat(E, H * Dv), vec(E, 0.2)
            H, D, Dv = r["heads"], r["dim"], r["vdim"]
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                w[q + "right." + n] = mat(rows, E)
            w[q + "right.o"], w[q + "right.norm"] = mat(E, H * Dv), vec(H * Dv, 0.2, 1.0)
            w[q + "right.i"], w[q + "right.i.b"] = mat(H, E, 0.7 if calm else 2.0), vec(H, 0.5 if calm else 1.0, -2.0 if calm else -1.0)
            w[q + "right.f"], w[q + "right.f.b"] = mat(H, E), vec(H, 1.5, 4.0)
        if layer.get("mlp"):
            F, rt = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]
            X = rt["experts"] + rt.get("identity", 0)
            q = p + "mlp."
            w[q + "router"], w[q + "correction"] = mat(X, E, 2.5), (torch.randperm(X, generator=g) * 0.08 if calm else vec(X, 0.1))
            for e in range(rt["experts"]):
                w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = mat(F, E, 1.5), mat(F, E, 1.5), mat(E, F, 1.0 if calm else 2.0)
    return {n: t.to(torch.bfloat16).float() for n, t in w.items()}


def calm(cfg: dict) -> dict:
    """The configuration for runs in bfloat16: the layers' eps so large that a recurrence's read-out of almost nothing is not
    blown up to unit size with the rounding it carries."""
    return dict(cfg, norm={"eps": 2e-2})


def write_folder(folder: Path, cfg: dict, weights: Dict[str, torch.Tensor]) -> Path:
    """config.json and model.safetensors (bfloat16) of a model."""
    from lgml_b200.weights import write_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {n: t.to(torch.bfloat16) for n, t in weights.items()})
    return folder


_oracle: Dict[Tuple[int, Tuple[int, ...]], torch.Tensor] = {}
_numpy: Dict[int, Tuple[dict, Dict[str, np.ndarray]]] = {}


def numpy_of(weights):
    if id(weights) not in _numpy:
        _numpy[id(weights)] = (weights, {n: t.double().numpy() for n, t in weights.items()})
    return _numpy[id(weights)][1]


def oracle_logits(cfg: dict, weights: Dict[str, torch.Tensor], ids: List[int]) -> torch.Tensor:
    numpy_of(weights)           # (keeps the weights, whose id is the key, alive)
    key = (id(weights), tuple(ids))
    if key not in _oracle:
        _oracle[key] = torch.from_numpy(P.forward(cfg, numpy_of(weights), list(ids)))
    return _oracle[key]


def clear_ids(cfg: dict, weights: Dict[str, torch.Tensor], n: int, seed: int, gap: float = 0.02) -> List[int]:
    """n random token ids on which no router of the plain model decides by less than ``gap``: a flipped choice is a
    discrete change that rounding is allowed to cause.  The model is causal, so the first such position is redrawn and
    the sequence looked at again."""
    rng = random.Random(seed)
    ids = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    for _ in range(40 * n):
        margins: list = []
        P.forward(cfg, numpy_of(weights), ids, margins=margins)
        close = np.nonzero(np.min(np.stack(margins), axis=0) < gap)[0] if margins else np.zeros(0, int)
        if close.size == 0:
            return ids
        for p in close[:1]:
            ids[int(p)] = rng.randrange(cfg["vocab"])
    raise AssertionError("no sequence without a close call was found")


def compare(got: Dict[Tuple[str, int], torch.Tensor], cfg, weights, seqs: Dict[str, List[int]], atol: float, rtol: float) -> float:
    """Largest error over all rows that ``got`` holds; raises naming the first wrong (request, position)."""
    worst = 0.0
    for rid, ids in seqs.items():
        ref = oracle_logits(cfg, weights, ids)
        for p in range(len(ids)):
            if (rid, p) not in got:
                continue
            row = got[(rid, p)].double()
            err = (row - ref[p]).abs()
            bound = atol + rtol * ref[p].abs().max()
            if bool((err > bound).any()):
                j = int(err.argmax())
                raise AssertionError(f"request {rid} position {p} (page {p // 64}, cell {p % 64}): logit {j} is {row[j]:.6g}, "
                                     f"oracle {ref[p, j]:.6g}, |diff| {err[j]:.3g} > {bound:.3g}")
            worst = max(worst, float(err.max()))
    return worst
