"""Test material for the Nelosun design: small configurations that differ from each other in every size
and option, random weights made so that the mechanisms show, and the oracle."""
from __future__ import annotations

import json
import math
from pathlib import Path
from typing import Dict, List, Tuple

import numpy as np
import torch

from tests.plain import nelosun_plain as P


def moe(ff, experts, top, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attention(heads, kv_heads, dim, vdim, scale, temp=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        m["q_temp"] = dict(zip(("coef", "every"), temp))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, rank, scale, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank,
                                                  "scale": scale, "rot": {"base": base, "dims": rot_dim}}, "mlp": mlp}


def rglru(width, blocks, taps, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": taps}, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, scale=None, loop=None):
    cfg = {"architecture": "Nelosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A loop in the middle that runs three times over a latent and a recurrent layer; values longer than keys; a layer without a
# feed-forward inside the loop; a recurrence narrower than the model; attention with and without a temperature.
LOOPED = config(97, 64, [
    attention(6, 2, 16, 24, 0.3, temp=(0.7, 13), mlp=moe(24, 5, 2, 0.9)),
    latent(3, 16, 8, 12, 20, 24, 0.25, base=5000.0),
    rglru(48, 3, 4, mlp=moe(16, 3, 1, 1.2)),
    attention(2, 2, 24, 8, 0.25, mlp=moe(40, 4, 4, 0.6)),
], eps=1e-5, scale=3.0, loop=(1, 3, 3))

# One head, widths that are no multiple of 8 or of 4, one expert, one tap, parts of 7 channels, no loop, no scale.
ODD = config(61, 37, [
    rglru(21, 3, 7, mlp=moe(10, 1, 1, 0.7)),
    attention(3, 1, 10, 5, 0.4, temp=(1.3, 1), mlp=moe(19, 6, 3, 5.0)),
    latent(1, 6, 2, 9, 11, 10, 0.4, base=77.0, mlp=moe(8, 2, 1, 0.5)),
    rglru(37, 1, 1),
], eps=3e-6)

# A loop over all layers from the first on; the recurrence first; every expert for every token; wider than the model.
ALL_LOOP = config(83, 48, [
    rglru(96, 2, 2, mlp=moe(16, 3, 3, 1.0)),
    latent(4, 8, 8, 8, 24, 16, 0.3, base=1000.0, mlp=moe(24, 7, 2, 0.8)),
    attention(4, 4, 8, 16, 0.35, temp=(-0.2, 40), mlp=moe(32, 9, 1, 1.5)),
], eps=1e-6, scale=0.5, loop=(0, 3, 2))

# Head sizes the tcgen05 and tensor-core split kernels take (64 and 128), cells of 128 and 64 numbers, parts of 64 channels, a loop
# at the end that runs once.
WIDE_HEADS = config(101, 96, [
    attention(4, 2, 64, 64, 0.12, temp=(0.4, 50), mlp=moe(40, 8, 2, 1.1)),
    latent(4, 32, 32, 32, 48, 96, 0.12, base=30000.0, mlp=moe(32, 4, 1, 0.9)),
    attention(8, 1, 128, 128, 0.09, mlp=moe(48, 12, 3, 2.0)),
    rglru(128, 2, 3, mlp=moe(16, 2, 2, 1.0)),
    latent(2, 64, 16, 64, 16, 48, 0.1, base=500.0),
], eps=1e-5, scale=2.0, loop=(2, 5, 1))

# Cells wider than any split kernel takes (288 and 544 numbers), a loop of one layer, more experts than tokens in most steps.
BIG_CELLS = config(211, 72, [
    latent(2, 16, 16, 16, 40, 272, 0.2, base=10000.0, mlp=moe(16, 40, 2, 0.8)),
    rglru(80, 5, 5, mlp=moe(24, 3, 2, 1.0)),
    latent(2, 24, 32, 8, 24, 512, 0.12, base=2000.0, mlp=moe(8, 5, 5, 1.0)),
], eps=1e-5, scale=1.0, loop=(0, 1, 4))

CONFIGS = {"looped": LOOPED, "odd": ODD, "all_loop": ALL_LOOP, "wide_heads": WIDE_HEADS, "big_cells": BIG_CELLS}


def random_weights(cfg: dict, seed: int, sharpen: float = 1.0) -> Dict[str, torch.Tensor]:
    """Weights as bfloat16-representable float32 tensors (the tables int32), scaled so that no mechanism is lost in the noise: attention far
    from uniform (``sharpen`` more so), head gates on both sides, decays from nearly nothing to nearly one, experts whose clamps are
    reached, channel scales away from one, tables whose rows differ."""
    g = torch.Generator().manual_seed(seed)
    E = cfg["width"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def vec(n, sd, mean=0.0):
        return torch.randn(n, generator=g) * sd + mean

    w = {"embed": torch.randn(cfg["vocab"], E, generator=g) / cfg.get("embedding", {}).get("scale", 1.0), "final.norm": vec(E, 0.2, 1.0)}
    if cfg.get("loop"):
        w["loop.in"] = torch.cat([mat(E, E, 0.9), mat(E, E, 0.5)], dim=1)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        w[p + "norm1"], w[p + "ls1"] = vec(E, 0.2, 1.0), vec(E, 0.3, 0.7)
        if layer["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w[p + "mix.q"], w[p + "mix.q.b"] = mat(H * D, E, 1.2 * sharpen), vec(H * D, 0.5)
            w[p + "mix.k"], w[p + "mix.k.b"] = mat(G * D, E, 1.2 * sharpen), vec(G * D, 0.5)
            w[p + "mix.v"], w[p + "mix.v.b"] = mat(G * Dv, E, 1.2), vec(G * Dv, 0.5)
            w[p + "mix.g"] = mat(H, E, 2.0)
            w[p + "mix.o"], w[p + "mix.o.b"] = mat(E, H * Dv, 1.5), vec(E, 0.3)
        elif layer["type"] == "latent_attention":
            H, D, Dr, Dv, Rq, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            w[p + "mix.dq"], w[p + "mix.dq.norm"] = mat(Rq, E), vec(Rq, 0.2, 1.0)
            w[p + "mix.uq"] = mat(H * (D + Dr), Rq, 1.3 * sharpen)
            w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = mat(R + Dr, E, 1.2), vec(R, 0.2, 1.0)
            w[p + "mix.uk"], w[p + "mix.uv"] = mat(H * D, R, 1.3), mat(H * Dv, R, 1.3)
            w[p + "mix.o"] = mat(E, H * Dv)
        else:
            C, B = m["width"], m["blocks"]
            n = C // B
            w[p + "mix.y"], w[p + "mix.y.b"] = mat(C, E, 1.5), vec(C, 0.5)
            w[p + "mix.x"], w[p + "mix.x.b"] = mat(C, E, 1.2), vec(C, 0.3)
            w[p + "mix.conv"], w[p + "mix.conv.b"] = torch.randn(C, m["conv"], generator=g) * 0.6, vec(C, 0.3)
            w[p + "mix.ra"], w[p + "mix.ri"] = (torch.randn(B, n, n, generator=g) * 1.5 / n ** 0.5 for _ in range(2))
            w[p + "mix.ra.b"], w[p + "mix.ri.b"] = vec(B * n, 0.5).reshape(B, n), vec(B * n, 0.5).reshape(B, n)
            w[p + "mix.lam"] = torch.rand(C, generator=g) * 8.0 - 8.0          # softplus from 3e-4 (a remembers hundreds of tokens) to 0.7
            w[p + "mix.o"] = mat(E, C, 1.5)
        f = layer.get("mlp")
        if f:
            F, X, top = f["expert"]["ff"], f["router"]["experts"], f["router"]["top"]
            w[p + "ls2"] = vec(E, 0.3, 0.7)
            for e in range(X):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"] = mat(F, E, 1.2), mat(F, E, 1.2)
                w[f"{p}mlp.e{e}.down"] = mat(E, F, 1.0 + 0.3 * (e % 3))
            w[p + "mlp.table"] = torch.stack([torch.randperm(X, generator=g)[:top] for _ in range(cfg["vocab"])]).to(torch.int32)
    return {n: t if t.dtype == torch.int32 else t.to(torch.bfloat16).float() for n, t in w.items()}


def write_folder(folder: Path, cfg: dict, weights: Dict[str, torch.Tensor]) -> Path:
    """config.json and model.safetensors (bfloat16, the tables int32) of a model."""
    from lgml_b200.weights import write_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {n: t if t.dtype == torch.int32 else t.to(torch.bfloat16) for n, t in weights.items()})
    return folder


_oracle: Dict[Tuple[int, Tuple[int, ...]], torch.Tensor] = {}
_numpy: Dict[int, Dict[str, np.ndarray]] = {}
_alive: list = []           # weights whose ids key the caches above


def with_scale(cfg: dict) -> dict:
    """The configuration with the keys that it leaves to their defaults."""
    return {**cfg, "embedding": cfg.get("embedding", {"scale": 1.0})}


def numpy_of(weights):
    if id(weights) not in _numpy:
        _alive.append(weights)
        _numpy[id(weights)] = {n: t.numpy() if t.dtype == torch.int32 else t.double().numpy() for n, t in weights.items()}
    return _numpy[id(weights)]


def oracle_logits(cfg: dict, weights: Dict[str, torch.Tensor], ids: List[int]) -> torch.Tensor:
    key = (id(weights), tuple(ids))
    if key not in _oracle:
        _oracle[key] = torch.from_numpy(P.forward(with_scale(cfg), numpy_of(weights), list(ids)))
    return _oracle[key]


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
            if bool((err > bound).any()) or not bool(torch.isfinite(row).all()):
                j = int(err.argmax())
                raise AssertionError(f"request {rid} position {p} (page {p // 64}, cell {p % 64}): logit {j} is {row[j]:.6g}, "
                                     f"oracle {ref[p, j]:.6g}, |diff| {err[j]:.3g} > {bound:.3g}")
            worst = max(worst, float(err.max()))
    return worst
