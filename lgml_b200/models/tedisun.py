"""The Tedisun decoder: which parts a ``TedisunConfig`` asks for, layer by layer.

The residual is several streams that all start as the embedding's rows times ``embedding.scale``; every sublayer reads a
weighted sum of them through an RMS norm whose stored weight is the distance from one, its result passes a sigmoid gate,
and all streams are made anew from the old ones and that result (``parts/streams.py``: ``HyperBlock``).  A layer's mixer is
either the gated delta rule with one decay per head (``parts/delta.py``: ``HeadDelta``) or two mixers side by side
(``parts/parallel.py``: ``SummedMixers``): attention with normed heads, a sink and a sliding window that keeps the first
tokens (``NormedAttention``), and a matrix memory with exponential gates (``MatrixMemory``).  The feed-forward is a mixture
of experts with softmax scores over all experts, some of which return their input (``parts/moe.py``).

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``, ``l<i>.rg1``, ``l<i>.rg2`` (and ``.b``),
``l<i>.mix.*`` (``l<i>.mix.left.*``, ``l<i>.mix.right.*``), ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import torch

from ..config import RopeScaling, TedisunConfig, register_architecture
from ..parts import LMHead, ResultGate, TokenEmbedding, make_part
from .decoder import DecoderModel


def rotation_of(dim: int, rot: dict):
    sc = rot.get("scaling")
    scaling = RopeScaling(rope_type="llama3", factor=sc["factor"], low_freq_factor=sc["low"], high_freq_factor=sc["high"],
                          original_max_position_embeddings=sc["original"]) if sc else None
    return make_part("position", "rope", head_dim=dim, theta=rot["base"], scaling=scaling, n_rot=rot["dims"])


def mixer_of(cfg: TedisunConfig, layer: dict):
    m = layer["mixer"]
    if layer["type"] == "delta":
        return make_part("mixer", "head_delta", width=cfg.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                         taps=m["conv"], eps=cfg.norm_eps)
    left, right = m["left"], m["right"]
    mask = left.get("mask") or {}
    attention = make_part("mixer", "normed_attention", width=cfg.width, n_heads=left["heads"], n_kv_heads=left["kv_heads"], head_dim=left["dim"],
                          v_head_dim=left["vdim"], scale=left["scale"], position=rotation_of(left["dim"], left["rot"]), eps=cfg.norm_eps,
                          window=mask.get("size"), keep_first=mask.get("keep_first", 0))
    memory = make_part("mixer", "matrix_memory", width=cfg.width, n_heads=right["heads"], head_dim=right["dim"], v_head_dim=right["vdim"],
                       gate_cap=right["gate_cap"], eps=cfg.norm_eps)
    return make_part("mixer", "summed", width=cfg.width, left=attention, right=memory, left_scale=m["left_scale"], right_scale=m["right_scale"])


def feed_forward_of(cfg: TedisunConfig, mlp):
    if mlp is None:
        return None
    r = mlp["router"]
    return make_part("feed_forward", "routed_experts", width=cfg.width, inner=mlp["expert"]["ff"], n_experts=r["experts"], top=r["top"],
                     router="softmax_all", n_identity=r.get("identity", 0), bias_name=".correction", router_rows=True)


def build_tedisun(cfg: TedisunConfig) -> DecoderModel:
    norm = lambda: make_part("norm", "stream_rmsnorm", width=cfg.width, eps=cfg.norm_eps, suffix="", one_plus=True)
    blocks = []
    for layer in cfg.layers:
        ffn = feed_forward_of(cfg, layer.get("mlp"))
        blocks.append(make_part("block", "hyper", streams=cfg.streams, mixer_norm=norm(), mixer=mixer_of(cfg, layer), mixer_gate=ResultGate(cfg.width),
                                ffn_norm=norm() if ffn else None, ffn=ffn, ffn_gate=ResultGate(cfg.width) if ffn else None))
    embedding = TokenEmbedding(cfg.vocab, cfg.width, name="embed")
    head = LMHead(cfg.vocab, cfg.width, name="head")
    return DecoderModel(cfg, embedding, blocks, norm(), head, block_prefix="l{}", final_norm_prefix="final.norm", streams=cfg.streams,
                        embed_scale=cfg.embed_scale if cfg.embed_scale != 1.0 else None, logit_softcap=cfg.logit_softcap, delta_dtype=torch.float32)


register_architecture("Tedisun", TedisunConfig, build_tedisun)
