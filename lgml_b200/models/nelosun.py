"""The Nelosun decoder: which parts a ``NelosunConfig`` asks for, layer by layer.

The embedding's rows times ``embedding.scale`` are the residual stream x.  Every layer is a ``ParallelBlock``: one RMS norm that both
sublayers read, x += ls1 mixer(h) + ls2 ff(h), the scales channel by channel.  The mixer is chosen per layer by ``type``:
``attention`` (``parts/sink_attention.py``: grouped heads with biases, a temperature on the queries, a one in the softmax's
denominator and a gate of one number per head), ``latent_attention`` (``parts/latent_attention.py``: queries and keys / values each through a
latent) or ``rglru`` (``parts/rglru.py``: a real-gated linear recurrent unit behind a short convolution).  The feed-forward is a mixture
of experts that a table names by the token's id (``parts/table_experts.py``).

``loop`` runs a range of layers several times with the same weights; every run of a layer is a schedule entry with a cache and
state of its own, and before the first layer of every pass x becomes W_in [x; the embedding's output] (``PassInput``).  The logits are
products with the embedding's table, without its scale.

Tensor names: ``embed``, ``loop.in``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.ls1``, ``l<i>.ls2``, ``final.norm``.
"""
from __future__ import annotations

import torch

from ..config import NelosunConfig, register_architecture
from ..parts import LMHead, TableRouting, TokenEmbedding, make_part
from .decoder import DecoderModel, LayerCall


def mixer_of(cfg: NelosunConfig, layer: dict):
    m = layer["mixer"]
    if layer["type"] == "attention":
        temp = m.get("q_temp")
        return make_part("mixer", "sink_attention", width=cfg.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                         scale=m["scale"], temperature=(temp["coef"], temp["every"]) if temp else None, slope_base=None, sink=0.0, gate="head", bias=True,
                         out_bias=True)
    if layer["type"] == "latent_attention":
        return make_part("mixer", "latent_attention", width=cfg.width, n_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
                         rank=m["kv_rank"], scale=m["scale"], eps=cfg.norm_eps, rope_base=m["rot"]["base"], rope_dims=m["rot"]["dims"], q_rank=m["q_rank"],
                         halves=True)
    return make_part("mixer", "rglru", width=cfg.width, inner=m["width"], blocks=m["blocks"], taps=m["conv"])


def build_nelosun(cfg: NelosunConfig) -> DecoderModel:
    norm = lambda: make_part("norm", "rmsnorm", width=cfg.width, eps=cfg.norm_eps, suffix="")
    routing = TableRouting()

    def feed_forward_of(mlp):
        if mlp is None:
            return None
        return make_part("feed_forward", "table_experts", width=cfg.width, inner=mlp["expert"]["ff"], n_experts=mlp["router"]["experts"],
                         top=mlp["router"]["top"], vocab=cfg.vocab, limit=mlp["expert"]["limit"], routing=routing)

    blocks = [make_part("block", "parallel", norm=norm(), mixer=mixer_of(cfg, layer), ffn=feed_forward_of(layer.get("mlp")), width=cfg.width)
              for layer in cfg.layers]
    embedding = TokenEmbedding(cfg.vocab, cfg.width, name="embed")
    pass_input = make_part("token_input", "pass_input", width=cfg.width, embedding=embedding, scale=cfg.embed_scale) if cfg.loop else None
    return DecoderModel(cfg, embedding, blocks, norm(), LMHead(cfg.vocab, cfg.width, tied_to=embedding, name="head"),
                        schedule=[LayerCall(i, begins_pass=number) for i, number in cfg.layer_runs()], block_prefix="l{}", final_norm_prefix="final.norm",
                        embed_scale=cfg.embed_scale if cfg.embed_scale != 1.0 else None, delta_dtype=torch.float32, pass_input=pass_input,
                        step_parts=[routing])


register_architecture("Nelosun", NelosunConfig, build_nelosun)
