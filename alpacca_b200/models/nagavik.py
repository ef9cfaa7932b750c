"""The Nagavik decoder, put together from the parts.

The stream starts as embedded tokens times a factor plus learned positions.  Every sub-layer has a norm before and a norm
after it, and what joins the stream is scaled column by column (taken into the weight of the norm after the sub-layer when
that is loaded).  A layer's mixer is a state-space mixer with one decay and one step size per head, or grouped attention with
a query/key norm over the whole projection, no rotation, scores bounded by a tanh, a penalty that grows linearly with
distance (a slope per head) and one added to the softmax's denominator.  The feed-forward is a gated one (tanh-GELU, biases),
or experts without gates (squared ReLU) chosen by sigmoid scores that multiply the experts' inputs, beside a shared expert.
The logits are bounded by a tanh.

Tensor names (matrices [out, in], named by their prefix alone):
    embed, pos, final.norm, head, l<i>.norm1, l<i>.norm1b, l<i>.ls1, l<i>.norm2, l<i>.norm2b, l<i>.ls2
    l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}                                         mamba2
    l<i>.mix.{q,k,v,o,q.norm,k.norm}                                                         attention
    l<i>.mlp.{gate,gate.b,up,up.b,down,down.b}                                               dense
    l<i>.mlp.router, l<i>.mlp.e<j>.{up,down}, l<i>.mlp.shared.{up,down}                      moe
"""
from __future__ import annotations

import torch

from ..config.nagavik import NagavikConfig
from ..config.registry import register_architecture
from ..engine.model import DecoderSpec
from ..parts import (BuildOptions, MapsAttention, PositionTable, RMSNorm, SandwichBlock, ScoredExperts, StateSpaceMixer,
                     SwiGLU, TokenEmbedding, VocabHead, alibi_slopes)


@register_architecture("Nagavik", NagavikConfig)
def build_nagavik(cfg: NagavikConfig, opts: BuildOptions) -> DecoderSpec:
    E, eps = cfg.width, cfg.eps

    def norm(name, columns=None):
        return RMSNorm(opts, E, eps, name, weight_suffix="", columns=columns)

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, mx = f"l{i}", layer["mixer"]
        # the sub-layers' outputs are normed right away: they leave their last product in float32
        if layer["type"] == "mamba2":
            mixer = StateSpaceMixer(opts, E, mx["heads"], mx["vdim"], mx["state"], mx["groups"], mx["conv"], mx["norm_groups"],
                                    eps, f"{p}.mix", out_dtype=torch.float32)
        else:
            mixer = MapsAttention(opts, E, mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], None, f"{p}.mix", mx["scale"], eps,
                                  qk_norm=True, qk_norm_rows=True, softcap=mx.get("softcap"), slopes=alibi_slopes(mx["heads"]),
                                  fixed_sink=0.0, out_dtype=torch.float32)
        mlp = layer.get("mlp")
        if mlp is None:
            layers.append(SandwichBlock(norm(f"{p}.norm1"), mixer, norm(f"{p}.norm1b", f"{p}.ls1")))
            continue
        if mlp["kind"] == "dense":
            ffn = SwiGLU(opts, E, mlp["ff"], f"{p}.mlp", bias=True, names=("gate", "up", "down"), weight_suffix="",
                         bias_suffix=".b", activation="gelu_tanh", out_dtype=torch.float32)
        else:
            shared = mlp.get("shared")
            ffn = ScoredExperts(opts, E, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"], f"{p}.mlp",
                                activation="relu2", score="sigmoid", weight_in=True, shared_inner=shared["ff"] if shared else 0)
        layers.append(SandwichBlock(norm(f"{p}.norm1"), mixer, norm(f"{p}.norm1b", f"{p}.ls1"), norm(f"{p}.norm2"), ffn,
                                    norm(f"{p}.norm2b", f"{p}.ls2")))
    embedding = TokenEmbedding(opts, cfg.vocab, E, "embed", weight_suffix="", scale=float(cfg.embedding["scale"]),
                               positions=PositionTable(opts, cfg.max_positions, E, "pos"))
    return DecoderSpec(
        embedding=embedding, layers=layers, final_norm=norm("final.norm"),
        head=VocabHead(opts, cfg.vocab, E, "head", weight_suffix="", softcap=cfg.logit_softcap),
        stop_token_ids=cfg.stop_tokens, vocab_size=cfg.vocab)
