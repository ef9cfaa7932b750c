"""The Ponusun decoder, put together from the parts.

The stream starts as embedded tokens plus learned positions.  A layer's mixer reads the stream plus a short causal
convolution of it, its feed-forward the stream itself; an RMS norm acts on each sub-layer's output before it joins the
stream; what a layer hands on is a learned average of its result, the results of all layers before it and the embedding
output.  The mixer is grouped attention with a query/key norm over the whole projection, no rotation, a penalty on
distance that grows with its logarithm, and a sliding window; a layer may read the keys and values of an earlier one.
The feed-forward is a plain one with GELU, or gated experts (SiLU) chosen by a table of token ids beside a shared expert
with a sigmoid gate.  The logits are bounded by a tanh.

Tensor names (matrices [out, in], named by their prefix alone):
    embed, pos, final.norm, head, l<i>.norm1, l<i>.norm2, l<i>.canon1, l<i>.dwa
    l<i>.mix.{q,k,v,o,q.norm,k.norm,r1,r2}          (no k, v and k.norm with kv_from)
    l<i>.mlp.{up,down}                                                                       dense
    l<i>.mlp.table, l<i>.mlp.e<j>.{gate,up,down}, l<i>.mlp.shared.{gate,up,down,sg}          moe
"""
from __future__ import annotations

import torch

from ..config.ponusun import PonusunConfig
from ..config.registry import register_architecture
from ..engine.model import DecoderSpec, Run
from ..parts import (BuildOptions, DepthAverage, InputConv, MapsAttention, PlainFeedForward, PositionTable, PostNormBlock,
                     RMSNorm, TableExperts, TokenEmbedding, VocabHead)


def _window(mx):
    return mx["mask"]["size"] if mx.get("mask") else None


@register_architecture("Ponusun", PonusunConfig)
def build_ponusun(cfg: PonusunConfig, opts: BuildOptions) -> DecoderSpec:
    E, eps = cfg.width, cfg.eps

    def norm(name):
        return RMSNorm(opts, E, eps, name, weight_suffix="")

    # a layer's keys and values serve the widest window among itself and the layers that read them
    keeps: dict = {}
    for i, layer in enumerate(cfg.layers):
        owner = layer["mixer"].get("kv_from")
        owner = i if owner is None else owner
        w = _window(layer["mixer"])
        keeps[owner] = "all" if w is None or keeps.get(owner) == "all" else max(w, keeps.get(owner, 0))

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, mx = f"l{i}", layer["mixer"]
        owner = mx.get("kv_from")
        schedule.append(Run(i, reads_entry_of=owner))          # a run per layer, in order
        # the sub-layers' outputs are normed right away: they leave their last product in float32
        mixer = MapsAttention(opts, E, mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], None, f"{p}.mix", mx["scale"], eps,
                              window=_window(mx), keep_window=keeps[i if owner is None else owner], qk_norm=True,
                              qk_norm_rows=True, distance=("r1", "r2"), own_kv=owner is None, out_dtype=torch.float32)
        mlp = layer.get("mlp")
        ffn = None
        if mlp is not None and mlp["kind"] == "dense":
            ffn = PlainFeedForward(opts, E, mlp["ff"], f"{p}.mlp", out_dtype=torch.float32)
        elif mlp is not None:
            shared = mlp.get("shared")
            ffn = TableExperts(opts, E, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"], cfg.vocab,
                               f"{p}.mlp", shared_inner=shared["ff"] if shared else 0)
        layers.append(PostNormBlock(mixer, norm(f"{p}.norm1"), ffn, norm(f"{p}.norm2") if ffn is not None else None,
                                    conv=InputConv(opts, E, cfg.canon["taps"], f"{p}.canon1"),
                                    average=DepthAverage(opts, i + 1, f"{p}.dwa")))
    embedding = TokenEmbedding(opts, cfg.vocab, E, "embed", weight_suffix="",
                               positions=PositionTable(opts, cfg.max_positions, E, "pos"))
    return DecoderSpec(
        embedding=embedding, layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        head=VocabHead(opts, cfg.vocab, E, "head", weight_suffix="", softcap=cfg.logit_softcap),
        stop_token_ids=cfg.stop_tokens, vocab_size=cfg.vocab)
