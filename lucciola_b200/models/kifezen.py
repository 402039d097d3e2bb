"""The Kifezen decoder, composed from parts.

    x_s = embed[token]  for each of `streams` residual streams
    each sublayer:  u = sum_s in[s] x_s;   y = sublayer(rmsnorm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y    (HyperConnectionBlock)
        mixer: attention on unit queries and keys, query temperature, a gate a head                     (UnitHeadAttention)
               or latent attention with a rotated part, a sink and a gate a head                        (RotaryLatentAttention)
        ffn:   down(silu(gate h) * (up h)), or such experts weighted by the softmax over the chosen     (GatedFeedForward, RoutedExperts)
    logits = head . rmsnorm(sum_s x_s)

Norm weights are stored around zero (but the latent's).  Tensor names: embed, head, final.norm and, for layer i, l<i>.{norm1,norm2},
l<i>.hc{1,2}.{in,out,mix}, l<i>.mix.*, l<i>.mlp.{gate,up,down} or l<i>.mlp.{router,e<j>.{gate,up,down}}.
"""
from __future__ import annotations

import torch

from ..config.kifezen_config import MOE, KifezenConfig
from ..config.registry import register_architecture
from ..parts.attention import UnitHeadAttention
from ..parts.base import Runtime
from ..parts.embedding import OutputHead, TokenEmbedding
from ..parts.experts import RoutedExperts
from ..parts.hyper_connection import HyperConnection, HyperConnectionBlock
from ..parts.latent_attention import RotaryLatentAttention
from ..parts.mlp import GatedFeedForward
from ..parts.norm import RMSNorm
from ..parts.rope import RotaryEmbedding
from .decoder import DecoderModel, LayerCall


def build_kifezen(cfg: KifezenConfig, rt: Runtime) -> DecoderModel:
    W, eps, f32 = cfg.width, cfg.norm_eps, torch.float32
    blocks, unused = [], []
    for i, l in enumerate(cfg.layers):
        p, f = f"l{i}", l.mlp
        if l.attention is not None:
            a = l.attention
            mixer = UnitHeadAttention(rt, f"{p}.mix", W, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, 0.0, None, 0, eps, out_dtype=f32,
                                      head_gate=True, temperature=(a.temp_coef, a.temp_every) if a.temp_every else None)
        else:
            b = l.latent
            r = b.rot
            rotary = RotaryEmbedding(rt, b.rot_dim, r.base, r.dims, yarn=(r.factor, r.original, r.fast, r.slow) if r.factor else None) if r.dims else None
            mixer = RotaryLatentAttention(rt, f"{p}.mix", W, b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.scale, rotary, eps, out_dtype=f32)
        ffn = None
        if f is not None and f.kind == MOE:
            ffn = RoutedExperts(rt, f"{p}.mlp", W, f.experts, f.top, f.ff, "silu", 0.0, 1.0, correction=False, out_dtype=f32, scores="softmax")
        elif f is not None:
            ffn = GatedFeedForward(rt, f"{p}.mlp.gate", f"{p}.mlp.up", f"{p}.mlp.down", W, f.ff, act="silu", out_dtype=f32)
        else:                   # what a checkpoint may carry for a feed-forward that is not there
            unused += [f"{p}.norm2", f"{p}.hc2.in", f"{p}.hc2.out", f"{p}.hc2.mix"]
        norm = lambda name: RMSNorm(rt, f"{p}.{name}", W, eps, around_zero=True)
        blocks.append(HyperConnectionBlock(mixer, ffn, norm("norm1"), norm("norm2") if ffn is not None else None,
                                           HyperConnection(rt, f"{p}.hc1", cfg.streams),
                                           HyperConnection(rt, f"{p}.hc2", cfg.streams) if ffn is not None else None, rt.act_dtype))
    calls = [LayerCall(i, i) for i in range(len(blocks))]
    head = OutputHead(rt, "head", cfg.vocab, W, None)
    return DecoderModel(rt, TokenEmbedding(rt, "embed", cfg.vocab, W), blocks, calls, RMSNorm(rt, "final.norm", W, eps, around_zero=True),
                        head, cfg.vocab, 0, cfg.eos_token_ids, ignored_names=unused)


register_architecture(KifezenConfig.ARCHITECTURE, KifezenConfig.from_dict, build_kifezen, replace=True)
