"""The Nulalorn decoder, composed from parts.

    x0 = embed[token];   x = x0
    the layers in order, of which layers loop.start .. loop.stop - 1 run loop.times times in a row (same weights, a cache of
    its own for every pass; in front of pass t:  x <- W_in [x ; x0] + step[t]):                             (StreamEntry)
        x += n1b(mixer(n1(x)));   x += n2b(ffn(n2(x)))                  (SandwichNormBlock; a layer may have no ffn)
        mixer: window attention with a capped score on rotated q and k of unit mean square       (UnitHeadAttention)
        ffn:   down(gelu(up h)), or such experts named by a table of the token ids, beside a shared one   (TableExperts)
    logits = cap(head . rmsnorm(x))

Tensor names: embed, head, final.norm, loop.in, loop.step and, for layer i, l<i>.{norm1,norm1b,norm2,norm2b}, l<i>.mix.{q,k,v,o},
l<i>.mlp.{up,down} or l<i>.mlp.{table,e<j>.{up,down},shared.{up,down,sg}}.
Every layer keeps pages of keys and values (window groups: pages go back as the window passes).
"""
from __future__ import annotations

import torch

from ..config.nulalorn_config import MOE, NeighbourRotarySpec, NulalornConfig
from ..config.registry import register_architecture
from ..parts.attention import UnitHeadAttention
from ..parts.base import Runtime
from ..parts.block import SandwichNormBlock
from ..parts.embedding import OutputHead, TokenEmbedding
from ..parts.experts import TableExperts
from ..parts.mlp import DenseFeedForward
from ..parts.norm import RMSNorm
from ..parts.rope import NeighbourRotary
from ..parts.stream_entry import StreamEntry
from .decoder import DecoderModel, LayerCall


def _rotary(rt: Runtime, dim: int, r: NeighbourRotarySpec):
    if r.dims <= 0:
        return None
    return NeighbourRotary(rt, dim, r.base, r.dims, bands=(r.factor, r.low, r.high, r.original) if r.factor else None)


def build_nulalorn(cfg: NulalornConfig, rt: Runtime) -> DecoderModel:
    W, eps, f32 = cfg.width, cfg.norm_eps, torch.float32
    blocks = []
    for i, l in enumerate(cfg.layers):
        p, a, f = f"l{i}", l.attention, l.mlp
        mixer = UnitHeadAttention(rt, f"{p}.mix", W, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, _rotary(rt, a.dim, a.rot),
                                      a.window, eps, out_dtype=f32)
        ffn = None
        if f is not None and f.kind == MOE:
            shared = None
            if f.shared_ff:
                shared = DenseFeedForward(rt, f"{p}.mlp.shared.up", f"{p}.mlp.shared.down", W, f.shared_ff, act="gelu", out_dtype=f32)
            ffn = TableExperts(rt, f"{p}.mlp", cfg.vocab, W, f.experts, f.top, f.ff, act="gelu", shared=shared)
        elif f is not None:
            ffn = DenseFeedForward(rt, f"{p}.mlp.up", f"{p}.mlp.down", W, f.ff, act="gelu", out_dtype=f32)
        norm = lambda name: RMSNorm(rt, f"{p}.{name}", W, eps)
        blocks.append(SandwichNormBlock(mixer, ffn, norm("norm1"), norm("norm1b"), norm("norm2") if ffn is not None else None,
                                        norm("norm2b") if ffn is not None else None, rt.act_dtype))
    # the order of runs: the layers before the loop, the looped run `times` times, the rest; a cache for every run
    a, b, n = cfg.loop_start, cfg.loop_stop, len(blocks)
    order = [(i, -1) for i in range(a)]
    for t in range(cfg.loop_times if cfg.loops else 0):
        order += [(i, t if i == a else -1) for i in range(a, b)]
    order += [(i, -1) for i in range(b, n)]
    calls = [LayerCall(i, j, True, entry=t) for j, (i, t) in enumerate(order)]
    entry = StreamEntry(rt, "loop.in", "loop.step", W, cfg.loop_times) if cfg.loops else None
    embedding = TokenEmbedding(rt, "embed", cfg.vocab, W)
    head = OutputHead(rt, "head", cfg.vocab, W, None, softcap=cfg.logit_softcap)
    # norms of a feed-forward that is not there, and the entry of a loop over no layers: a checkpoint may carry them
    unused = [f"l{i}.{name}" for i, l in enumerate(cfg.layers) if l.mlp is None for name in ("norm2", "norm2b")]
    unused += [] if cfg.loops else ["loop.in", "loop.step"]
    return DecoderModel(rt, embedding, blocks, calls, RMSNorm(rt, "final.norm", W, eps), head, cfg.vocab, 0, cfg.eos_token_ids,
                        ignored_names=unused, stream_entry=entry)


register_architecture(NulalornConfig.ARCHITECTURE, NulalornConfig.from_dict, build_nulalorn, replace=True)
