"""A feed-forward of many small experts of which each token uses a few, plus (optionally) one that every token uses.

RoutedExperts chooses by a router:

    z = W_router h (32-bit)         s = sigmoid(z)         choice score c = s + correction
    experts form `groups` equal groups of neighbours; a group is worth the sum of its two largest c; only experts of the
    `keep` best groups can be chosen; the `top` experts with the largest c are
    weights = s of the chosen / (their sum + 1e-20) * scale          (the correction steers the choice only)
    or, with `scores="softmax"`: c = z, and the weights are the softmax over the chosen z alone, times scale
    out = sum_k weight_k * expert_k(h) [+ shared(h)]

TableExperts has no router: a table [vocab, top] names the experts of every token id, and each counts 1 / top,

    out = sum_k expert_(table[id, k])(h) / top [+ sigmoid(w_sg . h) * shared(h)]

An expert is a gated feed-forward (GATE_ACTS of ops, e.g. "clamped_swish" with its limit) or an ungated one ("gelu"), without
biases.  The checkpoint holds each expert's matrices under <prefix>.e<j>.{gate,up,down} or .{up,down}; they are stacked
when bound ([experts, 2 ff, width] gate rows then up rows, or [experts, ff, width], and [experts, width, ff]).

Everything runs on the device with launches that do not depend on the choices (the pairs of token and choice are
sorted by expert by a kernel; the products walk a list of row tiles that the same kernel writes), so a step through
this part can be recorded.

Steps with many tokens (bfloat16 engine, `GROUPED_FROM` pairs an expert and more) take the tensor-memory product
instead: every expert's run of pairs is padded to whole tiles of 128 places, the tokens are gathered into that order,
and `gemm_tcgen05_grouped` multiplies every tile with its expert's matrix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional

import torch

from .. import ops
from .base import ExpertSum, FeedForward, ParamSpec, Part, Runtime, StepContext
from .linear import Linear


# From this many pairs of token and choice an expert (on average) the padded runs of the tensor-memory product cost
# less than they gain: the padding is 64 places an expert on average, 127 at most, and the product several times faster.
GROUPED_FROM = 96
# Up to so many pairs an expert (on average) a step is a stream of the experts' weights and takes the kernel made for it, with row
# tiles of 16 places (an expert with more reads its weights once a tile), or, for gated products, of 64 from FEW_UP_TO on.
FEW_UP_TO, SOME_UP_TO = 8, 48


@dataclass
class Dispatch:
    """Where the pairs of token and choice of a step stand, sorted by expert (device tensors, see ops.expert_dispatch)."""
    pair_at: torch.Tensor
    place_of: torch.Tensor
    meta: Optional[torch.Tensor] = None             # the row tiles of the runs; None: runs padded to whole tiles, then
    tile_group: Optional[torch.Tensor] = None       # the expert of each tile
    few: int = 0                                    # the kernel for few pairs an expert, see ops.expert_gemm


class ExpertBank(FeedForward):
    """The experts' matrices, the sorting of a step's pairs of token and choice, and the products over the sorted pairs."""
    recordable = True

    def __init__(self, rt: Runtime, prefix: str, width: int, experts: int, top: int, ff: int, act: str, limit: float = 0.0):
        if act not in ops.GATE_ACTS and act != "gelu":
            raise ValueError(f"activation {act!r} of an expert is not one of {['gelu', *sorted(ops.GATE_ACTS)]}")
        self.rt, self.prefix, self.width = rt, prefix, width
        self.experts, self.top, self.ff, self.act, self.limit = experts, top, ff, act, float(limit)
        self.gated = act in ops.GATE_ACTS
        self.interleaved = False
        self.gate_up: torch.Tensor | None = None        # [experts, 2 * ff, width], ungated [experts, ff, width]
        self.down: torch.Tensor | None = None           # [experts, width, ff]

    def expert_specs(self) -> list[ParamSpec]:
        p, specs = self.prefix, []
        for j in range(self.experts):
            if self.gated:
                specs.append(ParamSpec(f"{p}.e{j}.gate", (self.ff, self.width)))
            specs += [ParamSpec(f"{p}.e{j}.up", (self.ff, self.width)), ParamSpec(f"{p}.e{j}.down", (self.width, self.ff))]
        return specs

    def bind_experts(self, get: Callable[[str], torch.Tensor]) -> None:
        p = self.prefix
        ups = [get(f"{p}.e{j}.up") for j in range(self.experts)]
        fast = bool(self.rt.fast_kernels and ups[0].is_cuda and ups[0].dtype == torch.bfloat16 and self.width % 8 == 0)
        if not self.gated:
            self.grouped_ok = fast and self.ff % 8 == 0
            self.gate_up = torch.stack(ups).contiguous()
        else:
            # gate and up rows of an expert: interleaved in blocks of 64 where the products with the activation in their epilogue
            # want them so (both kinds of product then read that one copy), else all gate rows and then all up rows
            gates = [get(f"{p}.e{j}.gate") for j in range(self.experts)]
            self.interleaved = self.grouped_ok = fast and self.ff % 64 == 0
            if self.interleaved:
                self.gate_up = torch.stack([ops.interleave_gate_up(g, u) for g, u in zip(gates, ups)]).contiguous()
            else:
                self.gate_up = torch.stack([torch.cat([g, u], dim=0) for g, u in zip(gates, ups)]).contiguous()
        self.down = torch.stack([get(f"{p}.e{j}.down") for j in range(self.experts)]).contiguous()

    def dispatch(self, ids: torch.Tensor, num_tokens: int, tokens: Optional[torch.Tensor] = None) -> Dispatch:
        """Sort the pairs.  ids: [T, top], or a table [vocab, top] with the step's token ids as `tokens`.  Steps with many
        pairs an expert pad every expert's run to whole tiles of the tensor-memory product."""
        rt, E = self.rt, self.experts
        pairs = num_tokens * self.top
        place_of = rt.empty((pairs,), torch.int32)
        if self.grouped_ok and pairs >= GROUPED_FROM * E:
            places = ops.expert_padded_places(pairs, E)
            pair_at, tile_group = rt.empty((places,), torch.int32), rt.empty((places // ops.GROUP_TILE,), torch.int32)
            ops.expert_dispatch_padded(ids, E, pair_at, place_of, tile_group, rt.stream, tokens=tokens)
            return Dispatch(pair_at, place_of, tile_group=tile_group)
        offsets, pair_at = rt.empty((E + 1,), torch.int32), rt.empty((pairs,), torch.int32)
        few = 0 if not self.grouped_ok else 1 if pairs <= FEW_UP_TO * E else 2 if self.gated and pairs <= SOME_UP_TO * E else 0
        meta = rt.empty((4 + 3 * ops.expert_max_tiles(pairs, E, few),), torch.int32)
        ops.expert_dispatch(ids, E, offsets, pair_at, place_of, meta, rt.stream, tokens=tokens, few=few)
        return Dispatch(pair_at, place_of, meta=meta, few=few)

    def products(self, h: torch.Tensor, d: Dispatch) -> torch.Tensor:
        """The experts' outputs at their places, float32 [places, width]."""
        rt = self.rt
        places = d.pair_at.shape[0]
        inner, y = rt.empty((places, self.ff)), rt.empty((places, self.width), torch.float32)
        how = dict(act=self.act, limit=self.limit) if self.gated else dict(post=self.act)
        if d.tile_group is not None:
            xs = rt.empty((places, self.width))
            ops.expert_gather_rows(xs, h, d.pair_at, self.top, rt.stream)
            ops.gemm_tcgen05_grouped(inner, xs, self.gate_up, d.tile_group, rt.stream, **how)
            ops.gemm_tcgen05_grouped(y, inner, self.down, d.tile_group, rt.stream)
            return y
        ops.expert_gemm(inner, h, self.gate_up, d.meta, d.pair_at, self.top, True, rt.stream, fast=rt.fast_kernels,
                        interleaved=self.interleaved, few=d.few, **how)
        ops.expert_gemm(y, inner, self.down, d.meta, d.pair_at, self.top, False, rt.stream, fast=rt.fast_kernels, few=d.few % 2)
        return y


class RoutedExperts(ExpertBank):
    def __init__(self, rt: Runtime, prefix: str, width: int, experts: int, top: int, ff: int, act: str, limit: float,
                 router_scale: float, groups: int = 1, keep: int = 1, shared: Optional[FeedForward] = None,
                 correction: bool = True, out_dtype: Optional[torch.dtype] = None, scores: str = "sigmoid"):
        if scores not in ("sigmoid", "softmax") or (scores == "softmax" and correction):
            raise ValueError(f"scores {scores!r}: sigmoid, or softmax without a correction")
        if experts % groups or not (0 < keep <= groups) or not (0 < top <= keep * (experts // groups)):
            raise ValueError(f"{experts} experts, top {top}, {groups} groups of which {keep} are kept do not fit")
        super().__init__(rt, prefix, width, experts, top, ff, act, limit)
        self.router_scale, self.groups, self.keep = float(router_scale), groups, keep
        self.shared, self.has_correction = shared, correction
        self.out_dtype = out_dtype          # type of the result (None: the activation type)
        self.scores = scores
        self.router = Linear(rt, f"{prefix}.router", width, experts)
        self.correction: torch.Tensor | None = None

    def children(self) -> list[Part]:
        return [self.router] + ([self.shared] if self.shared is not None else [])

    def param_specs(self) -> list[ParamSpec]:
        specs = [ParamSpec(f"{self.prefix}.correction", (self.experts,), "linear")] if self.has_correction else []
        return specs + self.expert_specs()

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        if self.has_correction:
            self.correction = get(f"{self.prefix}.correction").to(torch.float32).contiguous()
        self.bind_experts(get)

    offers_unsummed = True

    def forward(self, h: torch.Tensor, step: StepContext, unsummed: bool = False):
        rt, top = self.rt, self.top
        T = h.shape[0]
        logits = self.router.forward(h, out_dtype=torch.float32)
        ids, weights = rt.empty((T, top), torch.int32), rt.empty((T, top), torch.float32)
        ops.route_topk(ids, weights, logits, self.correction, self.groups, self.keep, self.router_scale, rt.stream,
                       softmax=self.scores == "softmax")
        always = self.shared.forward(h, step) if self.shared is not None else None
        d = self.dispatch(ids, T)
        y = self.products(h, d)
        if unsummed:
            return ExpertSum(y, d.place_of, weights, always)
        out = rt.empty((T, self.width), self.out_dtype)
        ops.expert_combine(out, y, weights, d.place_of, rt.stream, always=always)
        return out


class TableExperts(ExpertBank):
    """Experts named by a table of the token ids: no router, equal weights.  `shared` runs for every token; its output
    counts times the sigmoid of one number a token, from the tensor <prefix>.shared.sg [1, width] (32-bit).

    The sorting of the pairs depends on the step's token ids alone: a block that runs several times in a step sorts once
    (StepContext.memo).  The part hands its output on unsummed (ExpertSum); the norm behind it forms the sum in its pass."""
    offers_unsummed = True

    def __init__(self, rt: Runtime, prefix: str, vocab: int, width: int, experts: int, top: int, ff: int, act: str = "gelu",
                 shared: Optional[FeedForward] = None, limit: float = 0.0):
        if not 0 < top <= experts:
            raise ValueError(f"{top} experts a token of {experts}")
        super().__init__(rt, prefix, width, experts, top, ff, act, limit)
        self.vocab, self.shared = vocab, shared
        self.table: torch.Tensor | None = None
        self.gate_weight: torch.Tensor | None = None

    def children(self) -> list[Part]:
        return [self.shared] if self.shared is not None else []

    def param_specs(self) -> list[ParamSpec]:
        specs = [ParamSpec(f"{self.prefix}.table", (self.vocab, self.top), integer=True, below=self.experts)] + self.expert_specs()
        if self.shared is not None:
            specs.append(ParamSpec(f"{self.prefix}.shared.sg", (1, self.width)))
        return specs

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        self.table = get(f"{self.prefix}.table").contiguous()
        low, high = int(self.table.min()), int(self.table.max())
        if low < 0 or high >= self.experts:
            raise ValueError(f"{self.prefix}.table names experts {low} .. {high}, there are {self.experts}")
        self.bind_experts(get)
        if self.shared is not None:
            self.gate_weight = get(f"{self.prefix}.shared.sg").to(torch.float32).reshape(-1).contiguous()

    def forward(self, h: torch.Tensor, step: StepContext, unsummed: bool = False):
        key = ("dispatch", self.prefix)
        d = step.memo.get(key)
        if d is None:
            d = step.memo[key] = self.dispatch(self.table, h.shape[0], tokens=step.token_ids)
        always = self.shared.forward(h, step) if self.shared is not None else None
        y = self.products(h, d)
        out = ExpertSum(y, d.place_of, 1.0 / self.top, always, h if always is not None else None, self.gate_weight)
        if unsummed:
            return out
        total = self.rt.empty((h.shape[0], self.width), torch.float32)
        ops.expert_combine(total, y, out.weights, d.place_of, self.rt.stream, always=always, gate_input=out.gate_input,
                           gate_weight=out.gate_weight)
        return total
