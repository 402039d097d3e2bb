"""Latent attention without positions: keys and values of all heads are linear maps of ONE normed latent
vector per token, and only that latent is kept.

    c_q = rmsnorm(W_dq u) * w_q         q_h = W_uq[h] c_q                       (heads x dim)
    c   = rmsnorm(W_dkv u) * w_kv       k_h = W_uk[h] c,  v_h = W_uv[h] c        (dim, vdim a head)
    o_h = softmax_j<=i( q_h . k_h,j * scale ) v_h,j ;  out = W_o ( concat_h o_h * sigmoid(W_g u) )

Because k and v are linear in c, the head's key map moves to the query and its value map behind the sum:
q_h . (W_uk[h] c_j) = (W_uk[h]^T q_h) . c_j and sum_j p_j W_uv[h] c_j = W_uv[h] (sum_j p_j c_j).  So the
attention itself runs as `heads` query heads of size kv_rank over one shared "head" whose keys and values
are both the cached latents, through the same paged attention kernels as grouped-query attention
(KVPages(1, kv_rank, shared=True): one vector a token, half the memory of separate keys and values), for
prompts and for decoding alike.  The three maps that read u (W_dq | W_dkv | W_g) are one product with
32-bit output; the two norms and the write into the pages are one kernel; the per-head maps are one
batched product each, the second with the sigmoid gate in its epilogue.

Where it costs no more multiplications than the two maps apart (kv_rank * q_rank <= dim * (q_rank + kv_rank):
latents no wider than about a head), the query's two maps are multiplied out once when the weights are bound,
W_qc[h] = W_uk[h]^T W_uq[h] ([kv_rank, q_rank], formed in 32-bit), and the query in latent space is one product
of the normed query latent with the stacked W_qc.
"""
from __future__ import annotations

from typing import Callable, Hashable, Optional

import numpy as np
import torch

from .. import ops
from .attention import BIG_PORTION, DECODE_ROWS, TILE_ROWS, plan_tiles, tiles_of
from .base import BatchShape, KVCacheView, KVPages, Mixer, ParamSpec, Part, PositionEncoding, Runtime, StepContext, StepPlan
from .linear import Linear

# Most bytes that a step's multiplied-out keys and values may take; portions beyond are left in latent space.
EXPANSION_BYTES = 1 << 30


class LatentAttention(Mixer):
    recordable = True

    def __init__(self, rt: Runtime, prefix: str, width: int, heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int,
                 scale: float, eps: float):
        self.rt, self.prefix = rt, prefix
        self.width, self.heads, self.dim, self.vdim = width, heads, dim, vdim
        self.q_rank, self.kv_rank, self.scale, self.eps = q_rank, kv_rank, float(scale), float(eps)
        # one product for everything that reads the mixer's input: query latent | key/value latent | gate
        self.down = Linear(rt, [f"{prefix}.dq", f"{prefix}.dkv", f"{prefix}.g"], width, [q_rank, kv_rank, heads * vdim])
        self.uq = Linear(rt, f"{prefix}.uq", q_rank, heads * dim)
        self.o = Linear(rt, f"{prefix}.o", heads * vdim, width)
        self.q_norm_w: torch.Tensor | None = None
        self.kv_norm_w: torch.Tensor | None = None
        self.uk_t: torch.Tensor | None = None       # [heads, kv_rank, dim]: W_uk[h]^T, the key map moved to the query
        self.uv: torch.Tensor | None = None         # [heads, vdim, kv_rank]
        # the query's two maps as one, where that is no more work (see the module's text)
        self.merge_query_maps = kv_rank * q_rank <= dim * (q_rank + kv_rank)
        self.qc: Linear | None = None               # [heads * kv_rank, q_rank] when merged

    def children(self) -> list[Part]:
        return [self.down, self.uq, self.o]

    def param_specs(self) -> list[ParamSpec]:
        p = self.prefix
        return [ParamSpec(f"{p}.dq.norm", (self.q_rank,), "norm"), ParamSpec(f"{p}.dkv.norm", (self.kv_rank,), "norm"),
                ParamSpec(f"{p}.uk", (self.heads * self.dim, self.kv_rank)), ParamSpec(f"{p}.uv", (self.heads * self.vdim, self.kv_rank))]

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        p = self.prefix
        self.q_norm_w = get(f"{p}.dq.norm").to(torch.float32).contiguous()
        self.kv_norm_w = get(f"{p}.dkv.norm").to(torch.float32).contiguous()
        self.uk_t = get(f"{p}.uk").view(self.heads, self.dim, self.kv_rank).transpose(1, 2).contiguous()
        self.uv = get(f"{p}.uv").view(self.heads, self.vdim, self.kv_rank).contiguous()

    def bind_all(self, get) -> None:
        super().bind_all(get)
        if self.merge_query_maps:
            uq = self.uq.weight.view(self.heads, self.dim, self.q_rank)
            merged = torch.bmm(self.uk_t.float(), uq.float()).reshape(self.heads * self.kv_rank, self.q_rank)
            self.qc = Linear(self.rt, f"{self.prefix}.uk^T.uq", self.q_rank, self.heads * self.kv_rank)
            self.qc.bind_tensor(merged.to(self.uq.weight.dtype).contiguous())
            self.uq.weight = None                   # the two maps are not needed apart
            self.uk_t = None

    def cache_request(self) -> KVPages:
        return KVPages(1, self.kv_rank, 0, shared=True)

    # The tile lists of the tensor-core attention kernels, as grouped-query attention makes them for a group of query
    # heads on one key/value head.  All heads read the one cached "head"; more than 16 of them are cut into `share`
    # equal groups of at most 16 (the rows of the decode kernels' tiles), each of which reads it on its own.  The work
    # items of the prompt kernel ("big") stay those of all heads together.
    @property
    def share(self) -> int:
        if self.heads <= DECODE_ROWS:
            return 1
        return next((s for s in range(2, self.heads + 1) if self.heads % s == 0 and self.heads // s <= DECODE_ROWS), 1)

    def plan_key(self) -> Optional[Hashable]:
        if not self.rt.fast_kernels or self.heads // self.share > TILE_ROWS:
            return None
        return ("attention tiles", self.heads, self.share)

    def plan(self, batch: BatchShape) -> Optional[StepPlan]:
        share = self.share
        key = (self.heads, share, len(batch.q_lens)) if batch.max_q_len == 1 else None
        if key is not None and key in self._plans_of_single_tokens:
            return self._plans_of_single_tokens[key]
        plan = plan_tiles(batch, self.heads // share)
        if share > 1 and "big" in plan.arrays:
            whole = plan_tiles(batch, self.heads)
            plan.arrays["big"] = whole.arrays["big"]
            plan.host["rows"]["big"] = whole.host["rows"]["big"]
        if key is not None:
            self._plans_of_single_tokens[key] = plan
        return plan

    _plans_of_single_tokens: dict = {}

    def forward(self, u: torch.Tensor, step: StepContext, cache: KVCacheView, write_cache: bool = True) -> torch.Tensor:
        rt = self.rt
        T, H = u.shape[0], self.heads
        if not write_cache:
            raise ops.KernelError("latent attention always writes its own latents")
        table = step.block_tables[cache.group]
        pre = self.down.forward(u, out_dtype=torch.float32)                  # [T, q_rank + kv_rank + H * vdim]
        c_q = rt.empty((T, self.q_rank))
        ops.latent_norm(pre, 0, self.q_rank, self.q_rank, self.kv_rank, self.q_norm_w, self.kv_norm_w, c_q, cache.k,
                        step, table, cache.page_size, self.eps, rt.stream)
        if self.qc is not None:
            q_lat = self.qc.forward(c_q).view(T, H, self.kv_rank)
        else:
            q = self.uq.forward(c_q).view(T, H, self.dim)
            q_lat = rt.empty((T, H, self.kv_rank))
            ops.gemm_heads(q_lat, q, self.uk_t, rt.stream)                   # the head's key map, applied to the query
        mix = rt.empty((T, H, self.kv_rank))
        ops.attention(q_lat, mix, cache.k, cache.v, step, cache.group, H, 1, self.kv_rank, cache.page_size, 0,
                      self.scale, rt.stream, plan=step.plans.get(self.plan_key()), kv_share=self.share)
        gated = rt.empty((T, H, self.vdim))
        ops.gemm_heads(gated, mix, self.uv, rt.stream, gate=pre[:, self.q_rank + self.kv_rank:])
        return self.o.forward(gated.view(T, H * self.vdim))


class RotaryLatentAttention(Mixer):
    """Latent attention whose keys carry a rotated part that all heads share, with a learned sink and a gate of one number a head:

        q_h = [q_u,h | rotate(q_r,h)]      from W_q u, head by head (dim | rot_dim entries)
        c = rmsnorm(.) * w (kv_rank entries),  k_r = rotate(.) (rot_dim entries)      from W_dkv u
        k_h = [W_uk[h] c | k_r],  v_h = W_uv[h] c
        w_j = exp(q_h . k_h,j * scale) / (exp(sink_h) + sum_j<=i exp(q_h . k_h,j * scale))
        out = W_o concat_h( sigmoid(W_g u)_h * sum_j w_j v_h,j )

    [c | k_r] is all that is cached: one vector of kv_rank + rot_dim entries a token, key and value of one "head" whose values
    are the first kv_rank entries (KVPages(1, kv_rank + rot_dim, shared=True)).  As in LatentAttention the head's key map moves
    to the query and its value map behind the sum: attention runs as `heads` query heads [W_uk[h]^T q_u | q_r] over the cached
    vectors (latent_flash.cu).  For longer portions that is several times the work of attention on the heads' own keys and
    values, so these are multiplied out of the gathered latents first (latent_prefill.cu) where that pays.  W_q | W_dkv |
    W_g are one product with 32-bit output; one kernel norms the latent, rotates, and writes the pages and the queries."""
    recordable = True

    def __init__(self, rt: Runtime, prefix: str, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int,
                 scale: float, position_encoding: Optional[PositionEncoding], eps: float, out_dtype: Optional[torch.dtype] = None):
        if position_encoding is not None and position_encoding.rotary_table() is None:
            raise ValueError("this attention rotates by a table of frequencies (rotary_table)")
        self.rt, self.prefix, self.width = rt, prefix, width
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.scale, self.eps, self.out_dtype = float(scale), float(eps), out_dtype
        self.position_encoding = position_encoding
        self.key_size = kv_rank + rot_dim
        self.expandable = ops.latent_prefill_ok(dim, rot_dim, vdim, kv_rank)
        self.proj = Linear(rt, [f"{prefix}.q", f"{prefix}.dkv", f"{prefix}.g"], width, [heads * (dim + rot_dim), self.key_size, heads])
        self.o = Linear(rt, f"{prefix}.o", heads * vdim, width)
        self.kv_norm_w: torch.Tensor | None = None
        self.sinks: torch.Tensor | None = None
        self.uk_t: torch.Tensor | None = None       # [heads, kv_rank, dim]: W_uk[h]^T, the key map moved to the query
        self.uv: torch.Tensor | None = None         # [heads, vdim, kv_rank]
        self.ukv: torch.Tensor | None = None        # [heads * (dim + vdim), kv_rank]: both maps as they are, all keys' rows first

    def children(self) -> list[Part]:
        return [self.proj, self.o]

    def param_specs(self) -> list[ParamSpec]:
        p = self.prefix
        return [ParamSpec(f"{p}.dkv.norm", (self.kv_rank,), "norm"), ParamSpec(f"{p}.uk", (self.heads * self.dim, self.kv_rank)),
                ParamSpec(f"{p}.uv", (self.heads * self.vdim, self.kv_rank)), ParamSpec(f"{p}.sink", (self.heads,))]

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        p = self.prefix
        self.kv_norm_w = get(f"{p}.dkv.norm").to(torch.float32).contiguous()
        self.sinks = get(f"{p}.sink").to(torch.float32).contiguous()
        self.uk_t = get(f"{p}.uk").view(self.heads, self.dim, self.kv_rank).transpose(1, 2).contiguous()
        self.uv = get(f"{p}.uv").view(self.heads, self.vdim, self.kv_rank).contiguous()
        if self.rt.fast_kernels and self.expandable:
            self.ukv = torch.cat([get(f"{p}.uk"), get(f"{p}.uv")], dim=0).contiguous()
            self.uv = self.ukv[self.heads * self.dim:].view(self.heads, self.vdim, self.kv_rank)       # the same memory

    def cache_request(self) -> KVPages:
        return KVPages(1, self.key_size, 0, shared=True)

    @property
    def group(self) -> int:
        """Heads that share a tile of query rows: all of them up to 64, else their largest equal groups of at most 64."""
        return next(self.heads // s for s in range(1, self.heads + 1) if self.heads % s == 0 and self.heads // s <= TILE_ROWS)

    def plan_key(self) -> Optional[Hashable]:
        if not self.rt.fast_kernels or not self.scale > 0:
            return None
        return ("latent tiles", self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank)

    def plan(self, batch: BatchShape) -> Optional[StepPlan]:
        """"big": the portions whose keys and values are worth multiplying out (ops.latent_expansion_pays), in items of up to 256
        tokens of the tensor-memory kernel, (first token, tokens, request, first row of the request), with "entries" (request,
        first row, rows, 0).  "rest": the other tokens, in tiles of up to 64 query rows; where single tokens are among
        them, of as few rows as one token needs (the kernel's work follows the largest tile).  The host's part says how many
        rows there are in all and between which tokens the rest lies."""
        key = (self.group, len(batch.q_lens)) if batch.max_q_len == 1 else None      # single tokens: the same tiles for every such step
        if key in self._plans_of_single_tokens:
            return self._plans_of_single_tokens[key]
        g, T = self.group, sum(batch.q_lens)
        spans = [batch.span_hint if batch.recorded else s + n for s, n in zip(batch.start_positions, batch.q_lens)]
        row_bytes = 2 * self.heads * (self.dim + self.vdim)
        entries, firsts, rows, t = [], {}, 0, 0
        for i, (n, span) in enumerate(zip(batch.q_lens, spans)):
            if (n >= BIG_PORTION and self.expandable and (rows + span) * row_bytes <= EXPANSION_BYTES
                    and ops.latent_expansion_pays(n, span, self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank)):
                entries.append((i, rows, span, 0))
                firsts[i] = rows
                rows += span
        arrays, host = {}, {"rows": rows, "lo": 0, "hi": T}
        if entries:
            ids = set(firsts)
            item = lambda n: [tl for tl in tiles_of(batch.q_lens, 1, n) if tl[2] in ids]
            big = item(256)
            if len(big) * self.heads < 148:                  # few items: half as long ones fill more SMs
                big = item(128)
            big.sort(key=lambda tl: -(batch.start_positions[tl[2]] + tl[3] + tl[1]))       # those that see the most keys first
            arrays["big"] = np.asarray([(a, n, i, firsts[i]) for a, n, i, _ in big], dtype=np.int32)
            arrays["entries"] = np.asarray(entries, dtype=np.int32)
        rest = [n for i, n in enumerate(batch.q_lens) if i not in firsts]
        if rest:
            tile_rows = -(-g // 16) * 16 if 1 in rest else TILE_ROWS
            tiles = [tl for tl in tiles_of(batch.q_lens, g, tile_rows) if tl[2] not in firsts]
            arrays["rest"] = np.asarray(tiles, dtype=np.int32).reshape(len(tiles), 4)
            host.update(tile_rows=max(n for _, n, _, _ in tiles) * g, lo=tiles[0][0], hi=tiles[-1][0] + tiles[-1][1])
        plan = StepPlan(arrays, host)
        if key is not None:
            self._plans_of_single_tokens[key] = plan
        return plan

    _plans_of_single_tokens: dict = {}

    def _in_latent_space(self, gated: torch.Tensor, q: torch.Tensor, q_lat: torch.Tensor, gate: torch.Tensor, step: StepContext,
                         cache: KVCacheView, plan, lo: int, hi: int) -> None:
        """The tokens lo .. hi - 1 (others among them are overwritten later): the head's key map applied to the query, attention over
        the cached vectors, the head's value map and gate."""
        rt, L = self.rt, self.kv_rank
        table = step.block_tables[cache.group]
        ops.gemm_heads(q_lat[lo:hi, :, :L], q[lo:hi, :, :self.dim], self.uk_t, rt.stream)
        mix = rt.empty((q.shape[0], self.heads, L))
        if plan is None or not ops.latent_flash_ok(self.key_size, L, self.group, cache.page_size):
            ops.attention_plain(q_lat, mix, cache.k, cache.v, step.positions, step.token_seq, table, self.heads, 1, self.key_size,
                                cache.page_size, 0, self.scale, rt.stream, v_dim=L, v_stride=self.key_size, sinks=self.sinks)
        else:
            tiles = plan.arrays["rest"]
            splits = ops.latent_flash_splits(tiles.shape[0], self.heads // self.group, step.span_hint or step.max_context_len)
            ops.latent_flash(q_lat, mix, cache.k, step.positions, table, tiles, plan.host["tile_rows"], self.group, cache.page_size, self.scale,
                             splits, rt.stream, sinks=self.sinks)
        ops.gemm_heads(gated[lo:hi], mix[lo:hi], self.uv, rt.stream, gate=gate[lo:hi])

    def _multiplied_out(self, gated: torch.Tensor, q: torch.Tensor, gate: torch.Tensor, step: StepContext, cache: KVCacheView, plan) -> None:
        """The portions whose keys and values are formed for every head first."""
        rt, rows = self.rt, plan.host["rows"]
        lat = rt.empty((rows, self.key_size))
        ops.latent_gather(lat, cache.k, plan.arrays["entries"], step.context_lens, step.block_tables[cache.group], cache.page_size, rt.stream)
        kv = rt.empty((rows, self.heads * (self.dim + self.vdim)))
        ops.linear(kv, lat[:, :self.kv_rank], self.ukv, rt.stream, fast=True)
        tiles = plan.arrays["big"]
        splits = ops.attention_tcgen05_splits(tiles.shape[0], self.heads, step.span_hint or step.max_context_len)
        ops.latent_prefill(q, gated, kv, lat, step.positions, tiles, self.dim, self.rot_dim, self.kv_rank, self.scale, rt.stream, sinks=self.sinks,
                           gate=gate, key_splits=splits)

    def forward(self, u: torch.Tensor, step: StepContext, cache: KVCacheView, write_cache: bool = True) -> torch.Tensor:
        rt = self.rt
        T, H = u.shape[0], self.heads
        if not write_cache:
            raise ops.KernelError("latent attention always writes its own latents")
        n_q = H * (self.dim + self.rot_dim)
        pre = self.proj.forward(u, out_dtype=torch.float32)                  # q | dkv | g
        gate = pre[:, n_q + self.key_size:]
        plan = step.plans.get(self.plan_key())
        big = plan is not None and "big" in plan.arrays
        rest = plan is None or "rest" in plan.arrays
        inv_freq, rot = self.position_encoding.rotary_table() if self.position_encoding is not None else (None, 0)
        q, q_lat = rt.empty((T, H, self.dim + self.rot_dim)), rt.empty((T, H, self.key_size)) if rest else None
        ops.latent_rope(pre, 0, n_q, H, self.dim, self.rot_dim, self.kv_rank, self.kv_norm_w, inv_freq, rot,
                        getattr(self.position_encoding, "magnitude", 1.0), q, q_lat, cache.k, step, step.block_tables[cache.group],
                        cache.page_size, self.eps, rt.stream)
        gated = rt.empty((T, H, self.vdim))
        if rest:
            self._in_latent_space(gated, q, q_lat, gate, step, cache, plan, plan.host["lo"] if plan else 0, plan.host["hi"] if plan else T)
        if big:
            self._multiplied_out(gated, q, gate, step, cache, plan)
        return self.o.forward(gated.view(T, H * self.vdim), out_dtype=self.out_dtype)
