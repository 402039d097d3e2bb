"""Kifezen in the engine against the plain implementation: every mechanism alone, then the whole model under every way of
cutting the work, with pages that are freed and used again, and generation through the entry point (GPU)."""
from types import SimpleNamespace

import pytest
import torch

import kifezen_util as kz
import plain_kifezen as plain
import replay_util as ru

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TYPES = [torch.float32, torch.bfloat16]
DEV = "cuda:0"


def stream():
    return torch.cuda.current_stream().cuda_stream


def batch_of(q_lens, starts=None, tokens=None):
    """What the kernels read of a step."""
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    seq = [i for i, n in enumerate(q_lens) for _ in range(n)]
    starts = starts or [0] * len(q_lens)
    pos = [s + j for s, n in zip(starts, q_lens) for j in range(n)]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    return SimpleNamespace(num_tokens=cu[-1], num_seqs=len(q_lens), token_seq=i32(seq), cu_tokens=i32(cu), positions=i32(pos),
                           context_lens=i32([s + n for s, n in zip(starts, q_lens)]), q_lens=list(q_lens), start_positions=list(starts),
                           max_q_len=max(q_lens), max_context_len=max(s + n for s, n in zip(starts, q_lens)), span_hint=0, plans={},
                           block_tables=[], token_ids=i32(tokens) if tokens is not None else None, memo={})


def runtime(dtype=torch.float32):
    from lucciola_b200.parts.base import Runtime
    rt = Runtime(DEV, dtype)
    rt.stream = stream()
    return rt


def close(got, want, dtype, exact=3e-6, rounded=1e-2):
    err = (got.double().cpu() - want.double().cpu()).abs().max().item()
    assert err <= (exact if dtype == torch.float32 else rounded) * max(want.abs().max().item(), 1e-3), err


# ---- each mechanism alone --------------------------------------------------------------------------------------------
def scattered(n_pages, page, rest, lens, starts, dtype, seed=0):
    """A pool [pages, *rest with the page size in place] of NaN, and block tables [S, pages a sequence] in a scrambled order."""
    need = [-(-(s + n) // page) for s, n in zip(starts, lens)]
    g = torch.Generator().manual_seed(seed)
    order = torch.randperm(n_pages, generator=g).tolist()
    assert sum(need) <= n_pages
    table = torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
    for i, k in enumerate(need):
        for j in range(k):
            table[i, j] = order.pop()
    pool = torch.full((n_pages, rest[0], page, rest[1]), float("nan"), dtype=dtype, device=DEV)
    return pool, table.to(DEV)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,width,S", [(7, 40, 1), (3, 74, 3), (5, 512, 4), (9, 4096, 4), (2, 8192, 2), (2, 9000, 4), (1, 1028, 3), (4, 6, 7), (3, 300, 12)])
def test_streams_are_written_read_and_normed_in_one_pass(dtype, rows, width, S):
    """The first read of one row for all streams, the first write behind it, later writes in place, the plain sum at the end
    on picked rows; the sublayer's output in either type."""
    from lucciola_b200 import ops
    r = lambda *s: torch.randn(*s, device=DEV)
    e, X, w = r(rows, width), r(rows, S, width), r(width)
    mix, out, read = r(S, S), r(S), r(S)
    norm = lambda u: plain.rms(u, 1e-5) * w.double()
    got = torch.empty(rows, width, dtype=dtype, device=DEV)
    ops.streams_norm(got, e, S, w, 1e-5, stream(), read=read)
    first = e.double()[:, None, :].repeat(1, S, 1)
    close(got, norm(plain.streams_in(first, read.double())), dtype)
    ops.streams_norm(got, X, S, w, 1e-5, stream(), read=read)
    close(got, norm(plain.streams_in(X.double(), read.double())), dtype)
    for y_dtype in TYPES:
        y = (r(rows, width) * 3).to(y_dtype)
        for x, x64 in ((e, first), (X, X.double())):
            new64 = plain.streams_out(x64, y.double(), mix.double(), out.double())
            new = torch.full((rows, S, width), float("nan"), device=DEV)
            ops.streams_norm(got, x, S, w, 1e-5, stream(), read=read, update=(mix, out, y), x_new=new)
            close(new, new64, torch.float32)
            close(got, norm(plain.streams_in(new64, read.double())), dtype, 2e-5)
            if x.dim() == 3:
                place = x.clone()
                ops.streams_norm(got, place, S, w, 1e-5, stream(), read=read, update=(mix, out, y), x_new=place)
                assert torch.equal(place, new)
            keep = x.clone()
            pick = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32, device=DEV)
            some = torch.empty(3, width, dtype=dtype, device=DEV)
            ops.streams_norm(some, x, S, w, 1e-5, stream(), update=(mix, out, y), rows=pick)
            assert torch.equal(x, keep)
            close(some, norm(new64.sum(1))[pick.long()], dtype, 2e-5)


@pytest.mark.parametrize("width,S,top", [(40, 1, 1), (74, 3, 3), (512, 4, 2), (4096, 4, 4), (9000, 2, 5)])
def test_the_experts_sum_inside_the_pass_over_the_streams(width, S, top):
    from lucciola_b200 import ops
    T, places = 6, 60
    r = lambda *s: torch.randn(*s, device=DEV)
    e, X, w, mix, out, read = r(places, width), r(T, S, width), r(width), r(S, S), r(S), r(S)
    place = torch.randperm(places, device=DEV)[:T * top].to(torch.int32)
    for weights in (0.3, torch.rand(T, top, device=DEV)):
        wt = weights.double() if torch.is_tensor(weights) else torch.full((T, top), weights, dtype=torch.float64, device=DEV)
        y = (e.double()[place.long()].reshape(T, top, width) * wt[:, :, None]).sum(1)
        got, new = torch.empty(T, width, device=DEV), torch.empty(T, S, width, device=DEV)
        ops.streams_norm(got, X, S, w, 1e-5, stream(), read=read, update=(mix, out, (e, place, weights)), x_new=new)
        want = plain.streams_out(X.double(), y, mix.double(), out.double())
        close(new, want, torch.float32, 5e-6)
        close(got, plain.rms(plain.streams_in(want, read.double()), 1e-5) * w.double(), torch.float32, 2e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,dim,rot,dims,rank,page", [(3, 10, 6, 6, 20, 8), (8, 128, 64, 64, 512, 16), (40, 24, 8, 8, 40, 16), (1, 5, 3, 2, 7, 4), (2, 64, 32, 0, 128, 32), (17, 32, 70, 66, 300, 8)])
def test_latents_are_normed_rotated_and_stored(dtype, heads, dim, rot, dims, rank, page):
    from lucciola_b200 import ops
    from lucciola_b200.parts.rope import RotaryEmbedding
    lens, starts = [5, 1, 3], [0, 700, 14]
    step = batch_of(lens, starts)
    T = sum(lens)
    yarn = (8.0, 100, 16.0, 1.0)
    pool, table = scattered(250, page, (1, rank + rot), lens, starts, dtype)
    pre = torch.randn(T, heads * (dim + rot) + rank + rot + heads, device=DEV)
    w = torch.rand(rank, device=DEV) + 0.5
    inv, mag = None, 1.0
    if dims:
        enc = RotaryEmbedding(runtime(dtype), rot, 1000.0, dims, yarn=yarn)
        inv, mag = enc.rotary_table()[0], enc.magnitude
    q = torch.empty(T, heads, dim + rot, dtype=dtype, device=DEV)
    lat = torch.full((T, heads, rank + rot), float("nan"), dtype=dtype, device=DEV)
    c = heads * (dim + rot)
    ops.latent_rope(pre, 0, c, heads, dim, rot, rank, w, inv, dims, mag, q, lat, pool, step, table, page, 1e-5, stream())
    p, pos = pre.double().cpu(), step.positions.cpu()
    rd = {"dims": dims, "base": 1000.0, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))}
    wq = p[:, :c].reshape(T, heads, dim + rot)
    turned = plain.rotate_halves(wq[..., dim:], pos, rd)
    close(q, torch.cat([wq[..., :dim], turned], dim=-1), dtype, 2e-4)
    close(lat[..., rank:], turned, dtype, 2e-4)
    assert torch.isnan(lat[..., :rank]).all()
    want = torch.cat([plain.rms(p[:, c:c + rank], 1e-5) * w.double().cpu(), plain.rotate_halves(p[:, None, c + rank:c + rank + rot], pos, rd)[:, 0]], dim=-1)
    seq = step.token_seq.cpu().tolist()
    for t in range(T):
        at = pool[int(table[seq[t], int(pos[t]) // page]), 0, int(pos[t]) % page]
        close(at, want[t], dtype, 2e-4)
    assert int(torch.isfinite(pool[:, 0, :, 0]).sum()) == T
    # without the second copy, and an entry that owns no page writes nothing
    pool.fill_(float("nan"))
    q2 = torch.empty_like(q)
    ops.latent_rope(pre, 0, c, heads, dim, rot, rank, w, inv, dims, mag, q2, None, pool, step, torch.full_like(table, -1), page, 1e-5, stream())
    assert torch.equal(q, q2) and torch.isnan(pool).all()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,temp", [(6, 3, 12, 20, (0.4, 7)), (4, 2, 128, 128, (0.2, 1)), (3, 1, 22, 12, None), (2, 1, 7, 5, (1.5, 100)), (1, 1, 300, 40, (0.1, 3))])
def test_unit_heads_with_a_query_temperature(dtype, heads, kv, dim, vdim, temp):
    """q and k divided by their root mean square without a rotation, q times its position's temperature (positions at, before and
    behind the places where it steps)."""
    from lucciola_b200 import ops
    page, lens, starts = 8, [9, 1, 6], [0, 699, 5]
    step = batch_of(lens, starts)
    T = sum(lens)
    kc, table = scattered(120, page, (kv, dim), lens, starts, dtype)
    vc = torch.full((120, kv, page, vdim), float("nan"), dtype=dtype, device=DEV)
    c1, c2 = heads * dim, (heads + kv) * dim
    pre = torch.randn(T, c2 + kv * vdim, device=DEV)
    q = torch.empty(T, heads, dim, dtype=dtype, device=DEV)
    ops.rope_kv(pre[:, :c1], pre[:, c1:c2], pre[:, c2:], q, step.positions, heads, kv, dim, 1e-5, stream(), k_cache=kc, v_cache=vc,
                token_seq=step.token_seq, block_table=table, page_size=page, v_dim=vdim, unit=True, temperature=temp)
    p, pos = pre.double().cpu(), step.positions.cpu()
    f = plain.query_temperature(pos, dict(zip(("coef", "every"), temp)) if temp else None)
    close(q, plain.rms(p[:, :c1].reshape(T, heads, dim), 1e-5) * f[:, None, None], dtype)
    wk, wv = plain.rms(p[:, c1:c2].reshape(T, kv, dim), 1e-5), p[:, c2:].reshape(T, kv, vdim)
    seq = step.token_seq.cpu().tolist()
    for t in range(T):
        pg, slot = int(table[seq[t], int(pos[t]) // page]), int(pos[t]) % page
        close(kc[pg, :, slot], wk[t], dtype)
        close(vc[pg, :, slot], wv[t], dtype)


def test_a_temperature_beside_norm_weights_and_a_rotation():
    """The option belongs to the kernel, not to unit heads: q = temperature * rotate(norm(q) * w)."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.rope import RotaryEmbedding
    T, H, D = 12, 3, 64
    step = batch_of([T], [95])
    x, w = torch.randn(T, H * D, device=DEV), torch.rand(D, device=DEV) + 0.5
    enc = RotaryEmbedding(runtime(), D, 1000.0, 32)
    q = torch.empty(T, H, D, device=DEV)
    ops.rope_kv(x, x, x, q, step.positions, H, 0, D, 1e-5, stream(), q_norm_w=w, k_norm_w=w, inv_freq=enc.inv_freq, rot_dim=32, temperature=(0.5, 4))
    pos = step.positions.cpu()
    want = plain.rotate_halves(plain.rms(x.double().cpu().reshape(T, H, D), 1e-5) * w.double().cpu(), pos, {"dims": 32, "base": 1000.0})
    close(q, want * plain.query_temperature(pos, {"coef": 0.5, "every": 4})[:, None, None], torch.float32, 5e-5)


@pytest.mark.parametrize("experts,top", [(1, 1), (5, 2), (8, 8), (64, 6), (300, 4)])
def test_router_with_a_softmax_over_the_chosen(experts, top):
    from lucciola_b200 import ops
    T = 50
    z = torch.randn(T, experts, device=DEV) * 8
    z[0] += 90.0
    z[1] -= 300.0
    ids, wts = torch.full((T, top), -1, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.route_topk(ids, wts, z, None, 1, 1, 1.0, stream(), softmax=True)
    best = z.double().topk(top, dim=-1)
    assert torch.equal(ids.long(), best.indices)
    close(wts, torch.softmax(best.values, dim=-1), torch.float32, 2e-6)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("experts,top,width,ff,lens", [(5, 2, 70, 28, [3, 1, 9]), (1, 1, 40, 32, [1]), (16, 4, 256, 64, [1] * 8), (12, 1, 200, 72, [40]), (16, 4, 264, 64, [60]), (3, 2, 128, 128, [20, 9]),
                                                       (2, 2, 256, 64, [130, 70]), (6, 3, 128, 192, [400, 3])])
def test_experts_weighted_by_a_softmax_over_the_chosen(dtype, experts, top, width, ff, lens):
    """The whole part with independent experts: short runs of tokens and runs long enough for the tensor-memory product
    (bfloat16); the sum formed by its own kernel and left to the reader."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.experts import RoutedExperts
    rt = runtime(dtype)
    cfg = kz._config(50, width, 2, 1e-5, [kz._unit(1, 1, 8, 8, 0.3, None, kz._moe(experts, top, ff))])
    w = {k[len("l0."):]: v.to(dtype) for k, v in kz.make_weights(cfg, experts, decisive=False).items() if k.startswith("l0.mlp.")}
    part = RoutedExperts(rt, "mlp", width, experts, top, ff, "silu", 0.0, 1.0, correction=False, out_dtype=torch.float32, scores="softmax")
    part.bind_all(lambda name: w[name].to(DEV))
    T = sum(lens)
    h = torch.randn(T, width, device=DEV).to(dtype)
    sub = {k[len("mlp."):]: v.double() for k, v in w.items()}
    h64 = h.double().cpu()
    z = (h64 @ sub["router"].T).sort(dim=-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == experts else (z[:, top - 1] - z[:, top]) > 1e-4       # a tie is anyone's choice
    assert clear.sum() >= 0.9 * T
    want = plain.routed_feed_forward(h64, sub, cfg["layers"][0]["mlp"])
    step = batch_of(lens)
    got = part.forward(h, step)
    close(got.cpu()[clear], want[clear], dtype, 2e-5, 1.5e-2)
    s = part.forward(h, step, unsummed=True)
    one, zero = torch.ones(width, device=DEV), torch.zeros(T, width, device=DEV)
    out, new = torch.empty(T, width, device=DEV), torch.empty(T, 1, width, device=DEV)
    ops.streams_norm(out, zero, 1, one, 1e-5, stream(), update=(torch.ones(1, 1, device=DEV), torch.ones(1, device=DEV), (s.rows, s.place_of, s.weights)), x_new=new)
    close(new[:, 0], got.double(), torch.float32, 1e-5)
    assert ops.device_error() == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,H,K,N", [(5, 3, 16, 24), (70, 8, 128, 512), (1, 2, 64, 40), (33, 4, 10, 14), (8, 5, 512, 128), (64, 3, 512, 136), (20, 2, 200, 33), (64, 2, 1000, 40)])
def test_per_head_products_on_parts_of_heads_with_a_gate_a_head(dtype, T, H, K, N):
    from lucciola_b200 import ops
    x, y = torch.randn(T, H, K + 8, device=DEV).to(dtype), torch.full((T, H, N + 16), float("nan"), device=DEV).to(dtype)
    w = (torch.randn(H, N, K, device=DEV) / K ** 0.5).to(dtype)
    pre = torch.randn(T, 5 + H, device=DEV)
    ops.gemm_heads(y[:, :, :N], x[:, :, :K], w, stream(), gate=pre[:, 5:])
    want = torch.einsum("thk,hnk->thn", x[:, :, :K].double(), w.double())
    close(y[:, :, :N], want * torch.sigmoid(pre[:, 5:].double())[:, :, None], dtype, 1e-5)
    assert torch.isnan(y[:, :, N:]).all()


def latent_case(lens, starts, heads, dk, dv, page, dtype, seed, standout=None):
    """Queries, a pool with the cached vectors of every sequence in scrambled pages (NaN elsewhere), and the plain result for given
    scale and sinks.  standout: for each sequence the position whose vector equals (4 times) the last query of head 0."""
    g = torch.Generator(device=DEV).manual_seed(seed)
    step = batch_of(lens, starts)
    T = sum(lens)
    n_pages = sum(-(-(s + n) // page) for s, n in zip(starts, lens)) + 3
    pool, table = scattered(n_pages, page, (1, dk), lens, starts, dtype, seed)
    q = torch.randn(T, heads, dk, device=DEV, generator=g).to(dtype)
    caches, t = [], 0
    for i, (s, n) in enumerate(zip(starts, lens)):
        c = torch.randn(s + n, dk, device=DEV, generator=g).to(dtype)
        if standout is not None:
            c[min(standout, s + n - 1)] = 4.0 * q[t + n - 1, 0]
        pos = torch.arange(s + n, device=DEV)
        pool[table[i, pos // page].long(), 0, pos % page] = c
        caches.append(c)
        t += n
    step.block_tables = [table]

    def want(scale, sinks):
        out, t = torch.zeros(T, heads, dv, dtype=torch.float64, device=DEV), 0
        for c, s, n in zip(caches, starts, lens):
            c = c.double()
            sc = torch.einsum("thd,jd->htj", q[t:t + n].double(), c) * scale
            j, i = torch.arange(s + n, device=DEV)[None], torch.arange(s, s + n, device=DEV)[:, None]
            sc = sc.masked_fill(j > i, float("-inf"))
            if sinks is not None:
                sc = torch.cat([sc, sinks.double()[:, None, None].expand(heads, n, 1)], dim=-1)
            wts = torch.softmax(sc, dim=-1)[..., :s + n]
            out[t:t + n] = torch.einsum("htj,jd->thd", wts, c[:, :dv])
            t += n
        return out
    return step, q, pool, table, want


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,dk,dv,page", [(4, 26, 20, 8), (8, 576, 512, 16), (24, 224, 192, 16), (96, 48, 40, 32), (2, 112, 88, 8), (3, 128, 96, 128), (32, 576, 512, 64), (1, 160, 128, 16), (16, 320, 256, 16),
                                              (5, 72, 64, 8), (64, 576, 512, 16)])
def test_many_heads_on_one_cached_vector(dtype, heads, dk, dv, page):
    """Decoded tokens, portions and both in one batch, over keys cut into one and several ranges; a standing-out key at the first
    place, at page borders, at a stage's edge, far back and at the query's own place; sinks far below, among and far above
    the scores; what pages hold behind a sequence's end is NaN."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.attention import tiles_of
    group = next(heads // s for s in range(1, heads + 1) if heads % s == 0 and heads // s <= 64)
    scale = 1.5 / dk ** 0.5
    batches = [([1, 1, 1], [0, 333, 63], 63), ([7], [120], 0), ([70, 1, 2], [0, 64, 15], page - 1), ([1], [5 * page], 4 * page), ([33, 20], [95, 0], 10 ** 6), ([1, 1], [700, 128], 128)]
    for k, (lens, starts, spot) in enumerate(batches):
        step, q, pool, table, want = latent_case(lens, starts, heads, dk, dv, page, dtype, 100 * heads + k, spot)
        for sinks in (None, torch.randn(heads, device=DEV) * 3, torch.full((heads,), 60.0, device=DEV), torch.full((heads,), -80.0, device=DEV)):
            ref = want(scale, sinks)
            outs = []
            out = torch.full((sum(lens), heads, dv), float("nan"), dtype=dtype, device=DEV)
            ops.attention_plain(q, out, pool, pool, step.positions, step.token_seq, table, heads, 1, dk, page, 0, scale, stream(), v_dim=dv, v_stride=dk, sinks=sinks)
            outs.append(("plain", out))
            if dtype == torch.bfloat16 and ops.latent_flash_ok(dk, dv, group, page):
                for rows, splits in ((-(-group // 16) * 16, 1), (64, 1), (64, 2), (64, 5), (-(-group // 16) * 16, 3)):
                    tiles = tiles_of(lens, group, rows)
                    most = max(t[1] for t in tiles) * group
                    out = torch.full((sum(lens), heads, dv), float("nan"), dtype=dtype, device=DEV)
                    ops.latent_flash(q, out, pool, step.positions, table, torch.tensor(tiles, dtype=torch.int32, device=DEV), most, group, page, scale, splits,
                                     stream(), sinks=sinks)
                    outs.append((f"{rows} rows, {splits} ranges", out))
            for which, out in outs:
                err = (out.double() - ref).abs().max().item()
                assert err <= (3e-5 if dtype == torch.float32 else 2e-2) * max(ref.abs().max().item(), 0.3), (which, lens, starts, err)
    assert ops.device_error() == 0


@pytest.mark.parametrize("dk,page", [(48, 8), (576, 16), (8, 32)])
def test_cached_vectors_are_gathered_row_by_row(dk, page):
    from lucciola_b200 import ops
    lens, starts = [3, 20, 1, 40], [0, 60, 9, 0]
    step, _, pool, table, _ = latent_case(lens, starts, 1, dk, dk, page, torch.bfloat16, dk)
    entries, first = [], 0
    for i, rows in ((1, 128), (3, 40), (0, 7)):
        entries.append((i, first, rows, 0))
        first += rows
    out = torch.full((first, dk), float("nan"), dtype=torch.bfloat16, device=DEV)
    ops.latent_gather(out, pool, torch.tensor(entries, dtype=torch.int32, device=DEV), step.context_lens, table, page, stream())
    for i, at, rows, _ in entries:
        n = starts[i] + lens[i]
        pos = torch.arange(n, device=DEV)
        assert torch.equal(out[at:at + n], pool[table[i, pos // page].long(), 0, pos % page]) and not out[at + n:at + rows].any()


@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(8, 128, 64, 128, 512), (3, 64, 32, 64, 192), (4, 32, 16, 64, 64), (5, 8, 8, 8, 40), (2, 40, 24, 104, 88), (2, 128, 0, 72, 64), (1, 72, 64, 128, 24)])
def test_portions_on_multiplied_out_keys_and_values(heads, dim, rot, vdim, rank):
    """Several portions of one batch, from the sequence's start and from further on, in items of one and two tiles and over key
    ranges; a standing-out key at a block's edge, far back, at the query's own place and just behind it (where it must not be
    seen); sinks and gates; rows behind a request's last one hold what would show."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.attention import tiles_of
    scale = 1.5 / (dim + rot) ** 0.5
    g = torch.Generator(device=DEV).manual_seed(heads * dim)
    r = lambda *s: torch.randn(*s, device=DEV, generator=g).to(torch.bfloat16)
    for lens, starts, spot in (([300], [0], 63), ([17, 129], [200, 0], 64), ([256, 40], [128, 500], 0), ([128], [900], 899), ([33], [31], 10 ** 6)):
        step = batch_of(lens, starts)
        T = sum(lens)
        firsts, rows = [], 0
        for s, n in zip(starts, lens):
            firsts.append(rows)
            rows += s + n + 5                                              # five rows behind each request's last
        q, kv, lat = r(T, heads, dim + rot), r(rows, heads * (dim + vdim)), r(rows, rank + rot)
        t = 0
        for f, s, n in zip(firsts, starts, lens):
            last = q[t + n - 1, 0]
            for at in ({min(spot, s + n - 1), s + n} if spot < 10 ** 6 else {s + n}):       # s + n: behind the last, not visible
                kv[f + at, :dim] = 4.0 * last[:dim]
                lat[f + at, rank:] = 4.0 * last[dim:]
            t += n
        pre = torch.randn(T, heads + 3, device=DEV, generator=g)
        for sinks, gate in ((None, None), (torch.randn(heads, device=DEV, generator=g) * 3, pre[:, 3:]), (torch.full((heads,), 50.0, device=DEV), None)):
            want = torch.zeros(T, heads, vdim, dtype=torch.float64, device=DEV)
            t = 0
            for f, s, n in zip(firsts, starts, lens):
                K = torch.cat([kv[f:f + s + n, :heads * dim].reshape(s + n, heads, dim), lat[f:f + s + n, None, rank:].expand(-1, heads, -1)], dim=-1).double()
                V = kv[f:f + s + n, heads * dim:].reshape(s + n, heads, vdim).double()
                sc = torch.einsum("thd,jhd->htj", q[t:t + n].double(), K) * scale
                j, i = torch.arange(s + n, device=DEV)[None], torch.arange(s, s + n, device=DEV)[:, None]
                sc = sc.masked_fill(j > i, float("-inf"))
                if sinks is not None:
                    sc = torch.cat([sc, sinks.double()[:, None, None].expand(heads, n, 1)], dim=-1)
                want[t:t + n] = torch.einsum("htj,jhd->thd", torch.softmax(sc, dim=-1)[..., :s + n], V)
                t += n
            if gate is not None:
                want = want * torch.sigmoid(gate.double())[:, :, None]
            for size in (256, 128):
                tiles = torch.tensor([(a, n, 0, firsts[i]) for a, n, i, _ in tiles_of(lens, 1, size)], dtype=torch.int32, device=DEV)
                for splits in (1, 2, 5):
                    out = torch.full((T, heads, vdim), float("nan"), dtype=torch.bfloat16, device=DEV)
                    ops.latent_prefill(q, out, kv, lat, step.positions, tiles, dim, rot, rank, scale, stream(), sinks=sinks, gate=gate, key_splits=splits)
                    err = (out.double() - want).abs().max().item()
                    assert err <= 1.5e-2 * max(want.abs().max().item(), 0.3), (lens, starts, size, splits, err)
    assert ops.device_error() == 0


def test_padding_entries_of_a_recorded_step_read_nothing():
    """An entry that owns no page beside one that does: finite output for it, whatever page 0 holds."""
    from lucciola_b200 import ops
    heads, dk, dv, page = 4, 128, 96, 16
    step, q, pool, table, want = latent_case([1, 1], [40, 0], heads, dk, dv, page, torch.bfloat16, 3)
    table[1] = -1
    out = torch.full((2, heads, dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    pool[0] = pool[0].where(torch.tensor(bool((table == 0).any()), device=DEV), torch.tensor(float("nan"), device=DEV).to(torch.bfloat16))
    tiles = torch.tensor([(0, 1, 0, 0), (1, 1, 1, 0)], dtype=torch.int32, device=DEV)
    for splits in (1, 2):
        out.fill_(float("nan"))
        ops.latent_flash(q, out, pool, step.positions, table, tiles, heads, heads, page, 0.1, splits, stream(), sinks=torch.zeros(heads, device=DEV))
        close(out[:1], want(0.1, torch.zeros(heads, device=DEV))[:1], torch.bfloat16)
        assert torch.isfinite(out).all()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("way", ["as it comes", "multiplied out", "in latent space"])
@pytest.mark.parametrize("layer", [("C", 0), ("C", 1), ("C", 2), ("C", 3), ("C", 4), ("A", 0), ("A", 1), ("D", 0), ("D", 1)])
def test_a_mixer_alone(dtype, layer, way, monkeypatch):
    """Both kinds of mixer by themselves: a batch of unequal sequences that start at position 0, then one more token each, then
    portions behind that; latent attention also with one of its two ways forced on every portion."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.base import BatchShape, KVCacheView, PlanView
    from lucciola_b200.config.registry import resolve_architecture
    name, i = layer
    cfg = kz.CONFIGS[name]
    w = kz.make_weights(cfg, 9)
    rt = runtime(dtype)
    arch = resolve_architecture(cfg)
    model = arch.build(arch.config_from_dict(cfg), rt)
    part = model.blocks[i].mixer
    part.bind_all(lambda n: w[n].to(dtype).to(DEV))
    kind, m = cfg["layers"][i]["type"], cfg["layers"][i]["mixer"]
    if way != "as it comes":
        if kind != "latent_attention" or dtype == torch.float32:
            pytest.skip("one way only")
        monkeypatch.setattr(ops, "latent_expansion_pays", lambda *a: way == "multiplied out")
    sub = {k[len(f"l{i}.mix."):]: v.double() for k, v in w.items() if k.startswith(f"l{i}.mix.")}
    req, page = part.cache_request(), 16
    lens, more, n_pages = [40, 3, 1, 130], [17, 2, 150, 16], 40
    k_pool, table = scattered(n_pages, page, (req.num_kv_heads, req.head_dim), [n + 1 + k for n, k in zip(lens, more)], [0] * 4, dtype)
    v_pool = k_pool if req.shared else torch.full((n_pages, req.num_kv_heads, page, req.v_head_dim or req.head_dim), float("nan"), dtype=dtype, device=DEV)
    cache, past = KVCacheView(k_pool, v_pool, 0, page), [None] * len(lens)
    W = cfg["width"]
    for q_lens, starts in ((lens, [0] * 4), ([1] * 4, lens), (more, [n + 1 for n in lens])):
        step = batch_of(q_lens, starts)
        step.block_tables = [table]
        if part.plan_key() is not None:
            made = part.plan(BatchShape(list(q_lens), list(starts), max(q_lens), step.max_context_len, step.max_context_len))
            step.plans[part.plan_key()] = PlanView({k: torch.from_numpy(a).to(DEV) for k, a in made.arrays.items()}, made.host)
        h = torch.randn(sum(q_lens), W, device=DEV).to(dtype)
        got, t = part.forward(h, step, cache), 0
        for s, n in enumerate(q_lens):
            want, past[s] = plain.MIXERS[kind](h[t:t + n].double().cpu(), sub, m, cfg["norm"]["eps"], past[s])
            close(got[t:t + n], want, dtype, 3e-5, 2.5e-2)
            t += n


# ---- the whole model -------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, folder).  Beside the four: "Asharp" / "Csharp", whose attentions pick out single keys."""
    out = {}
    for name, cfg in kz.CONFIGS.items():
        w = kz.make_weights(cfg, 100 + len(out))
        out[name] = (cfg, w, kz.write_model(tmp_path_factory.mktemp(f"kifezen_{name}"), cfg, w))
    for base in ("A", "C"):
        cfg = kz.sharpened(kz.CONFIGS[base], 4.0)
        w = kz.make_weights(cfg, 200 + len(out))
        out[base + "sharp"] = (cfg, w, kz.write_model(tmp_path_factory.mktemp(f"kifezen_{base}sharp"), cfg, w))
    return out


def make_runner(models, name, dtype, num_pages, graphs=False, slots=4, **kw):
    from lucciola_b200.config import EngineOptions
    from lucciola_b200.engine.load import build_runner
    page = kz.PAGE[name[0]]
    return build_runner(models[name][2], EngineOptions(dtype=dtype, block_size=page, max_blocks=num_pages, max_num_seqs=slots,
                                                       use_cuda_graph=graphs, graph_after=1, max_shape_graphs=1000, **kw),
                        num_pages=num_pages)


TOL_SHARP = {"float32": 1e-4, "bfloat16": 0.12}


def check(models, name, dtype, steps, reqs, graphs=False, poison=True, tol=None, slots=4):
    page = kz.PAGE[name[0]]
    cfg, w, _ = models[name]
    if tol is None:
        tol = kz.bound(dtype, cfg, w, reqs, TOL_SHARP[dtype] if "sharp" in name else None)
    runner = make_runner(models, name, dtype, max(ru.max_live_tokens(steps) // page, 1), graphs=graphs, slots=slots)
    got = ru.replay(runner, steps, poison=poison)
    worst = kz.compare(got, name, cfg, w, reqs, dtype, tol)
    assert runner.manager.num_requests() == 0 and all(p.num_free == p.num_pages for p in runner.manager.pools)
    return runner, got, worst


LENGTHS = {"A": [1, 2, 15, 16, 17, 47, 130], "B": [1, 7, 8, 9, 64, 120], "C": [3, 31, 32, 33, 129, 300], "D": [1, 16, 65, 140, 400]}


def requests_for(models, name):
    cfg = models[name][0]
    return {f"{name}{n}": kz.tokens(cfg, n, salt=len(name)) for n in LENGTHS[name[0]]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "Asharp", "Csharp"])
@pytest.mark.parametrize("cut", ["whole", "tail_decoded", "portions"])
def test_each_request_alone(models, name, dtype, cut):
    """Whole prompts (lengths at and beside page borders), prompt then token-by-token decoding, and portions of
    1 to 31 tokens, each request by itself."""
    reqs = requests_for(models, name)
    check(models, name, dtype, getattr(ru, cut)(reqs), reqs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "Csharp"])
@pytest.mark.parametrize("seed", [0, 1])
def test_mixed_batches_with_reused_pages_and_slots(models, name, dtype, seed):
    """Up to four live requests of unequal length, portions beside single tokens; nine requests through four slots and
    fewer pages than they need together; what a freed page held is overwritten with NaN."""
    cfg = models[name][0]
    reqs = {f"m{i}": kz.tokens(cfg, n, salt=seed + 3) for i, n in enumerate((70, 9, 120, 33, 101, 2, 64, 47, 90))}
    steps = ru.mixed(reqs, seed=seed)
    assert ru.max_live_tokens(steps) < sum(ru.ceil64(len(v)) for v in reqs.values())
    check(models, name, dtype, steps, reqs, slots=4)
    assert max(len(s["entries"]) for s in steps) >= 3


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
@pytest.mark.parametrize("cut", ["tail_decoded", "portions", "mixed_decodes_first"])
def test_every_cutting_through_recorded_graphs(models, name, cut):
    """bfloat16 with recordings on: the trace runs twice through one runner; the second pass replays the CUDA graphs the
    first recorded, with other pages under the same requests."""
    cfg, w, _ = models[name]
    if cut.startswith("mixed"):
        reqs = {f"m{i}": kz.tokens(cfg, n, salt=5) for i, n in enumerate((70, 9, 120, 33, 101, 2, 64, 47, 90))}
        steps = ru.mixed(reqs, seed=4, decodes_first=True)
    else:
        reqs = requests_for(models, name)
        steps = getattr(ru, cut)(reqs)
    page = kz.PAGE[name[0]]
    runner = make_runner(models, name, "bfloat16", max(ru.max_live_tokens(steps) // page, 1), graphs=True)
    assert runner._can_record
    tol = kz.bound("bfloat16", cfg, w, reqs)
    first = ru.replay(runner, steps, poison=True)
    kz.compare(first, name, cfg, w, reqs, "bfloat16", tol)
    recorded, replays = len(runner._graphs), runner.graph_replays
    assert recorded > 0
    second = ru.replay(runner, steps, poison=True)
    kz.compare(second, name, cfg, w, reqs, "bfloat16", tol)
    assert len(runner._graphs) == recorded and runner.graph_replays - replays == sum(1 for s in steps if s["entries"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_cutting_does_not_change_float32_results_at_all(models, name, dtype):
    """In 32-bit every sum's order is fixed by the model's sizes alone, so whole prompts, portions, single tokens and
    mixed batches agree to the last bit; in bfloat16 within rounding."""
    reqs = requests_for(models, name)
    runs = []
    for steps in (ru.whole(reqs), ru.portions(reqs), ru.mixed(reqs, seed=3), ru.tail_decoded(reqs, tail=40)):
        runner = make_runner(models, name, dtype, 200)
        runs.append(ru.replay(runner, steps))
    common = set(runs[0]) & set(runs[1]) & set(runs[2])
    assert len(common) > 50
    for key in common:
        for other in runs[1:]:
            if key not in other:
                continue
            if dtype == "float32":
                assert torch.equal(runs[0][key], other[key]), key
            else:
                assert (runs[0][key] - other[key]).abs().max() <= 2 * kz.TOL[dtype] * runs[0][key].abs().max(), key


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["Asharp", "Csharp", "D"])
def test_long_decoding(models, name, dtype):
    """A short prompt, then hundreds of tokens decoded one by one."""
    cfg = models[name][0]
    ids = kz.tokens(cfg, 390, salt=9)
    steps = ru.tail_decoded({"long": ids}, tail=387)
    _, got, _ = check(models, name, dtype, steps, {"long": ids})
    assert len(got) == 388


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["Asharp", "Csharp"])
def test_small_faults_really_show(models, name, dtype):
    """The sharpened models must be ones in which a small fault shows: a temperature that steps one position late, a sink that
    is left out, a key that is rotated one position further, one lost token far back, each changes the logits by far more
    than the 32-bit tolerance.  Then the engine, the prompt in portions that end at, before and behind the borders of pages and
    the steps of the temperatures, against the plain implementation."""
    import json
    cfg, w, _ = models[name]
    ids = kz.tokens(cfg, 200, salt=21)
    a = kz.plain_logits(name, cfg, w, ids)
    shows = lambda b, lo=0: (a - b)[lo:].abs().max() > 20 * TOL_SHARP["float32"] * a.abs().max()
    every = next(l["mixer"]["q_temp"]["every"] for l in cfg["layers"] if l["mixer"].get("q_temp"))
    late = json.loads(json.dumps(cfg))
    for l in late["layers"]:
        if l["mixer"].get("q_temp"):
            l["mixer"]["q_temp"]["every"] += 1
    assert shows(kz.plain_logits((name, "late"), late, w, ids))
    for i, l in enumerate(cfg["layers"]):
        if l["type"] != "latent_attention":
            continue
        without = dict(w)
        without[f"l{i}.mix.sink"] = w[f"l{i}.mix.sink"] - 50.0
        assert shows(kz.plain_logits((name, "sink", i), cfg, without, ids))
    moved = plain.rotate_halves
    try:
        plain.rotate_halves = lambda x, pos, rot: moved(x, pos + (1 if x.shape[1] == 1 else 0), rot)       # the shared key part alone
        assert shows(kz.PlainKifezen(cfg, w).forward(ids))
    finally:
        plain.rotate_halves = moved
    other = list(ids)
    other[0] = (ids[0] + 1) % cfg["vocab"]
    assert shows(kz.plain_logits((name, "far"), cfg, w, other), 150)
    page = kz.PAGE[name[0]]
    steps = ru.portions({"edge": ids}, sizes=(page - 1, 2, page, page + 1, every, max(every - 1, 1), 2, every + 1, 2 * page - 2, 3, 1, 1, 2))
    check(models, name, dtype, steps, {"edge": ids})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_first_tokens_of_a_sequence(models, name, dtype):
    """Positions 0 to 5: a single key, a page with one token."""
    cfg = models[name][0]
    for n in (1, 2, 3, 6):
        ids = kz.tokens(cfg, n, salt=n)
        for steps in (ru.whole({"f": ids}), ru.tail_decoded({"f": ids}, tail=n - 1) if n > 1 else ru.whole({"f": ids})):
            check(models, name, dtype, steps, {"f": ids})


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_against_each_alone(models, dtype):
    """Five unequal prompts in one step, then their next tokens in one step: every row equals the request run alone."""
    name = "C"
    cfg = models[name][0]
    reqs = {f"b{n}": kz.tokens(cfg, n, salt=31) for n in (2, 40, 17, 128, 65)}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": ids[:-1], "want": [len(ids) - 2]} for r, ids in reqs.items()], "end": []},
             {"step": 1, "entries": [{"id": r, "tokens": ids[-1:], "want": [0]} for r, ids in reqs.items()], "end": list(reqs)}]
    _, together, _ = check(models, name, dtype, steps, reqs, slots=8)
    for r, ids in reqs.items():
        _, alone, _ = check(models, name, dtype, ru.whole({r: ids}), {r: ids})
        for p in (len(ids) - 2, len(ids) - 1):
            if dtype == "float32":
                assert torch.equal(together[(r, p)], alone[(r, p)]), (r, p)


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Every size drawn at random: the 32-bit engine must agree with the plain implementation to 32-bit rounding under
    every cutting; the bfloat16 engine within its bound."""
    from lucciola_b200.config import EngineOptions
    from lucciola_b200.engine.load import build_runner
    cfg = kz.random_config(seed)
    reqs = {f"q{i}": kz.tokens(cfg, n, salt=seed) for i, n in enumerate((1, 23, 97, 200, 64))}
    w = kz.make_weights(cfg, 300 + seed)
    folder = kz.write_model(tmp_path / "model", cfg, w)
    for dtype in DTYPES:
        for cut in ("whole", "portions", "mixed", "tail_decoded"):
            steps = getattr(ru, cut)(reqs)
            pages = max(ru.max_live_tokens(steps) // 16, 1)
            runner = build_runner(folder, EngineOptions(dtype=dtype, block_size=16, max_blocks=pages, max_num_seqs=4,
                                                        use_cuda_graph=(cut == "mixed"), graph_after=1), num_pages=pages)
            got = ru.replay(runner, steps, poison=True)
            kz.compare(got, ("drawn", seed), cfg, w, reqs, dtype, tol=5e-5 if dtype == "float32" else kz.bound(dtype, cfg, w, reqs, 5e-2))


# ---- through the entry point -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,slack", [("float32", 1e-4), ("bfloat16", 0.3)])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(models, name, dtype, slack):
    """Engine.generate with the scheduler's own batching: prompts longer than a step's budget (so they are read in
    portions beside decoding requests), more requests than slots.  Every generated token must be the plain
    implementation's choice for the same prefix, or lose to it by a near-tie."""
    from lucciola_b200 import Engine, EngineOptions, SamplingParams
    cfg, w, folder = models[name]
    eng = Engine(folder, options=EngineOptions(dtype=dtype, block_size=kz.PAGE[name[0]], max_blocks=64, max_tokens_per_step=48, max_num_seqs=3))
    prompts = [kz.tokens(cfg, n, salt=41) for n in (5, 70, 33, 1, 100)]
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert all(len(o) == 6 for o in outs)
    for prompt, out in zip(prompts, outs):
        ids = list(prompt)
        for k, tok in enumerate(out):
            row = kz.plain_logits(name, cfg, w, ids)[-1]
            assert row.max() - row[tok] <= slack * row.abs().max().clamp(min=1.0), f"token {k}: chose {tok}, plain chooses {int(row.argmax())}"
            ids.append(tok)
    assert eng.runner.manager.num_requests() == 0 and all(p.num_free == p.num_pages for p in eng.runner.manager.pools)


def test_generation_under_page_pressure_recomputes(models):
    """Fewer pages than the requests need together: a request is preempted, gives its pages and its slot back and is
    recomputed later from its prompt and what it had generated; the output is the same as with pages to spare."""
    from lucciola_b200 import Engine, EngineOptions, SamplingParams
    cfg, w, folder = models["D"]
    prompts = [kz.tokens(cfg, n, salt=51) for n in (60, 50, 40, 30)]
    params = SamplingParams(max_new_tokens=40, ignore_eos=True)
    roomy = Engine(folder, options=EngineOptions(dtype="float32", block_size=32, max_blocks=64, max_tokens_per_step=64, max_num_seqs=4))
    want = roomy.generate(prompts, params)
    tight = Engine(folder, options=EngineOptions(dtype="float32", block_size=32, max_blocks=8, max_tokens_per_step=64, max_num_seqs=4))
    got = tight.generate(prompts, params)
    assert got == want
    assert tight.stats()["preemptions"] > 0 and roomy.stats()["preemptions"] == 0


# ---- the programs ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,graphs", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
def test_trace_run_program(models, tmp_path, dtype, graphs):
    """bin/trace_run as a user runs it on a Kifezen folder: the model is chosen by config.json, steps come on standard
    input, <step>.f32 files go out; six requests through its four slots."""
    import json
    import subprocess
    import sys

    import numpy as np

    from conftest import ROOT
    name = "A"
    cfg, w, folder = models[name]
    reqs = {f"t{i}": kz.tokens(cfg, n, salt=61) for i, n in enumerate((70, 33, 90, 5, 64, 41))}
    steps = ru.mixed(reqs, seed=5, max_live=4)
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(ru.max_live_tokens(steps))] + (["--cuda-graph"] if graphs else []),
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    got, held = {}, {}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        f = out / f"{s['step']}.f32"
        assert f.exists() == (wanted > 0)
        rows = np.fromfile(f, dtype="<f4").reshape(wanted, cfg["vocab"]) if wanted else None
        r = 0
        for e in s["entries"]:
            start = held.get(e["id"], 0)
            for k in e["want"]:
                got[(e["id"], start + k)] = torch.from_numpy(rows[r].astype(np.float64)); r += 1
            held[e["id"]] = start + len(e["tokens"])
    kz.compare(got, name, cfg, w, reqs, dtype, kz.bound(dtype, cfg, w, reqs))


def test_chat_program_and_random_model_program(tmp_path):
    """bin/lucciola_random_model writes a Kifezen folder from a config.json; bin/lucciola_chat generates from it, and its
    greedy tokens are the plain implementation's."""
    import json
    import subprocess
    import sys

    from conftest import ROOT
    from lucciola_b200.weights.safetensors_io import SafetensorsFile
    cfg = kz.CONFIGS["A"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    folder = tmp_path / "model"
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "lucciola_random_model"), "--config", str(tmp_path / "config.json"), "--seed", "3",
                        "--out", str(folder), "--std", "0.2", "--norm-std", "0.1"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    prompt = kz.tokens(cfg, 19, salt=71)
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "lucciola_chat"), "--model", str(folder), "--dtype", "float32", "--max-blocks", "32",
                        "--block-size", "8", "--max-new-tokens", "5", "--ignore-eos", "--prompt-ids", " ".join(map(str, prompt))],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [int(x) for x in p.stdout.split()[-5:]]
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.get(n).clone() for n in f.names()}
    ids = list(prompt)
    for tok in out:
        row = plain.PlainKifezen(cfg, w).forward(ids)[-1]
        assert row.max() - row[tok] <= 1e-4 * row.abs().max(), (tok, int(row.argmax()))
        ids.append(tok)
