"""Nulalorn in the engine against the plain implementation: every mechanism alone, then the whole model under every way of
cutting the work, with pages that are freed and used again, and generation through the entry point (GPU)."""
from types import SimpleNamespace

import pytest
import torch

import nulalorn_util as nz
import plain_nulalorn as plain
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
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("in_dtype", TYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,dims", [(3, 1, 20, 12, 10), (4, 2, 96, 40, 26), (2, 2, 128, 128, 128), (8, 2, 64, 128, 0), (2, 1, 200, 256, 64),
                                                    (3, 1, 18, 26, 18), (2, 1, 7, 5, 2), (1, 1, 258, 3, 130)])
def test_rotation_in_pairs_with_unit_heads_behind_it(dtype, in_dtype, heads, kv, dim, vdim, dims):
    """q, k rotated by neighbours and divided by their root mean square, k and v written to scrambled pages; sizes of the
    kernel that works in registers and of the one that takes any."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.rope import NeighbourRotary
    if in_dtype == torch.bfloat16 and dtype == torch.float32:
        pytest.skip("products of the 32-bit engine are 32-bit")
    page, lens, starts = 8, [5, 1, 3], [0, 700, 14]
    step = batch_of(lens, starts)
    T = sum(lens)
    c1, c2, c3 = heads * dim, (heads + kv) * dim, (heads + kv) * dim + kv * vdim
    pre = torch.randn(T, c3, device=DEV).to(in_dtype)
    bands = (4.0, 1.0, 4.0, 64)
    enc = NeighbourRotary(runtime(dtype), dim, 1000.0, dims, bands=bands)
    inv, rot = enc.pair_table()
    width = 100
    table = torch.full((3, width), -1, dtype=torch.int32)
    free = torch.randperm(40, generator=torch.Generator().manual_seed(dim)).tolist()
    for i, (s, n) in enumerate(zip(starts, lens)):
        for pg in range(s // page, (s + n - 1) // page + 1):
            table[i, pg] = free.pop()
    kc = torch.full((40, kv, page, dim), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((40, kv, page, vdim), float("nan"), dtype=dtype, device=DEV)
    q = torch.empty(T, heads, dim, dtype=dtype, device=DEV)
    ops.rope_kv(pre[:, :c1], pre[:, c1:c2], pre[:, c2:], q, step.positions, heads, kv, dim, 1e-5, stream(), inv_freq=inv, rot_dim=rot, k_cache=kc,
                v_cache=vc, token_seq=step.token_seq, block_table=table.to(DEV), page_size=page, v_dim=vdim, pairs=True, unit=True)
    p, pos = pre.double().cpu(), step.positions.cpu()
    rd = {"dims": dims, "base": 1000.0, "scaling": dict(zip(("factor", "low", "high", "original"), bands))}
    turn = lambda x: plain.rms_norm(plain.rotate_neighbours(x, pos, rd), None, 1e-5)
    wq, wk = turn(p[:, :c1].reshape(T, heads, dim)), turn(p[:, c1:c2].reshape(T, kv, dim))
    wv = p[:, c2:].reshape(T, kv, vdim)
    # the angle is a 32-bit product: at position p it is off by up to p * 2^-24 of a turn's radian
    tol = (2e-4, 1e-2)
    close(q, wq, dtype, *tol)
    seq = step.token_seq.cpu().tolist()
    for t in range(T):
        pg, slot = int(table[seq[t], int(pos[t]) // page]), int(pos[t]) % page
        close(kc[pg, :, slot], wk[t], dtype, *tol)
        close(vc[pg, :, slot], wv[t], dtype, *tol)
    assert torch.isnan(kc).any() and int(torch.isfinite(kc[:, 0, :, 0]).sum()) == T


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("dim,dims", [(64, 32), (18, 18)])
def test_the_rotation_alone_applies_in_place(dtype, dim, dims):
    """NeighbourRotary.apply(): what a mixer that knows no pairs calls."""
    from lucciola_b200.parts.rope import NeighbourRotary
    T = 6
    q, k = torch.randn(T, 3, dim, device=DEV).to(dtype), torch.randn(T, 1, dim, device=DEV).to(dtype)
    pos = torch.tensor([0, 1, 7, 40, 300, 2], dtype=torch.int32, device=DEV)
    want = [plain.rotate_neighbours(x.double().cpu(), pos.cpu(), {"dims": dims, "base": 10000.0}) for x in (q, k)]
    enc = NeighbourRotary(runtime(dtype), dim, 10000.0, dims)
    assert enc.rotary_table() is None
    enc.apply(q, k, pos)
    close(q, want[0], dtype, 1e-4)
    close(k, want[1], dtype, 1e-4)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,width", [(7, 40), (3, 74), (5, 512), (9, 4096), (2, 8192), (2, 9000), (1, 1028), (4, 6)])
def test_two_norms_and_the_adds_between_them(dtype, rows, width):
    """Every term of the pass alone and together, with all rows and with some; the stream changes only with all rows."""
    from lucciola_b200 import ops
    r = lambda *s: torch.randn(*s, device=DEV)
    res, a0, a1, vec, yw, w = r(rows, width), r(rows, width), r(rows, width), r(width), r(width), r(width)
    for y_dtype in TYPES:
        y = (r(rows, width) * 3).to(y_dtype)
        for adds, v, have in (((), None, True), ((a0,), vec, False), ((a0, a1), vec, True), ((), None, False)):
            want = res.double()
            for a in adds:
                want = want + a.double()
            if v is not None:
                want = want + v.double()
            if have:
                want = want + plain.rms_norm(y.double(), yw.double(), 1e-4)
            kw = dict(adds=adds, vec=v, y=y if have else None, y_weight=yw if have else None, y_eps=1e-4)
            normed = plain.rms_norm(want, w.double(), 1e-5)
            got_res, out = res.clone(), torch.empty(rows, width, dtype=dtype, device=DEV)
            ops.stream_norm(got_res, stream(), out=out, weight=w, eps=1e-5, **kw)
            close(got_res, want, torch.float32)
            close(out, normed, dtype)
            pick = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32, device=DEV)
            got_res, out = res.clone(), torch.empty(3, width, dtype=dtype, device=DEV)
            ops.stream_norm(got_res, stream(), out=out, weight=w, eps=1e-5, rows=pick, **kw)
            assert torch.equal(got_res, res)
            close(out, normed[pick.long()], dtype)
            got_res = res.clone()
            ops.stream_norm(got_res, stream(), **kw)
            close(got_res, want, torch.float32)
            parts = torch.empty(2 * rows, width, dtype=torch.bfloat16, device=DEV)
            got_res = res.clone()
            ops.stream_norm(got_res, stream(), parts=(parts[:rows], parts[rows:]), **kw)
            hi, lo = parts[:rows].double(), parts[rows:].double()
            assert ((hi + lo - want).abs() <= 2.0 ** -16 * want.abs() + 1e-5).all() and torch.equal(got_res, res)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,top", [(40, 1), (74, 3), (512, 2), (4096, 4), (9000, 2)])
@pytest.mark.parametrize("shared", [False, True])
def test_the_experts_sum_inside_the_norm_and_alone(dtype, width, top, shared):
    from lucciola_b200 import ops
    T, places = 6, 40
    r = lambda *s: torch.randn(*s, device=DEV)
    e, res, yw, w = r(places, width), r(T, width), r(width), r(width)
    place = torch.randperm(places, device=DEV)[:T * top].to(torch.int32)
    s = r(T, width).to(dtype) if shared else None
    x, gate = r(T, width).to(dtype), r(width) / width ** 0.5
    for weights in (1.0 / top, torch.rand(T, top, device=DEV)):
        for g in ((gate, None) if shared else (None,)):
            wt = weights.double() if torch.is_tensor(weights) else torch.full((T, top), weights, dtype=torch.float64, device=DEV)
            y = (e.double()[place.long()].reshape(T, top, width) * wt[:, :, None]).sum(1)
            if shared:
                y = y + s.double() * (torch.sigmoid(x.double() @ g.double())[:, None] if g is not None else 1.0)
            out = torch.empty(T, width, dtype=dtype, device=DEV)
            got = res.clone()
            ops.stream_norm(got, stream(), out=out, weight=w, eps=1e-5, y_weight=yw, y_eps=1e-5,
                            experts=(e, place, weights, s, x if g is not None else None, g))
            want = res.double() + plain.rms_norm(y, yw.double(), 1e-5)
            close(got, want, torch.float32, 5e-6)
            close(out, plain.rms_norm(want, w.double(), 1e-5), dtype, 5e-6)
            alone = torch.empty(T, width, device=DEV)
            ops.expert_combine(alone, e, weights, place, stream(), always=s, gate_input=x if g is not None else None, gate_weight=g)
            close(alone, y, torch.float32, 5e-6)


@pytest.mark.parametrize("post,c", [("gelu", 0.0), ("cap", 3.0)])
@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (3, 200, 4096), (8, 4096, 512), (40, 96, 264), (130, 500, 1024), (300, 256, 64), (700, 1040, 192)])
def test_element_operations_in_the_products(post, c, M, N, K):
    """Every place where a tensor-core product stores its sums (unsplit, over a cluster, through the workspace, many tokens
    with one CTA and with pairs), and the product on the ordinary pipes."""
    from lucciola_b200 import ops
    x, w = torch.randn(M, K, device=DEV), torch.randn(N, K, device=DEV) * (2.0 / K ** 0.5)
    f = (lambda z: plain.gelu(z)) if post == "gelu" else (lambda z: plain.cap(z, c))
    y = torch.empty(M, N, device=DEV)
    ops.gemm_plain(y, x, w, stream(), post=post, post_c=c)
    close(y, f(x.double() @ w.double().T), torch.float32, 2e-5)
    xb, wb = x.to(torch.bfloat16), w.to(torch.bfloat16)
    want = f(xb.double() @ wb.double().T)
    ways = [(0, 0)] + ([(16, 1), (16, 2), (16, -2)] if M <= 16 and K >= 512 else []) + ([(-1, 0), (-2, 0)] if M >= 128 else [])
    for dt in TYPES:
        for bt, splits in ways:
            y = torch.full((M, N), float("nan"), dtype=dt, device=DEV)
            ops.gemm_tcgen05(y, xb, wb, stream(), force_bt=bt, force_splits=splits, post=post, post_c=c)
            close(y, want, dt, 2e-5)
    assert ops.device_error() == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("experts,top,width,ff,shared,lens", [(5, 2, 74, 28, 36, [3, 1, 9]), (1, 1, 40, 32, None, [1]), (16, 4, 256, 64, 64, [1] * 8), (16, 4, 200, 72, None, [5]), (4, 1, 128, 520, 24, [30]), (40, 2, 64, 16, None, [90, 3]),
                                                              (2, 2, 256, 64, 128, [130, 70]), (6, 1, 128, 152, 24, [700]), (3, 3, 64, 12, 20, [300, 5])])
def test_experts_named_by_a_table(dtype, experts, top, width, ff, shared, lens):
    """Short runs of tokens and runs long enough for the tensor-memory product (bfloat16), summed in the norm's kernel and
    alone; an expert that nobody names; a second call in one step uses the first one's sorting."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.experts import GROUPED_FROM, TableExperts
    from lucciola_b200.parts.mlp import DenseFeedForward
    rt = runtime(dtype)
    vocab = 60
    cfg = nz._config(vocab, width, 1e-5, 0.0, None, [nz._layer(1, 1, 8, 8, 0.3, 0.0, 4, None, nz._moe(experts, top, ff, shared))])
    w = {k[len("l0."):]: (v.to(dtype) if v.is_floating_point() else v) for k, v in nz.make_weights(cfg, experts).items() if k.startswith("l0.mlp.")}
    if experts > top + 1:
        w["mlp.table"] = w["mlp.table"].where(w["mlp.table"] != experts - 1, w["mlp.table"].new_tensor(-1))
        for row in w["mlp.table"]:                                    # nobody names the last expert
            for k in range(top):
                if row[k] < 0:
                    row[k] = next(e for e in range(experts - 1) if e not in row.tolist())
    sh = DenseFeedForward(rt, "mlp.shared.up", "mlp.shared.down", width, shared, act="gelu", out_dtype=torch.float32) if shared else None
    part = TableExperts(rt, "mlp", vocab, width, experts, top, ff, act="gelu", shared=sh)
    part.bind_all(lambda name: w[name].to(DEV))
    T = sum(lens)
    ids = torch.randint(0, vocab, (T,), generator=torch.Generator().manual_seed(T)).tolist()
    step = batch_of(lens, tokens=ids)
    sub = {k[len("mlp."):]: (v.double() if v.is_floating_point() else v) for k, v in w.items()}
    for _ in range(2):
        h = torch.randn(T, width, device=DEV).to(dtype)
        want = plain.expert_feed_forward(h.double().cpu(), ids, sub, cfg["layers"][0]["mlp"])
        got = part.forward(h, step)
        close(got, want, dtype, 2e-5, 1.5e-2)
        s = part.forward(h, step, unsummed=True)
        total, one = torch.zeros(T, width, device=DEV), torch.ones(width, device=DEV)
        ops.stream_norm(total, stream(), y_weight=one, y_eps=1e-5, experts=(s.rows, s.place_of, s.weights, s.always, s.gate_input, s.gate_weight))
        close(total, plain.rms_norm(got.double(), None, 1e-5), torch.float32, 1e-5)
    assert len(step.memo) == 1
    padded = next(iter(step.memo.values())).tile_group is not None
    assert padded == (dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0 and T * top >= GROUPED_FROM * experts)
    assert ops.device_error() == 0


def test_a_table_that_names_an_expert_that_is_not_there_is_refused():
    from lucciola_b200.parts.experts import TableExperts
    part = TableExperts(runtime(), "m", 4, 8, 2, 1, 8)
    get = lambda n: torch.tensor([[0], [1], [2], [0]], dtype=torch.int32) if n == "m.table" else torch.zeros(8, 8)
    with pytest.raises(ValueError):
        part.bind_all(lambda n: get(n).to(DEV))


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,width,pending", [(1, 256, True), (9, 74, True), (40, 128, False), (300, 256, True)])
def test_the_entry_of_a_pass(dtype, T, width, pending):
    """W [x ; x0] + step[t] of a stream to which a sublayer's normed output is still to be added: in the bfloat16 engine the
    stream keeps 16 of its bits through the product."""
    from lucciola_b200.parts.base import Pending
    from lucciola_b200.parts.norm import RMSNorm
    from lucciola_b200.parts.stream_entry import StreamEntry
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(T)
    w_in = (torch.randn(width, 2 * width, generator=g) / width ** 0.5).to(torch.bfloat16).to(dtype)
    steps = torch.randn(3, width, generator=g).to(torch.bfloat16).to(dtype)
    entry = StreamEntry(rt, "in", "step", width, 3)
    entry.bind(lambda n: {"in": w_in, "step": steps}[n].to(DEV))
    x0 = torch.randn(T, width, generator=g).to(torch.bfloat16)
    x, y, yw = torch.randn(T, width, generator=g) * 5, torch.randn(T, width, generator=g), torch.rand(width, generator=g) + 0.5
    norm = RMSNorm(rt, "n", width, 1e-5)
    norm.weight = yw.to(DEV)
    half = entry.embedding_half(x0.to(dtype).to(DEV))
    stream_, rest = entry.forward(x.clone().to(DEV), Pending(output=y.to(DEV), norm=norm) if pending else None, half, 1)
    assert stream_.is_contiguous()
    first = RMSNorm(rt, "f", width, 1e-5)
    first.weight = torch.ones(width, device=DEV)
    h = first.add_forward(stream_, rest, torch.float32)
    xx = x.double() + (plain.rms_norm(y.double(), yw.double(), 1e-5) if pending else 0.0)
    want = torch.cat([xx, x0.double()], dim=-1) @ w_in.double().T + steps.double()[1]
    close(stream_, want, dtype, 1e-5, 3e-5)
    close(h, plain.rms_norm(want, None, 1e-5), dtype, 1e-5, 3e-5)


def test_the_embedding_writes_its_rows_twice_in_either_type():
    from lucciola_b200 import ops
    table = torch.randn(20, 36, device=DEV).to(torch.bfloat16)
    ids = torch.tensor([3, 19, 0, 3], dtype=torch.int32, device=DEV)
    for dt in TYPES:
        a, b = torch.empty(4, 36, device=DEV), torch.full((4, 36), float("nan"), dtype=dt, device=DEV)
        ops.embedding(a, ids, table, stream(), copy=b)
        assert torch.equal(a, table[ids.long()].float()) and torch.equal(b.float(), a)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,page,size,cap", [(3, 1, 20, 12, 8, 24, 9.0), (4, 2, 64, 64, 16, 40, 12.0), (8, 2, 128, 128, 16, 33, 15.0), (2, 1, 64, 128, 16, 20, 11.0),
                                                             (8, 8, 88, 40, 32, 70, 12.0), (16, 1, 128, 64, 8, 12, 10.0), (4, 4, 128, 128, 64, 64, 14.0), (1, 1, 16, 24, 8, 1, 8.0),
                                                             (4, 2, 72, 128, 16, 50, 0.0), (6, 2, 104, 56, 128, 100, 13.0), (2, 2, 128, 128, 12, 30, 9.0)])
def test_a_query_finds_its_one_key_at_every_edge(dtype, heads, kv, dim, vdim, page, size, cap):
    """Keys and values of a long sequence in pages that lie in a scrambled order; what the window can no longer reach is
    overwritten with NaN.  One key far above all others stands in turn at the first place the last query sees, at the
    place before it, at the last query's own place, far back, and at a page's first and last slot; the query is the last
    token alone (a decoded token) or the last of a portion that crosses the edge.  Scores are capped, values have sizes of
    their own.  The kernels must agree with a plain softmax over exactly the visible keys."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.attention import plan_tiles
    from lucciola_b200.parts.base import BatchShape, PlanView
    n = 4 * size + 2 * page + 27
    g = torch.Generator(device=DEV).manual_seed(n + heads)
    last = n - 1
    first_seen = max(0, last - size + 1)
    spots = {first_seen, max(0, first_seen - 1), last, 0, (first_seen // page) * page, min(last, (first_seen // page) * page + page - 1)}
    scale = 0.25
    pages = -(-n // page)
    table = torch.arange(pages, dtype=torch.int32, device=DEV).flip(0).reshape(1, pages).contiguous()
    per = heads // kv
    for spot in sorted(spots):
        K = torch.randn(n, kv, dim, device=DEV, generator=g)
        V = torch.randn(n, kv, vdim, device=DEV, generator=g)
        longest = min(37, n - 1)
        q = torch.randn(longest, heads, dim, device=DEV, generator=g)
        K[spot] = 4.0 * q[-1].reshape(kv, per, dim)[:, 0]
        kc = torch.zeros(pages, kv, page, dim, dtype=dtype, device=DEV)
        vc = torch.zeros(pages, kv, page, vdim, dtype=dtype, device=DEV)
        pos = torch.arange(n, device=DEV)
        kc[table[0, pos // page].long(), :, pos % page] = K.to(dtype)
        vc[table[0, pos // page].long(), :, pos % page] = V.to(dtype)
        gone = torch.arange(0, max(0, n - longest - size + 1), device=DEV)
        gone = gone[(gone // page) < (max(0, n - longest - size + 1) // page)]                       # whole pages only
        if gone.numel():
            kc[table[0, gone // page].long(), :, gone % page] = float("nan")
            vc[table[0, gone // page].long(), :, gone % page] = float("nan")
        Kc, Vc = K.to(dtype).double(), V.to(dtype).double()
        for qs, starts in (([1], [last]), ([3], [n - 3]), ([longest], [n - longest]), ([1, longest], [last, n - longest]), ([2, 1, 5], [n - 2, last, n - 5])):
            step = batch_of(qs, starts)
            tb = table.repeat(len(qs), 1).contiguous()
            qq = torch.cat([q[longest - (n - st): longest - (n - st) + c] for c, st in zip(qs, starts)]).to(dtype).contiguous()
            T = sum(qs)
            outs = []
            out = torch.full((T, heads, vdim), float("nan"), dtype=dtype, device=DEV)
            ops.attention_plain(qq, out, kc, vc, step.positions, step.token_seq, tb, heads, kv, dim, page, size, scale, stream(), v_dim=vdim, softcap=cap)
            outs.append(("plain", out))
            if dtype == torch.bfloat16 and ops.attention_flash_ok(qq, heads, kv, dim, vdim):
                made = plan_tiles(BatchShape(list(qs), list(starts), max(qs), n, n), per)
                view = PlanView({k: torch.from_numpy(a).to(DEV) for k, a in made.arrays.items()}, made.host)
                step.block_tables = [tb]
                out = torch.full((T, heads, vdim), float("nan"), dtype=dtype, device=DEV)
                ops.attention(qq, out, kc, vc, step, 0, heads, kv, dim, page, size, scale, stream(), plan=view, v_dim=vdim, softcap=cap)
                outs.append(("tensor cores", out))
                rows = min(made.host["rows"]["all"], 64)
                for splits, ws, tma in ((1, False, True), (1, False, False), (2, False, True), (2, False, False), (3, True, True), (3, True, False)):
                    if splits > 1 and not ws and rows > 16:
                        ws = True                                    # only tiles of at most 16 rows combine in a cluster
                    out = torch.full((T, heads, vdim), float("nan"), dtype=dtype, device=DEV)
                    ops.attention_flash(qq, out, kc, vc, step.positions, tb, view.arrays["all"], rows, heads, kv, dim, page, size, scale, splits,
                                        stream(), force_workspace=ws, tma=tma, v_dim=vdim, softcap=cap)
                    outs.append((f"tensor cores, {splits} key ranges, workspace {ws}, TMA {tma}", out))
                if vdim == 128 == dim and "big" in view.arrays and ops.attention_tcgen05_ok(qq, heads, kv, dim, page, pages):
                    for splits in (1, 2):
                        out = torch.full((T, heads, vdim), float("nan"), dtype=dtype, device=DEV)
                        ops.attention_tcgen05(qq, out, kc, vc, step.positions, tb, view.arrays["big"], heads, kv, dim, page, size, scale, stream(),
                                              key_splits=splits, softcap=cap)
                        outs.append((f"tensor memory, {splits} key ranges", out))
            posn = step.positions.cpu().tolist()
            want = torch.zeros(T, heads, vdim, dtype=torch.float64, device=DEV)
            for r, i in enumerate(posn):
                lo = max(0, i - size + 1)
                for j in range(kv):
                    s = plain.cap(qq[r, j * per:(j + 1) * per].double() @ Kc[lo:i + 1, j].T * scale, cap)
                    want[r, j * per:(j + 1) * per] = torch.softmax(s, dim=-1) @ Vc[lo:i + 1, j]
            for which, out in outs:
                o = out.double()
                if which.startswith("tensor memory"):                   # entries of few tokens are not that kernel's
                    big = torch.tensor([c >= 16 for c in qs for _ in range(c)], device=DEV)
                    o, ref = o[big], want[big]
                else:
                    ref = want
                err = (o - ref).abs().max().item()
                assert err <= (1e-5 if dtype == torch.float32 else 3e-2) * max(ref.abs().max().item(), 0.3), (which, spot, qs, err)
    assert ops.device_error() == 0


@pytest.mark.parametrize("scale,cap,terms", [(0.1, 30.0, 5), (0.12, 20.0, 7), (0.09, 12.0, 7), (0.2, 10.0, 0), (0.9, 90.0, 0)])
@pytest.mark.parametrize("heads,kv,window", [(4, 2, 33), (8, 1, 100), (2, 2, 0)])
def test_capped_scores_with_a_known_bound(scale, cap, terms, heads, kv, window):
    """Heads of unit mean square: the cap as a polynomial without a running maximum where the bound allows it, and the
    ordinary way where it does not, agree with a plain softmax; the key that equals the query stands at the bound itself, inside
    the window, at its first place and at the place before it."""
    from lucciola_b200 import ops
    from lucciola_b200.parts.attention import plan_tiles
    from lucciola_b200.parts.base import BatchShape
    D, page, n, T = 128, 16, 330, 200
    coef = ops.cap_polynomial(scale, cap, 1.02 * D)
    assert (len(coef) if coef else 0) == terms
    if coef:
        s = torch.linspace(-D, D, 5001, dtype=torch.float64)
        got = s * sum(c * s ** (2 * i) for i, c in enumerate(coef))
        assert (got - cap * torch.tanh(s * scale / cap) / torch.log(torch.tensor(2.0, dtype=torch.float64))).abs().max() <= 1e-5
    g = torch.Generator(device=DEV).manual_seed(heads)
    unit = lambda x: x / x.pow(2).mean(-1, keepdim=True).sqrt()
    per = heads // kv
    table = torch.randperm(-(-n // page), generator=g, device=DEV).to(torch.int32).reshape(1, -1)
    for back in (0, 1, max(window - 1, 5), window or 50):
        q, K, V = unit(torch.randn(T, heads, D, device=DEV, generator=g)), unit(torch.randn(n, kv, D, device=DEV, generator=g)), torch.randn(n, kv, D, device=DEV, generator=g)
        for t in range(0, T, 37):
            K[n - T + t - back] = q[t].reshape(kv, per, D)[:, 0] * (1.0 if t % 2 else -1.0)
        kc = torch.full((table.shape[1], kv, page, D), float("nan"), dtype=torch.bfloat16, device=DEV)
        vc = kc.clone()
        pos = torch.arange(n, device=DEV)
        kc[table[0, pos // page].long(), :, pos % page] = K.to(torch.bfloat16)
        vc[table[0, pos // page].long(), :, pos % page] = V.to(torch.bfloat16)
        qb, Kd, Vd = q.to(torch.bfloat16), K.to(torch.bfloat16).double(), V.to(torch.bfloat16).double()
        step = batch_of([T], [n - T])
        made = plan_tiles(BatchShape([T], [n - T], T, n, n), per)
        tiles = torch.from_numpy(made.arrays["big"]).to(DEV)
        i = torch.arange(n - T, n, device=DEV)[:, None]
        j = torch.arange(n, device=DEV)[None]
        seen = (j <= i) & ((j > i - window) if window else (j >= 0))
        want = torch.zeros(T, heads, D, dtype=torch.float64, device=DEV)
        for h in range(heads):
            s = plain.cap(qb[:, h].double() @ Kd[:, h // per].T * scale, cap).masked_fill(~seen, float("-inf"))
            want[:, h] = torch.softmax(s, dim=-1) @ Vd[:, h // per]
        for splits in (1, 3):
            out = torch.full((T, heads, D), float("nan"), dtype=torch.bfloat16, device=DEV)
            ops.attention_tcgen05(qb, out, kc, vc, step.positions, table, tiles, heads, kv, D, page, window, scale, stream(), key_splits=splits,
                                  softcap=cap, score_bound=1.02 * D)
            close(out, want, torch.bfloat16, rounded=1.2e-2)
    assert ops.device_error() == 0


# ---- the whole model -------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, folder).  Beside the four: "Asharp" / "Csharp", whose attentions pick out single keys."""
    out = {}
    for name, cfg in nz.CONFIGS.items():
        w = nz.make_weights(cfg, 100 + len(out))
        out[name] = (cfg, w, nz.write_model(tmp_path_factory.mktemp(f"nulalorn_{name}"), cfg, w))
    for base in ("A", "C"):
        cfg = nz.sharpened(nz.CONFIGS[base], 4.0)
        w = nz.make_weights(cfg, 200 + len(out))
        out[base + "sharp"] = (cfg, w, nz.write_model(tmp_path_factory.mktemp(f"nulalorn_{base}sharp"), cfg, w))
    return out


def make_runner(models, name, dtype, num_pages, graphs=False, slots=4, **kw):
    from lucciola_b200.config import EngineOptions
    from lucciola_b200.engine.load import build_runner
    page = nz.PAGE[name[0]]
    return build_runner(models[name][2], EngineOptions(dtype=dtype, block_size=page, max_blocks=num_pages, max_num_seqs=slots,
                                                       use_cuda_graph=graphs, graph_after=1, max_shape_graphs=1000, **kw),
                        num_pages=num_pages)


TOL_SHARP = {"float32": 1e-4, "bfloat16": 0.12}


def check(models, name, dtype, steps, reqs, graphs=False, poison=True, tol=None, slots=4):
    page = nz.PAGE[name[0]]
    cfg, w, _ = models[name]
    if tol is None:
        tol = nz.bound(dtype, cfg, w, reqs, TOL_SHARP[dtype] if "sharp" in name else None)
    runner = make_runner(models, name, dtype, max(ru.max_live_tokens(steps) // page, 1), graphs=graphs, slots=slots)
    got = ru.replay(runner, steps, poison=poison)
    worst = nz.compare(got, name, cfg, w, reqs, dtype, tol)
    assert runner.manager.num_requests() == 0 and all(p.num_free == p.num_pages for p in runner.manager.pools)
    return runner, got, worst


LENGTHS = {"A": [1, 2, 15, 16, 17, 47, 130], "B": [1, 7, 8, 9, 64, 120], "C": [3, 31, 32, 33, 129, 300], "D": [1, 16, 65, 140, 400]}


def requests_for(models, name):
    cfg = models[name][0]
    return {f"{name}{n}": nz.tokens(cfg, n, salt=len(name)) for n in LENGTHS[name[0]]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "Asharp", "Csharp"])
@pytest.mark.parametrize("cut", ["whole", "tail_decoded", "portions"])
def test_each_request_alone(models, name, dtype, cut):
    """Whole prompts (lengths at and beside page borders and windows), prompt then token-by-token decoding, and portions of
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
    reqs = {f"m{i}": nz.tokens(cfg, n, salt=seed + 3) for i, n in enumerate((70, 9, 120, 33, 101, 2, 64, 47, 90))}
    steps = ru.mixed(reqs, seed=seed)
    assert ru.max_live_tokens(steps) < sum(ru.ceil64(len(v)) for v in reqs.values())
    check(models, name, dtype, steps, reqs, slots=4)
    assert max(len(s["entries"]) for s in steps) >= 3


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
@pytest.mark.parametrize("cut", ["tail_decoded", "portions", "mixed_decodes_first"])
def test_every_cutting_through_recorded_graphs(models, name, cut):
    """bfloat16 with recordings on: the trace runs twice through one runner; the second pass replays the CUDA graphs the
    first recorded, with other pages under the same requests (and other tokens under the experts' sorting)."""
    cfg, w, _ = models[name]
    if cut.startswith("mixed"):
        reqs = {f"m{i}": nz.tokens(cfg, n, salt=5) for i, n in enumerate((70, 9, 120, 33, 101, 2, 64, 47, 90))}
        steps = ru.mixed(reqs, seed=4, decodes_first=True)
    else:
        reqs = requests_for(models, name)
        steps = getattr(ru, cut)(reqs)
    page = nz.PAGE[name[0]]
    runner = make_runner(models, name, "bfloat16", max(ru.max_live_tokens(steps) // page, 1), graphs=True)
    assert runner._can_record
    tol = nz.bound("bfloat16", cfg, w, reqs)
    first = ru.replay(runner, steps, poison=True)
    nz.compare(first, name, cfg, w, reqs, "bfloat16", tol)
    recorded, replays = len(runner._graphs), runner.graph_replays
    assert recorded > 0
    second = ru.replay(runner, steps, poison=True)
    nz.compare(second, name, cfg, w, reqs, "bfloat16", tol)
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
                assert (runs[0][key] - other[key]).abs().max() <= 2 * nz.TOL[dtype] * runs[0][key].abs().max(), key


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["Asharp", "Csharp", "D"])
def test_long_decoding_past_windows(models, name, dtype):
    """A short prompt, then hundreds of tokens decoded one by one: every window passes over decoded tokens (pages are given
    back as it does)."""
    cfg = models[name][0]
    ids = nz.tokens(cfg, 390, salt=9)
    steps = ru.tail_decoded({"long": ids}, tail=387)
    _, got, _ = check(models, name, dtype, steps, {"long": ids})
    assert len(got) == 388


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("Asharp", 0), ("Asharp", 2), ("Csharp", 0), ("Csharp", 2)])
def test_the_edges_of_windows_really_matter(models, name, layer, dtype):
    """The sharpened models must be ones in which single keys matter: letting one layer's window see one token more or one
    less changes the logits by far more than the 32-bit tolerance.  Then the engine, the prompt in portions that end at,
    before and behind the borders of pages and windows, against the plain implementation."""
    import json
    cfg, w, _ = models[name]
    size = cfg["layers"][layer]["mixer"]["mask"]["size"]
    ids = nz.tokens(cfg, 200, salt=21)
    a = nz.plain_logits(name, cfg, w, ids)
    for other in (size - 1, size + 1):
        moved = json.loads(json.dumps(cfg))
        moved["layers"][layer]["mixer"]["mask"]["size"] = other
        b = nz.plain_logits((name, layer, other), moved, w, ids)
        assert (a - b)[size:].abs().max() > 20 * TOL_SHARP["float32"] * a.abs().max()
    page = nz.PAGE[name[0]]
    steps = ru.portions({"edge": ids}, sizes=(page - 1, 2, page, page + 1, size, size - 1 or 1, 2, size + 1, 2 * page - 2, 3, 1, 1, 2))
    check(models, name, dtype, steps, {"edge": ids})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_first_tokens_of_a_sequence(models, name, dtype):
    """Positions 0 to 5: a single key, fewer tokens than a window holds, a page with one token."""
    cfg = models[name][0]
    for n in (1, 2, 3, 6):
        ids = nz.tokens(cfg, n, salt=n)
        for steps in (ru.whole({"f": ids}), ru.tail_decoded({"f": ids}, tail=n - 1) if n > 1 else ru.whole({"f": ids})):
            check(models, name, dtype, steps, {"f": ids})


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_against_each_alone(models, dtype):
    """Five unequal prompts in one step, then their next tokens in one step: every row equals the request run alone."""
    name = "C"
    cfg = models[name][0]
    reqs = {f"b{n}": nz.tokens(cfg, n, salt=31) for n in (2, 40, 17, 128, 65)}
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
    cfg = nz.random_config(seed)
    reqs = {f"q{i}": nz.tokens(cfg, n, salt=seed) for i, n in enumerate((1, 23, 97, 200, 64))}
    w = nz.make_weights(cfg, 300 + seed)
    folder = nz.write_model(tmp_path / "model", cfg, w)
    for dtype in DTYPES:
        for cut in ("whole", "portions", "mixed", "tail_decoded"):
            steps = getattr(ru, cut)(reqs)
            pages = max(ru.max_live_tokens(steps) // 16, 1)
            runner = build_runner(folder, EngineOptions(dtype=dtype, block_size=16, max_blocks=pages, max_num_seqs=4,
                                                        use_cuda_graph=(cut == "mixed"), graph_after=1), num_pages=pages)
            got = ru.replay(runner, steps, poison=True)
            nz.compare(got, ("drawn", seed), cfg, w, reqs, dtype, tol=5e-5 if dtype == "float32" else nz.bound(dtype, cfg, w, reqs, 5e-2))


# ---- through the entry point -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,slack", [("float32", 1e-4), ("bfloat16", 0.3)])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(models, name, dtype, slack):
    """Engine.generate with the scheduler's own batching: prompts longer than a step's budget (so they are read in
    portions beside decoding requests), more requests than slots.  Every generated token must be the plain
    implementation's choice for the same prefix, or lose to it by a near-tie."""
    from lucciola_b200 import Engine, EngineOptions, SamplingParams
    cfg, w, folder = models[name]
    eng = Engine(folder, options=EngineOptions(dtype=dtype, block_size=nz.PAGE[name[0]], max_blocks=64, max_tokens_per_step=48, max_num_seqs=3))
    prompts = [nz.tokens(cfg, n, salt=41) for n in (5, 70, 33, 1, 100)]
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert all(len(o) == 6 for o in outs)
    for prompt, out in zip(prompts, outs):
        ids = list(prompt)
        for k, tok in enumerate(out):
            row = nz.plain_logits(name, cfg, w, ids)[-1]
            assert row.max() - row[tok] <= slack * row.abs().max().clamp(min=1.0), f"token {k}: chose {tok}, plain chooses {int(row.argmax())}"
            ids.append(tok)
    assert eng.runner.manager.num_requests() == 0 and all(p.num_free == p.num_pages for p in eng.runner.manager.pools)


def test_generation_under_page_pressure_recomputes(models):
    """Fewer pages than the requests need together: a request is preempted, gives its pages and its slot back and is
    recomputed later from its prompt and what it had generated; the output is the same as with pages to spare."""
    from lucciola_b200 import Engine, EngineOptions, SamplingParams
    cfg, w, folder = models["D"]                # its windows are longer than the sequences: pages are kept
    prompts = [nz.tokens(cfg, n, salt=51) for n in (60, 50, 40, 30)]
    params = SamplingParams(max_new_tokens=40, ignore_eos=True)
    roomy = Engine(folder, options=EngineOptions(dtype="float32", block_size=16, max_blocks=64, max_tokens_per_step=64, max_num_seqs=4))
    want = roomy.generate(prompts, params)
    tight = Engine(folder, options=EngineOptions(dtype="float32", block_size=16, max_blocks=16, max_tokens_per_step=64, max_num_seqs=4))
    got = tight.generate(prompts, params)
    assert got == want
    assert tight.stats()["preemptions"] > 0 and roomy.stats()["preemptions"] == 0


# ---- the programs ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,graphs", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
def test_trace_run_program(models, tmp_path, dtype, graphs):
    """bin/trace_run as a user runs it on a Nulalorn folder: the model is chosen by config.json, steps come on standard
    input, <step>.f32 files go out; six requests through its four slots."""
    import json
    import subprocess
    import sys

    import numpy as np

    from conftest import ROOT
    name = "A"
    cfg, w, folder = models[name]
    reqs = {f"t{i}": nz.tokens(cfg, n, salt=61) for i, n in enumerate((70, 33, 90, 5, 64, 41))}
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
    nz.compare(got, name, cfg, w, reqs, dtype, nz.bound(dtype, cfg, w, reqs))


def test_chat_program_and_random_model_program(tmp_path):
    """bin/lucciola_random_model writes a Nulalorn folder from a config.json; bin/lucciola_chat generates from it, and its
    greedy tokens are the plain implementation's."""
    import json
    import subprocess
    import sys

    from conftest import ROOT
    from lucciola_b200.weights.safetensors_io import SafetensorsFile
    cfg = nz.CONFIGS["A"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    folder = tmp_path / "model"
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "lucciola_random_model"), "--config", str(tmp_path / "config.json"), "--seed", "3",
                        "--out", str(folder), "--std", "0.2", "--norm-std", "0.1"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    prompt = nz.tokens(cfg, 19, salt=71)
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "lucciola_chat"), "--model", str(folder), "--dtype", "float32", "--max-blocks", "32",
                        "--block-size", "8", "--max-new-tokens", "5", "--ignore-eos", "--prompt-ids", " ".join(map(str, prompt))],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [int(x) for x in p.stdout.split()[-5:]]
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.get(n).clone() for n in f.names()}
    ids = list(prompt)
    for tok in out:
        row = plain.PlainNulalorn(cfg, w).forward(ids)[-1]
        assert row.max() - row[tok] <= 1e-4 * row.abs().max(), (tok, int(row.argmax()))
        ids.append(tok)
