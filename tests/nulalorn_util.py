"""Tiny Nulalorn configurations with weights made here, model folders of them, and the comparison of what the engine
returns with the plain implementation (plain_nulalorn.py)."""
from __future__ import annotations

import json
import random

import torch

from plain_nulalorn import PlainNulalorn


def _rot(dims, base, bands=None):
    r = {"dims": dims, "base": base}
    if bands is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return r


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        d["shared"] = {"ff": shared}
    return d


def _layer(heads, kv_heads, dim, vdim, scale, softcap, window, rot, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = rot
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _config(vocab, width, eps, cap, loop, layers):
    d = {"architecture": "Nulalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap:
        d["logit_softcap"] = cap
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# A: sizes that are no multiples of 8 (the bfloat16 engine falls back to its plain products), values smaller and larger than
#    keys, windows shorter than two pages, scaled frequencies on part of a head, a loop over the two middle layers, experts
#    with and without a shared one, a layer without feed-forward, rows that are no multiple of four.
# B: everything that can be 1 is 1: one head each, a window of one token, one expert of which one is used, one pass of the
#    loop (its entry still in front of it), no caps, no rotation in one layer and the whole head in another.
# C: sizes at which the bfloat16 engine takes its tensor-core kernels: key and value heads of 64 and 128 in every pairing,
#    windows across several pages and none at all, as many kv heads as heads, three passes, experts whose runs of tokens are long
#    enough for the tensor-memory product beside ones whose runs are short.
# D: windows longer than any test sequence, the loop over all layers, sizes inside the kernels' padding, no logit cap.
CONFIGS = {
    "A": _config(211, 74, 1e-5, 8.0, (1, 3, 2), [
        _layer(3, 1, 20, 12, 0.25, 6.0, 10, _rot(10, 1000.0, (4.0, 1.0, 4.0, 64)), _dense(100)),
        _layer(4, 2, 18, 26, 0.22, 9.0, 24, _rot(18, 500.0), _moe(5, 2, 28, 36)),
        _layer(2, 2, 24, 24, 0.3, 4.0, 6, _rot(4, 10000.0, (8.0, 0.5, 2.0, 32)), _moe(3, 1, 44)),
        _layer(4, 1, 12, 28, 0.3, 5.0, 24, _rot(12, 100.0), None)]),
    "B": _config(97, 40, 1e-6, 0.0, (0, 1, 1), [
        _layer(1, 1, 16, 16, 0.25, 0.0, 1, None, _moe(1, 1, 32)),
        _layer(1, 1, 16, 24, 0.3, 2.0, 1, _rot(16, 100.0, (1.0, 1.0, 2.0, 8)), None)]),
    "C": _config(331, 256, 1e-5, 20.0, (1, 3, 3), [
        _layer(8, 2, 64, 64, 0.125, 10.0, 33, _rot(32, 500000.0, (8.0, 1.0, 4.0, 256)), _dense(512)),
        _layer(4, 2, 128, 128, 0.09, 12.0, 70, _rot(128, 10000.0), _moe(2, 2, 64, 128)),
        _layer(4, 4, 64, 128, 0.125, 7.0, 40, _rot(64, 10000.0, (2.0, 1.0, 3.0, 100)), _moe(16, 4, 64, 64)),
        _layer(8, 2, 128, 64, 0.09, 9.0, 0, _rot(64, 10000.0), _moe(12, 1, 72))]),
    "D": _config(150, 256, 1e-6, 0.0, (0, 3, 2), [
        _layer(6, 2, 72, 40, 0.11, 15.0, 1000, _rot(24, 10000.0), _dense(128)),
        _layer(2, 1, 128, 128, 0.09, 20.0, 1000, _rot(64, 300000.0), _moe(6, 3, 40, 24)),
        _layer(3, 3, 48, 104, 0.14, 0.0, 1000, _rot(48, 10000.0, (4.0, 1.0, 4.0, 512)), None)]),
}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 16}


def sharpened(cfg: dict, factor: float) -> dict:
    """The same design with steeper scores and wider caps, so that a few keys carry a query's whole weight and one that is
    lost, misplaced or wrongly let through an edge changes the output by its full size.  (The queries have unit mean
    square, so larger weights would change nothing.)"""
    cfg = json.loads(json.dumps(cfg))
    for layer in cfg["layers"]:
        layer["mixer"]["scale"] *= factor
        if layer["mixer"].get("softcap"):
            layer["mixer"]["softcap"] *= factor
    return cfg


def make_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16 as a checkpoint holds them; the experts' tables as int32."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    rnd = lambda *shape, std=1.0: torch.randn(*shape, generator=g) * std
    lin = lambda o, i, gain=1.0: rnd(o, i, std=gain / i ** 0.5)
    w = {"embed": rnd(V, W), "head": lin(V, W, 3.0), "final.norm": 1 + rnd(W, std=0.2)}
    loop = cfg.get("loop")
    if loop is not None and loop["stop"] > loop["start"]:
        w["loop.in"], w["loop.step"] = lin(W, 2 * W), rnd(loop["times"], W, std=0.5)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = 1 + rnd(W, std=0.2), 1 + rnd(W, std=0.2)
        w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"], w[p + "mix.o"] = lin(H * D, W), lin(G * D, W), lin(G * Vd, W), lin(W, H * Vd)
        f = layer["mlp"]
        if f is None:
            continue
        w[p + "norm2"], w[p + "norm2b"] = 1 + rnd(W, std=0.2), 1 + rnd(W, std=0.2)
        q = p + "mlp."
        if f["kind"] == "dense":
            w[q + "up"], w[q + "down"] = lin(f["ff"], W, 1.5), lin(W, f["ff"])
            continue
        E, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
        for j in range(E):
            w[q + f"e{j}.up"], w[q + f"e{j}.down"] = lin(ff, W, 1.5), lin(W, ff)
        w[q + "table"] = torch.rand(V, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32)
        if f.get("shared") is not None:
            s = f["shared"]["ff"]
            w[q + "shared.up"], w[q + "shared.down"], w[q + "shared.sg"] = lin(s, W, 1.5), lin(W, s), lin(1, W, 2.0)
    return {k: v.to(torch.bfloat16) if v.is_floating_point() else v for k, v in w.items()}


def write_model(folder, cfg: dict, weights: dict[str, torch.Tensor]):
    from lucciola_b200.weights.safetensors_io import write_safetensors
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", weights)
    return folder


def tokens(cfg: dict, n: int, salt: int = 0) -> list[int]:
    g = torch.Generator().manual_seed(7919 * salt + n)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


_plain: dict = {}


def plain_logits(key, cfg: dict, weights: dict, ids: list[int]) -> torch.Tensor:
    """Float64 logits of the whole sequence at every position, by the plain implementation (cached)."""
    k = (key, tuple(ids))
    if k not in _plain:
        _plain[k] = PlainNulalorn(cfg, weights).forward(ids)
    return _plain[k]


# Largest |engine - plain| as a fraction of the sequence's largest |logit|.
TOL = {"float32": 3e-5, "bfloat16": 4e-2}


def compare(got: dict, key, cfg: dict, weights: dict, reqs: dict[str, list[int]], dtype: str, tol=None) -> float:
    """`tol`: one bound, or one for each request (see bound)."""
    bounds = tol if isinstance(tol, dict) else {rid: (TOL[dtype] if tol is None else tol) for rid in reqs}
    worst = 0.0
    assert got, "the trace asked for no logits"
    for rid, ids in reqs.items():
        ref = plain_logits(key, cfg, weights, ids)
        scale = ref.abs().max().item()
        tol = bounds[rid]
        for p in range(len(ids)):
            if (rid, p) not in got:
                continue
            row = got[(rid, p)]
            assert torch.isfinite(row).all(), f"request {rid} position {p}: logits are not finite"
            err = (row - ref[p]).abs().max().item() / scale
            assert err <= tol, f"request {rid}: first wrong position {p} (error {err:.3g} of scale, allowed {tol:.3g})"
            worst = max(worst, err)
    return worst


def rounding_alone(cfg: dict, weights: dict, ids: list[int]) -> float:
    """What rounding alone does to this model's logits: the largest change, as a fraction of the largest |logit|, when
    the plain implementation rounds to bfloat16 wherever a 16-bit engine may (the inputs of products, what the cache
    holds: plain_nulalorn.ROUND) and nothing else."""
    import plain_nulalorn as plain
    exact = PlainNulalorn(cfg, weights).forward(ids)
    try:
        plain.ROUND = lambda x: x.to(torch.bfloat16).to(torch.float64)
        rounded = PlainNulalorn(cfg, weights).forward(ids)
    finally:
        plain.ROUND = None
    return ((rounded - exact).abs().max() / exact.abs().max()).item()


_rounding: dict = {}


def bound(dtype: str, cfg: dict, weights: dict, reqs: dict, base: float | None = None) -> dict:
    """The bound of a comparison, request by request: the type's own, or for bfloat16 three times what rounding alone
    does to this model on that request if that is more."""
    base = TOL[dtype] if base is None else base
    if dtype != "bfloat16":
        return {rid: base for rid in reqs}
    out = {}
    for rid, ids in reqs.items():
        k = (id(weights), tuple(ids))
        if k not in _rounding:
            _rounding[k] = (weights, rounding_alone(cfg, weights, ids))      # the weights are held so that their id stays theirs
        out[rid] = max(base, 3 * _rounding[k][1])
    return out


def random_config(seed: int) -> dict:
    """A configuration whose every size is drawn: widths, the number and order of layers, the loop, head counts and
    groupings, sizes that are no multiples of 4 or 8, values larger and smaller than keys, windows from one token to longer
    than the sequences, caps or none, scaled frequencies or not, dense and expert layers, layers without feed-forward."""
    rng = random.Random(seed)
    width = rng.choice([24, 36, 42, 64, 72, 100, 128, 200])
    layers = []
    for _ in range(rng.randint(1, 4)):
        kv = rng.choice([1, 2, 3])
        dim = rng.choice([4, 8, 10, 16, 24, 64, 88, 130])
        bands = rng.choice([None, (rng.choice([1.5, 4.0, 16.0]), rng.choice([0.5, 1.0]), rng.choice([2.0, 4.0]), rng.choice([16, 64, 300]))])
        rot = rng.choice([None, _rot(rng.choice([2, dim // 2 * 2, max(dim // 4 * 2, 2)]), rng.choice([100.0, 10000.0, 1e6]), bands)])
        ff = rng.choice([24, 60, 64, 128])
        experts = rng.choice([1, 2, 3, 8, 20])
        mlp = rng.choice([None, _dense(rng.choice([24, 64, 100, 192])), _moe(experts, rng.randint(1, min(experts, 4)), ff, rng.choice([None, 16, 36, 64])),
                          _moe(experts, 1, ff, rng.choice([None, 48]))])
        layers.append(_layer(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([4, 8, 12, 20, 32, 72, 96]), rng.choice([0.1, 0.2, 0.3]),
                             rng.choice([0.0, 3.0, 20.0]), rng.choice([0, 1, 2, 7, 16, 33, 64, 150, 500]), rot, mlp))
    start = rng.randint(0, len(layers))
    stop = rng.randint(start, len(layers))
    loop = rng.choice([None, (start, stop, rng.randint(1, 3))]) if start < stop else None
    return _config(rng.choice([64, 97, 300]), width, rng.choice([1e-5, 1e-6]), rng.choice([0.0, 5.0, 30.0]), loop, layers)
