"""Tiny Kifezen configurations with weights made here, model folders of them, and the comparison of what the engine
returns with the plain implementation (plain_kifezen.py)."""
from __future__ import annotations

import json
import random

import torch

from plain_kifezen import PlainKifezen


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def _rot(dims, base, yarn=None):
    r = {"dims": dims, "base": base}
    if yarn is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return r


def _unit(heads, kv_heads, dim, vdim, scale, temp, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, rot, mlp):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot is not None:
        m["rot"] = rot
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _config(vocab, width, streams, eps, layers):
    return {"architecture": "Kifezen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}


# A: sizes that are no multiples of 8 (the bfloat16 engine falls back to its plain products and attention), three streams,
#    values smaller and larger than keys, a layer without feed-forward, temperatures that change every few tokens.
# B: everything that can be 1 is 1: one stream, one head each, one expert of which one is used, a temperature that changes
#    with every token, a rotated part of one pair, no scaling.
# C: sizes at which the bfloat16 engine takes its tensor-core kernels: a latent of 512 entries with 64 rotated ones, one of 192
#    and one of 64, heads of 128 and 64, experts whose runs of tokens are long enough for the tensor-memory product beside ones whose
#    runs are short.
# D: five streams and a row that is no multiple of 4 (the kernel for any sizes), more heads than a tile has rows, no rotation at
#    all in one layer, sizes inside the kernels' padding.
CONFIGS = {
    "A": _config(203, 70, 3, 1e-5, [
        _latent(3, 10, 6, 14, 20, 0.3, _rot(6, 1000.0, (4.0, 64, 16.0, 1.0)), _moe(5, 2, 28)),
        _unit(6, 3, 12, 20, 0.35, (0.4, 7), _dense(100)),
        _latent(4, 18, 10, 8, 12, 0.25, _rot(10, 500.0), None),
        _unit(4, 1, 22, 12, 0.3, None, _moe(3, 3, 44))]),
    "B": _config(101, 44, 1, 1e-6, [
        _latent(1, 16, 2, 16, 16, 0.3, _rot(2, 100.0), _moe(1, 1, 32)),
        _unit(1, 1, 16, 16, 0.25, (0.5, 1), _dense(64))]),
    "C": _config(333, 384, 4, 1e-5, [
        _latent(8, 128, 64, 128, 512, 0.07, _rot(64, 10000.0, (8.0, 128, 32.0, 1.0)), _dense(512)),
        _unit(8, 2, 128, 128, 0.09, (0.2, 50), _moe(2, 2, 64)),
        _latent(24, 64, 32, 64, 192, 0.1, _rot(32, 50000.0, (16.0, 64, 8.0, 1.0)), _moe(16, 4, 64)),
        _latent(4, 32, 16, 64, 64, 0.15, _rot(16, 1000.0), _moe(12, 1, 72)),
        _unit(4, 4, 64, 128, 0.125, (0.3, 33), None)]),
    "D": _config(150, 266, 5, 1e-6, [
        _latent(96, 8, 8, 8, 40, 0.3, _rot(8, 10000.0, (2.0, 32, 4.0, 0.5)), _dense(128)),
        _latent(2, 40, 24, 104, 88, 0.15, None, _moe(6, 3, 40)),
        _unit(6, 2, 72, 40, 0.11, (0.1, 200), _dense(96))]),
}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 32}


def sharpened(cfg: dict, factor: float) -> dict:
    """The same design with steeper scores, so that a few keys carry a query's whole weight and one that is lost or misplaced
    changes the output by its full size."""
    cfg = json.loads(json.dumps(cfg))
    for layer in cfg["layers"]:
        layer["mixer"]["scale"] *= factor
    return cfg


def make_weights(cfg: dict, seed: int, decisive: bool = True) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16 as a checkpoint holds them.  `decisive`: no choice of experts is a near-tie, which
    16-bit rounding could turn into another choice: the first few entries of a token's embedding hold its class (id modulo
    their number) as one large entry, no sublayer writes there, and the routers read only there, with well spaced weights."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    rnd = lambda *shape, std=1.0: torch.randn(*shape, generator=g) * std
    lin = lambda o, i, gain=1.0: rnd(o, i, std=gain / i ** 0.5)
    w = {"embed": rnd(V, W), "head": lin(V, W, 3.0), "final.norm": rnd(W, std=0.2)}

    def connection(p):
        w[p + ".in"], w[p + ".out"] = 1.0 / S + rnd(S, std=0.3), 0.7 + rnd(S, std=0.3)
        w[p + ".mix"] = 0.8 * torch.eye(S) + rnd(S, S, std=0.25)

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, D, Vd = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = rnd(W, std=0.2)
        connection(p + "hc1")
        q = p + "mix."
        if layer["type"] == "attention":
            G = m["kv_heads"]
            w[q + "q"], w[q + "k"], w[q + "v"] = lin(H * D, W), lin(G * D, W), lin(G * Vd, W)
        else:
            R, L = m["rot_dim"], m["kv_rank"]
            w[q + "q"], w[q + "dkv"], w[q + "dkv.norm"] = lin(H * (D + R), W), lin(L + R, W), 1 + rnd(L, std=0.2)
            w[q + "uk"], w[q + "uv"], w[q + "sink"] = lin(H * D, L), lin(H * Vd, L), rnd(H)
        w[q + "g"], w[q + "o"] = lin(H, W, 1.5), lin(W, H * Vd)
        f = layer["mlp"]
        if f is None:
            continue
        w[p + "norm2"] = rnd(W, std=0.2)
        connection(p + "hc2")
        q = p + "mlp."
        if f["kind"] == "dense":
            w[q + "gate"], w[q + "up"], w[q + "down"] = lin(f["ff"], W, 1.5), lin(f["ff"], W), lin(W, f["ff"])
            continue
        E, ff = f["router"]["experts"], f["expert"]["ff"]
        w[q + "router"] = lin(E, W, 2.0)
        for j in range(E):
            w[q + f"e{j}.gate"], w[q + f"e{j}.up"], w[q + f"e{j}.down"] = lin(ff, W, 1.5), lin(ff, W), lin(W, ff)
    if decisive:
        K = min(8, W // 4)
        w["embed"][:, :K] = 4.0 * torch.nn.functional.one_hot(torch.arange(V) % K, K)
        for k, v in w.items():
            if k.endswith(".router"):
                v[:] = 0.0
                for c in range(K):
                    v[:, c] = 0.5 * torch.randperm(v.shape[0], generator=g)
            elif k.endswith((".mix.o", ".down")):
                v[:K] = 0.0
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


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
        _plain[k] = PlainKifezen(cfg, weights).forward(ids)
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
    holds: plain_kifezen.ROUND) and nothing else."""
    import plain_kifezen as plain
    exact = PlainKifezen(cfg, weights).forward(ids)
    try:
        plain.ROUND = lambda x: x.to(torch.bfloat16).to(torch.float64)
        rounded = PlainKifezen(cfg, weights).forward(ids)
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
    """A configuration whose every size is drawn: widths, streams, the number and order of layers, head counts and groupings,
    sizes that are no multiples of 4 or 8, latents smaller and larger than heads, scaled frequencies, plain ones and no
    rotation, temperatures or none, dense and expert layers, layers without feed-forward."""
    rng = random.Random(seed)
    width = rng.choice([24, 36, 42, 64, 72, 100, 128, 200])
    layers = []
    for _ in range(rng.randint(1, 4)):
        experts = rng.choice([1, 2, 3, 8, 20])
        mlp = rng.choice([None, _dense(rng.choice([24, 64, 100, 192])), _moe(experts, rng.randint(1, min(experts, 4)), rng.choice([24, 60, 64, 128])),
                          _moe(experts, 1, rng.choice([32, 64]))])
        scale = rng.choice([0.1, 0.2, 0.3])
        if rng.random() < 0.4:
            kv = rng.choice([1, 2, 3])
            temp = rng.choice([None, (rng.choice([0.1, 0.5]), rng.choice([1, 2, 16, 50, 1000]))])
            layers.append(_unit(kv * rng.choice([1, 2, 4]), kv, rng.choice([4, 8, 10, 16, 24, 64, 88, 130]), rng.choice([4, 8, 12, 20, 32, 72, 96]), scale, temp, mlp))
            continue
        rot_dim = rng.choice([2, 4, 8, 16, 30, 64])
        yarn = rng.choice([None, (rng.choice([1.5, 4.0, 40.0]), rng.choice([16, 64, 300]), rng.choice([8.0, 32.0]), rng.choice([0.5, 1.0]))])
        rot = rng.choice([None, _rot(rot_dim, rng.choice([100.0, 10000.0, 1e6]), yarn), _rot(rot_dim, 10000.0, yarn)])
        layers.append(_latent(rng.choice([1, 2, 3, 8, 20, 70]), rng.choice([4, 8, 10, 32, 64]), rot_dim, rng.choice([4, 8, 12, 40, 64]),
                              rng.choice([8, 10, 24, 64, 136, 264, 520]), scale, rot, mlp))
    return _config(rng.choice([64, 97, 300]), width, rng.choice([1, 2, 3, 4, 6]), rng.choice([1e-5, 1e-6]), layers)
