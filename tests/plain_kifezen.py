"""The Kifezen decoder, plainly: one slow function per mechanism, on the CPU, in float64 unless told otherwise.

This file is what the engine's kernels are compared with.  It shares no code with the package: it takes a
configuration as the dictionary of config.json and the weights as a dictionary of tensors by checkpoint name,
and runs one sequence at a time, either whole or in portions with an explicit past.

Notation.  X: the streams [T, s, width], all equal to embed[token] at the start.  A sublayer f (a layer's mixer, then its
feed-forward) with the numbers a (in), b (out) and M (mix, from row to column) computes y = f(n(sum_s a_s X_s)) and then
X_t <- sum_s M[s, t] X_s + b_t y.  n is an RMS norm times 1 + w.  Linear weights are [out, in].
"""
from __future__ import annotations

import math

import torch


# Where an engine that serves in 16 bits may round: the inputs of products and what a cache holds.  None: nowhere (this
# file's own arithmetic is exact to its type); the tests set it to see what such rounding alone does to a model's logits.
ROUND = None


def _r(x: torch.Tensor) -> torch.Tensor:
    return x if ROUND is None else ROUND(x)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def norm_around_zero(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + weight)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def streams_in(X: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """What a sublayer reads: the streams [T, s, width] added with the weights a."""
    return (X * a[None, :, None]).sum(dim=1)


def streams_out(X: torch.Tensor, y: torch.Tensor, M: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """The streams after a sublayer: new stream t is the sum of the old ones with column t of M, plus b_t y."""
    s = X.shape[1]
    new = [sum(M[r, t] * X[:, r] for r in range(s)) + b[t] * y for t in range(s)]
    return torch.stack(new, dim=1)


def query_temperature(positions: torch.Tensor, temp) -> torch.Tensor:
    """The factor of the query at each position, 1 + coef ln(floor((p + 1) / every) + 1); 1 without the option."""
    if temp is None:
        return torch.ones(positions.shape[0], dtype=torch.float64)
    return torch.tensor([1.0 + temp["coef"] * math.log((int(p) + 1) // temp["every"] + 1) for p in positions], dtype=torch.float64)


def rotary_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(the dims / 2 frequencies, the factor on sine and cosine): base^(-2i/dims), with `scaling` (YaRN) those of pairs that
    make few turns within `original` positions divided by `factor`, with a linear ramp in between."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return torch.tensor(f, dtype=torch.float64), 1.0
    place = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(sc["fast"])), 0), min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * ramp + x * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot) -> torch.Tensor:
    """x [T, heads, n]: entries i and i + dims/2 are a pair, turned by position * f_i; entries from dims on pass."""
    if rot is None or rot["dims"] == 0:
        return x
    f, mag = rotary_frequencies(rot)
    a = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = (torch.cos(a) * mag)[:, None, :].to(x.dtype), (torch.sin(a) * mag)[:, None, :].to(x.dtype)
    h = rot["dims"] // 2
    u, v = x[..., :h], x[..., h:2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], dim=-1)


def causal_softmax_attention(q, k, v, start: int, scale: float, sinks=None):
    """q [T, H, D] at positions start .. over keys k [n, G, D] and values v [n, G, V] at positions 0 .. n - 1; with `sinks`
    [H] the denominator of head h also holds exp(sinks[h])."""
    T, H, D = q.shape
    G, V = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, V, dtype=q.dtype)
    for t in range(T):
        n = start + t + 1
        s = q[t].reshape(G, H // G, D) @ k[:n].permute(1, 2, 0) * scale                          # [G, H / G, n]
        if sinks is not None:
            s = torch.cat([s, sinks.to(s.dtype).reshape(G, H // G, 1)], dim=-1)
        out[t] = (torch.softmax(s, dim=-1)[..., :n] @ v[:n].permute(1, 0, 2)).reshape(H, V)
    return out


def head_gated(out: torch.Tensor, h: torch.Tensor, wg: torch.Tensor) -> torch.Tensor:
    """Head outputs [T, H, V] times one sigmoid a head."""
    return out * torch.sigmoid(h @ wg.T)[:, :, None]


def attention(h: torch.Tensor, w: dict, m: dict, eps: float, past):
    """w: q, k, v, g, o.  Unit queries and keys, queries times their temperature, causal softmax, a gate a head.
    past: (keys as the cache holds them [n, G, D], values [n, G, V]) or None."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    start = 0 if past is None else past[0].shape[0]
    h = _r(h)
    temp = query_temperature(torch.arange(start, start + T), m.get("q_temp")).to(h.dtype)
    q = rms((h @ w["q"].T).reshape(T, H, D), eps) * temp[:, None, None]
    k = rms((h @ w["k"].T).reshape(T, G, D), eps)
    v = (h @ w["v"].T).reshape(T, G, V)
    q, k, v = _r(q), _r(k), _r(v)
    if past is not None:
        k, v = torch.cat([past[0], k], dim=0), torch.cat([past[1], v], dim=0)
    out = head_gated(_r(causal_softmax_attention(q, k, v, start, m["scale"])), h, w["g"])
    return _r(out.reshape(T, H * V)) @ w["o"].T, (k, v)


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float, past):
    """w: q, dkv, dkv.norm, uk, uv, sink, g, o.  Every head's key is (W_uk c, one rotated part all heads share), its value
    W_uv c with the normed latent c.  past: (latents [n, rank], rotated key parts [n, R]) or None."""
    H, D, R, V, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    start = 0 if past is None else past[0].shape[0]
    pos = torch.arange(start, start + T)
    h = _r(h)
    q = (h @ w["q"].T).reshape(T, H, D + R)
    q_rot = rotate_halves(q[..., D:], pos, m.get("rot"))
    down = h @ w["dkv"].T
    c = _r(rms(down[:, :L], eps) * w["dkv.norm"])
    k_rot = _r(rotate_halves(down[:, None, L:], pos, m.get("rot"))[:, 0])
    if past is not None:
        c, k_rot = torch.cat([past[0], c], dim=0), torch.cat([past[1], k_rot], dim=0)
    n = c.shape[0]
    k = torch.cat([_r((c @ w["uk"].T).reshape(n, H, D)), k_rot[:, None, :].expand(n, H, R)], dim=-1)
    v = _r((c @ w["uv"].T).reshape(n, H, V))
    q = _r(torch.cat([q[..., :D], q_rot], dim=-1))
    out = head_gated(_r(causal_softmax_attention(q, k, v, start, m["scale"], w["sink"])), h, w["g"])
    return _r(out.reshape(T, H * V)) @ w["o"].T, (c, k_rot)


def gated_feed_forward(h: torch.Tensor, w: dict) -> torch.Tensor:
    """down( silu(gate h) * (up h) ); w: gate, up, down."""
    h = _r(h)
    return _r(silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def routed_feed_forward(h: torch.Tensor, w: dict, mlp: dict) -> torch.Tensor:
    """The `top` experts with the largest router logits, weighted by the softmax over those logits alone."""
    top = mlp["router"]["top"]
    out = torch.zeros_like(h)
    z = _r(h) @ w["router"].T
    for t in range(h.shape[0]):
        chosen = sorted(range(z.shape[1]), key=lambda e: -z[t, e].item())[:top]
        weights = torch.softmax(z[t, chosen], dim=-1)
        for e, x in zip(chosen, weights):
            out[t] += x * gated_feed_forward(h[t:t + 1], {n: w[f"e{e}.{n}"] for n in ("gate", "up", "down")})[0]
    return out


MIXERS = {"attention": attention, "latent_attention": latent_attention}


class PlainKifezen:
    def __init__(self, cfg: dict, weights: dict, dtype=torch.float64):
        self.cfg = cfg
        self.w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
        self.dtype = dtype

    def _sub(self, prefix: str) -> dict:
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def _sublayer(self, X, p: str, q: int, f):
        eps = self.cfg["norm"]["eps"]
        hc = self._sub(f"{p}hc{q}.")
        y = f(norm_around_zero(streams_in(X, hc["in"]), self.w[f"{p}norm{q}"], eps))
        return streams_out(X, y, hc["mix"], hc["out"])

    def run(self, ids, past=None, layers_out: list | None = None):
        """Logits [T, vocab] of the tokens `ids`, which follow what `past` holds (None: a sequence's start), and the
        new past (one entry a layer).  layers_out, if a list, receives the sum of the streams after every layer."""
        eps = self.cfg["norm"]["eps"]
        x = self.w["embed"][torch.as_tensor(ids, dtype=torch.long)]
        X = x[:, None, :].repeat(1, self.cfg["streams"], 1)
        past = past if past is not None else [None] * len(self.cfg["layers"])
        new_past = []
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."

            def mixer(h):
                y, state = MIXERS[layer["type"]](h, self._sub(p + "mix."), layer["mixer"], eps, past[i])
                new_past.append(state)
                return y

            X = self._sublayer(X, p, 1, mixer)
            mlp = layer.get("mlp")
            if mlp is not None:
                w = self._sub(p + "mlp.")
                X = self._sublayer(X, p, 2, lambda h: gated_feed_forward(h, w) if mlp["kind"] == "dense" else routed_feed_forward(h, w, mlp))
            if layers_out is not None:
                layers_out.append(X.sum(dim=1))
        h = norm_around_zero(X.sum(dim=1), self.w["final.norm"], eps)
        return _r(h) @ self.w["head"].T, new_past

    def forward(self, ids, layers_out: list | None = None) -> torch.Tensor:
        return self.run(ids, None, layers_out)[0]
