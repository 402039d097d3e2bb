"""The Nulalorn decoder, plainly: one slow function per mechanism, on the CPU, in float64 unless told otherwise.

This file is what the engine's kernels are compared with.  It shares no code with the package: it takes a
configuration as the dictionary of config.json and the weights as a dictionary of tensors by checkpoint name,
and runs one sequence at a time, either whole or in portions with an explicit past.

Notation.  x: residual stream [T, width].  A layer computes x <- x + n1b(mixer(n1(x))) and then, if it has a feed-forward,
x <- x + n2b(ff(n2(x))): a norm in front of and a norm behind every sublayer.  Linear weights are [out, in].  Layers
`loop.start .. loop.stop - 1` run `loop.times` times in a row with the same weights and a past of their own for every
pass; in front of pass t the stream becomes W_in [x ; x0] + step[t] with x0 the embedding's output.
"""
from __future__ import annotations

import math

import torch


# Where an engine that serves in 16 bits may round: the inputs of products and what a cache holds.  None: nowhere (this
# file's own arithmetic is exact to its type); the tests set it to see what such rounding alone does to a model's logits.
ROUND = None


def _r(x: torch.Tensor) -> torch.Tensor:
    return x if ROUND is None else ROUND(x)


def rms_norm(x: torch.Tensor, weight, eps: float) -> torch.Tensor:
    y = x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def gelu(z: torch.Tensor) -> torch.Tensor:
    """z times the standard normal distribution function at z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def cap(z: torch.Tensor, c) -> torch.Tensor:
    return z if not c else c * torch.tanh(z / c)


def rotary_frequencies(rot: dict) -> torch.Tensor:
    """The dims / 2 frequencies base^(-2i/dims); with `scaling`, those whose wavelength is longer than original / low are
    divided by `factor`, those shorter than original / high are kept, and in between the two are blended linearly in
    original / wavelength."""
    dims = rot["dims"]
    out = []
    for i in range(dims // 2):
        f = rot["base"] ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc is not None:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot) -> torch.Tensor:
    """x [T, heads, dim]: entries 2i and 2i + 1 are a pair, turned by position * f_i; entries from dims on pass."""
    if rot is None or rot["dims"] == 0:
        return x
    a = positions.to(torch.float64)[:, None] * rotary_frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :].to(x.dtype), torch.sin(a)[:, None, :].to(x.dtype)
    y = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    y[..., 0:rot["dims"]:2] = u * c - v * s
    y[..., 1:rot["dims"]:2] = v * c + u * s
    return y


def capped_attention(q, k, v, start: int, scale: float, softcap, window: int):
    """q [T, H, D] at positions start .. start + T - 1 over keys k [n, G, D] and values v [n, G, V] at positions 0 ..
    n - 1.  Position i sees itself and the window - 1 tokens before it (window 0: everything before it)."""
    T, H, _ = q.shape
    G, V = k.shape[1], v.shape[2]
    per = H // G
    out = torch.zeros(T, H, V, dtype=q.dtype)
    for t in range(T):
        i = start + t
        lo = max(0, i - window + 1) if window else 0
        for g in range(G):
            s = cap((q[t, g * per:(g + 1) * per] @ k[lo:i + 1, g].T) * scale, softcap)
            out[t, g * per:(g + 1) * per] = torch.softmax(s, dim=-1) @ v[lo:i + 1, g]
    return out


def attention(h: torch.Tensor, w: dict, m: dict, eps: float, past):
    """w: q, k, v, o.  Rotation, then q and k of every head divided by their root mean square, then attention with a
    capped score over a sliding window.  past: (keys as the cache holds them [n, G, D], values [n, G, V]) or None."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    start = 0 if past is None else past[0].shape[0]
    pos = torch.arange(start, start + T)
    h = _r(h)
    q = rms_norm(rotate_neighbours((h @ w["q"].T).reshape(T, H, D), pos, m.get("rot")), None, eps)
    k = rms_norm(rotate_neighbours((h @ w["k"].T).reshape(T, G, D), pos, m.get("rot")), None, eps)
    v = (h @ w["v"].T).reshape(T, G, V)
    q, k, v = _r(q), _r(k), _r(v)
    if past is not None:
        k, v = torch.cat([past[0], k], dim=0), torch.cat([past[1], v], dim=0)
    window = (m.get("mask") or {"size": 0})["size"]
    out = capped_attention(q, k, v, start, m["scale"], m.get("softcap"), window)
    return _r(out.reshape(T, H * V)) @ w["o"].T, (k, v)


def dense_feed_forward(h: torch.Tensor, w: dict) -> torch.Tensor:
    """down( gelu(up h) ); w: up, down."""
    return _r(gelu(_r(h) @ w["up"].T)) @ w["down"].T


def expert_feed_forward(h: torch.Tensor, ids, w: dict, mlp: dict) -> torch.Tensor:
    """Each token's experts stand in the table's row of the token's id and count 1 / top each; with `shared`, one more
    feed-forward of every token, times the sigmoid of one number a token.  w: table, e<j>.up, e<j>.down, shared.*."""
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=h.dtype)
    top = mlp["router"]["top"]
    for t, token in enumerate(ids):
        row = w["table"][int(token)].tolist()
        assert len(row) == top
        for e in row:
            one = {"up": w[f"e{e}.up"], "down": w[f"e{e}.down"]}
            out[t] = out[t] + dense_feed_forward(h[t:t + 1], one)[0] / top
    if mlp.get("shared") is not None:
        gate = torch.sigmoid(_r(h) @ w["shared.sg"].T)                                           # [T, 1]
        out = out + gate * dense_feed_forward(h, {"up": w["shared.up"], "down": w["shared.down"]})
    return out


def layer_runs(cfg: dict) -> list[tuple[int, int]]:
    """The layers in the order they run: (layer, the number of the pass that starts before it, or -1)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, -1) for i in range(a)]
    for p in range(times if b > a else 0):
        runs += [(i, p if i == a else -1) for i in range(a, b)]
    return runs + [(i, -1) for i in range(max(a, b), n)]


class PlainNulalorn:
    def __init__(self, cfg: dict, weights: dict, dtype=torch.float64):
        self.cfg = cfg
        self.w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
        self.dtype = dtype
        self.runs = layer_runs(cfg)

    def _sub(self, prefix: str) -> dict:
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def run(self, ids, past=None, layers_out: list | None = None):
        """Logits [T, vocab] of the tokens `ids`, which follow what `past` holds (None: a sequence's start), and the
        new past (one entry for every layer run).  layers_out, if a list, receives the residual stream after every run."""
        eps = self.cfg["norm"]["eps"]
        x0 = self.w["embed"][torch.as_tensor(ids, dtype=torch.long)]
        x = x0.clone()
        past = past if past is not None else [None] * len(self.runs)
        new_past = []
        for r, (i, starts_pass) in enumerate(self.runs):
            layer, p = self.cfg["layers"][i], f"l{i}."
            if starts_pass >= 0:
                x = torch.cat([x, x0], dim=-1) @ self.w["loop.in"].T + self.w["loop.step"][starts_pass]
            a, state = attention(rms_norm(x, self.w[p + "norm1"], eps), self._sub(p + "mix."), layer["mixer"], eps, past[r])
            new_past.append(state)
            x = x + rms_norm(a, self.w[p + "norm1b"], eps)
            mlp = layer.get("mlp")
            if mlp is not None:
                h = rms_norm(x, self.w[p + "norm2"], eps)
                w = self._sub(p + "mlp.")
                b = dense_feed_forward(h, w) if mlp["kind"] == "dense" else expert_feed_forward(h, ids, w, mlp)
                x = x + rms_norm(b, self.w[p + "norm2b"], eps)
            if layers_out is not None:
                layers_out.append(x.clone())
        logits = _r(rms_norm(x, self.w["final.norm"], eps)) @ self.w["head"].T
        return cap(logits, self.cfg.get("logit_softcap")), new_past

    def forward(self, ids, layers_out: list | None = None) -> torch.Tensor:
        return self.run(ids, None, layers_out)[0]
