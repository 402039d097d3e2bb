"""The plain Kifezen implementation against hand-made values and against itself (whole, portions, token by token), the
configuration reader, and what the host plans for a step of latent attention (CPU)."""
import json
import math

import numpy as np
import pytest
import torch

import kifezen_util as kz
import plain_kifezen as plain

F = torch.float64


def test_streams_by_hand():
    """Two streams of one entry: the mix is indexed from, to; the sublayer reads with one set of numbers and writes with another."""
    X = torch.tensor([[[2.0], [3.0]]], dtype=F)
    assert plain.streams_in(X, torch.tensor([10.0, 1.0], dtype=F)).item() == 23.0
    M = torch.tensor([[1.0, 2.0], [0.0, 5.0]], dtype=F)                         # from 0 to 0, from 0 to 1; from 1 to 0, from 1 to 1
    new = plain.streams_out(X, torch.tensor([[7.0]], dtype=F), M, torch.tensor([0.0, 1.0], dtype=F))
    assert new[0, 0, 0].item() == 2.0 and new[0, 1, 0].item() == 2 * 2.0 + 5 * 3.0 + 7.0


def test_norm_weights_are_stored_around_zero():
    x = torch.tensor([[3.0, -3.0]], dtype=F)
    assert torch.allclose(plain.norm_around_zero(x, torch.tensor([0.0, 1.0], dtype=F), 0.0), torch.tensor([[1.0, -2.0]], dtype=F))
    from lucciola_b200.parts.base import Runtime
    from lucciola_b200.parts.norm import RMSNorm
    norm = RMSNorm(Runtime("cpu", torch.float32), "n", 2, 1e-6, around_zero=True)
    norm.bind(lambda name: torch.tensor([0.0, 1.0], dtype=torch.bfloat16))
    assert norm.weight.tolist() == [1.0, 2.0]


def test_temperature_by_hand():
    """It steps where p + 1 is a multiple of `every`."""
    f = plain.query_temperature(torch.tensor([0, 2, 3, 6, 7, 8, 11]), {"coef": 0.5, "every": 4})
    want = [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(4)]
    assert torch.allclose(f, torch.tensor(want, dtype=F))
    assert plain.query_temperature(torch.tensor([5]), None).tolist() == [1.0]


def test_scaled_rotation_by_hand():
    """Fast pairs keep their frequency, slow ones are divided, one in between is blended; sines and cosines carry the factor."""
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    f, mag = plain.rotary_frequencies(rot)
    place = lambda t: 8 * math.log(64 / (2 * math.pi * t)) / (2 * math.log(100.0))
    lo, hi = max(math.floor(place(8.0)), 0), min(math.ceil(place(1.0)), 7)
    assert (lo, hi) == (0, 3)
    for i in range(4):
        raw, ramp = 100.0 ** (-2 * i / 8), min(max(i / 3, 0.0), 1.0)
        assert math.isclose(f[i].item(), raw / 4 * ramp + raw * (1 - ramp), rel_tol=1e-12)
    assert math.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    x = torch.zeros(1, 1, 8, dtype=F)
    x[0, 0, 1], x[0, 0, 5] = 1.0, 2.0                                          # entries 1 and 5 are a pair
    y = plain.rotate_halves(x, torch.tensor([3]), rot)[0, 0]
    c, s = math.cos(3 * f[1].item()) * mag, math.sin(3 * f[1].item()) * mag
    assert math.isclose(y[1].item(), c - 2 * s, rel_tol=1e-12) and math.isclose(y[5].item(), 2 * c + s, rel_tol=1e-12)
    from lucciola_b200.parts.base import Runtime
    from lucciola_b200.parts.rope import RotaryEmbedding
    enc = RotaryEmbedding(Runtime("cpu", torch.float32), 8, 100.0, 8, yarn=(4.0, 64, 8.0, 1.0))
    assert torch.equal(enc.inv_freq, f.to(torch.float32)) and math.isclose(enc.magnitude, mag)


def test_a_sink_takes_weight_and_gives_nothing():
    """Scale 0: every visible key and the sink of 0 count alike; a sink of ln 3 counts as three keys."""
    v = torch.tensor([[[1.0]], [[5.0]]], dtype=F)
    k = q = torch.zeros(2, 1, 1, dtype=F)
    out = plain.causal_softmax_attention(q, k, v, 0, 0.0, torch.zeros(1, dtype=F))
    assert torch.allclose(out.flatten(), torch.tensor([0.5, 2.0], dtype=F))
    out = plain.causal_softmax_attention(q, k, v, 0, 0.0, torch.full((1,), math.log(3.0), dtype=F))
    assert torch.allclose(out.flatten(), torch.tensor([0.25, 1.2], dtype=F))


def test_experts_by_hand():
    """The two largest logits choose; their softmax alone weighs."""
    one = torch.ones(1, 1, dtype=F)
    w = {"router": torch.tensor([[0.0], [1.0], [2.0]], dtype=F)}
    for j in range(3):
        w[f"e{j}.gate"], w[f"e{j}.up"], w[f"e{j}.down"] = one, one, one * 10 ** j
    out = plain.routed_feed_forward(torch.tensor([[1.0]], dtype=F), w, {"router": {"experts": 3, "top": 2}})
    g = plain.silu(torch.tensor(1.0, dtype=F)).item()
    a = 1 / (1 + math.exp(-1.0))
    assert math.isclose(out.item(), g * (a * 100 + (1 - a) * 10), rel_tol=1e-12)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_and_single_tokens_equal_the_whole(name):
    cfg = kz.CONFIGS[name]
    w = kz.make_weights(cfg, 11)
    ids = kz.tokens(cfg, 50, salt=3)
    model = plain.PlainKifezen(cfg, w)
    whole = model.forward(ids)
    past, got, at = None, [], 0
    for n in (1, 7, 2, 1, 1, 19, 3, 16):
        logits, past = model.run(ids[at:at + n], past)
        got.append(logits)
        at += n
    assert at == 50
    assert (torch.cat(got) - whole).abs().max() <= 1e-9 * whole.abs().max()


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_configuration_reader_and_tensor_list(name):
    """config.json -> typed configuration -> config.json again; the model the registry composes asks for exactly the
    tensors a checkpoint of this design has, in their shapes."""
    from lucciola_b200.config.registry import resolve_architecture
    from lucciola_b200.parts.base import Runtime
    cfg = kz.CONFIGS[name]
    arch = resolve_architecture(cfg)
    typed = arch.config_from_dict(cfg)
    assert typed.to_dict() == json.loads(json.dumps(cfg))
    w = kz.make_weights(cfg, 5)
    model = arch.build(typed, Runtime("cpu", torch.float32))
    assert {s.name: tuple(s.shape) for s in model.all_param_specs()} == {k: tuple(v.shape) for k, v in w.items()}
    assert len(model.calls) == len(cfg["layers"])


def test_tensors_of_a_feed_forward_that_is_not_there_are_no_fault():
    from lucciola_b200.config.registry import resolve_architecture
    from lucciola_b200.parts.base import Runtime
    cfg = kz.CONFIGS["A"]
    arch = resolve_architecture(cfg)
    ignored = arch.build(arch.config_from_dict(cfg), Runtime("cpu", torch.float32)).ignored_names()
    assert {"l2.norm2", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"} <= set(ignored) and "l1.norm2" not in ignored


def test_configurations_that_are_refused():
    from lucciola_b200.config.kifezen_config import KifezenConfig
    from lucciola_b200.config.model_config import ConfigError

    def broken(change):
        d = json.loads(json.dumps(kz.CONFIGS["A"]))
        change(d)
        with pytest.raises(ConfigError):
            KifezenConfig.from_dict(d)
    broken(lambda d: d["layers"][0].update(type="hyena"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="gelu"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=5))
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"))
    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=0))
    broken(lambda d: d.update(streams=0))
    broken(lambda d: d["layers"][0]["mixer"].pop("kv_rank"))
    broken(lambda d: d.pop("norm"))


def test_a_block_of_several_streams_stands_among_its_own_kind():
    """A block that knows one stream cannot follow one that keeps several: said, not mixed up."""
    from lucciola_b200 import ops
    from lucciola_b200.models.decoder import DecoderModel
    from lucciola_b200.parts.base import StreamUpdate
    with pytest.raises(ops.KernelError):
        DecoderModel._settle(None, torch.zeros(1, 2, 4), StreamUpdate(torch.zeros(1, 4), None))


def latent_part(heads=4, dim=128, rot=64, vdim=128, rank=512):
    from lucciola_b200.parts.base import Runtime
    from lucciola_b200.parts.latent_attention import RotaryLatentAttention
    return RotaryLatentAttention(Runtime("cpu", torch.bfloat16), "m", 64, heads, dim, rot, vdim, rank, 0.1, None, 1e-5)


def test_the_plan_of_latent_attention_covers_every_token_once():
    """Portions worth multiplying out, short ones and single tokens in one step: every token stands in exactly one tile, tiles
    carry how far into their request's tokens they start, rows of the portions lie one behind the other."""
    from lucciola_b200.parts.base import BatchShape
    part = latent_part(heads=16)
    for q_lens, starts in (([1, 700, 3, 1, 300], [900, 0, 64, 5, 128]), ([2, 15, 9], [0, 7, 100]), ([600], [0]), ([1, 1], [3, 80])):
        shape = BatchShape(list(q_lens), list(starts), max(q_lens), max(s + n for s, n in zip(starts, q_lens)), 1024)
        plan = part.plan(shape)
        first = np.concatenate(([0], np.cumsum(q_lens)))
        seen = []
        for t0, n, i, off in plan.arrays.get("rest", np.zeros((0, 4), int)).tolist():
            assert t0 == first[i] + off and n * part.group <= plan.host["tile_rows"] <= 64
            assert plan.host["lo"] <= t0 and t0 + n <= plan.host["hi"]
            seen += range(t0, t0 + n)
        rows = {i: (at, k) for i, at, k, _ in plan.arrays.get("entries", np.zeros((0, 4), int)).tolist()}
        for t0, n, i, at in plan.arrays.get("big", np.zeros((0, 4), int)).tolist():
            assert n <= 256 and rows[i] == (at, starts[i] + q_lens[i])
            seen += range(t0, t0 + n)
        assert sorted(seen) == list(range(sum(q_lens)))
        ends = sorted(rows.values())
        assert all(a + k == b for (a, k), (b, _) in zip(ends, ends[1:])) and sum(k for _, k in ends) == plan.host["rows"]
        assert ("big" in plan.arrays) == any(n >= 16 for n in q_lens)
    # a recorded step plans by the bound on the context, whatever the requests' places are
    a, b = (part.plan(BatchShape([600], [s], 600, s + 600, 1024, True)) for s in (0, 300))
    assert a.host == b.host and {k: v.shape for k, v in a.arrays.items()} == {k: v.shape for k, v in b.arrays.items()} and a.host["rows"] == 1024


def test_tiles_say_how_far_into_their_request_they_start():
    from lucciola_b200.parts.attention import tiles_of
    assert tiles_of([5, 1, 4], 8, 16) == [(0, 2, 0, 0), (2, 2, 0, 2), (4, 1, 0, 4), (5, 1, 1, 0), (6, 2, 2, 0), (8, 2, 2, 2)]


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random_build(seed):
    from lucciola_b200.config.registry import resolve_architecture
    from lucciola_b200.parts.base import Runtime
    cfg = kz.random_config(seed)
    arch = resolve_architecture(cfg)
    model = arch.build(arch.config_from_dict(cfg), Runtime("cpu", torch.float32))
    w = kz.make_weights(cfg, seed)
    assert {s.name: tuple(s.shape) for s in model.all_param_specs()} == {k: tuple(v.shape) for k, v in w.items()}
    ids = kz.tokens(cfg, 12, salt=seed)
    assert torch.isfinite(plain.PlainKifezen(cfg, w).forward(ids)).all()
