"""The plain Nulalorn implementation against hand-made values and against itself (whole, portions, token by token), the
configuration reader, the order of layer runs, and the scaled frequencies (CPU)."""
import json
import math

import pytest
import torch

import nulalorn_util as nz
import plain_nulalorn as plain

F = torch.float64


def test_gelu_by_hand():
    z = torch.tensor([-6.0, -1.0, 0.0, 0.5, 3.0], dtype=F)
    want = [x * 0.5 * math.erfc(-x / math.sqrt(2.0)) for x in z.tolist()]
    assert torch.allclose(plain.gelu(z), torch.tensor(want, dtype=F), atol=1e-12)


def test_rotation_in_pairs_of_neighbours_by_hand():
    """A quarter turn of the first pair, an eighth of that of the second; entries behind dims pass."""
    x = torch.tensor([[[1.0, 0.0, 1.0, 0.0, 7.0]]], dtype=F)
    rot = {"dims": 4, "base": 64.0}                                           # frequencies 1 and 64^(-1/2) = 1/8
    y = plain.rotate_neighbours(x, torch.tensor([3]), rot)[0, 0]
    want = [math.cos(3.0), math.sin(3.0), math.cos(3.0 / 8), math.sin(3.0 / 8), 7.0]
    assert torch.allclose(y, torch.tensor(want, dtype=F))


def test_scaled_frequencies_by_hand():
    """Frequencies whose wavelength stands below, between and above the two borders, each by its rule; the package's table is
    the same numbers rounded once."""
    from lucciola_b200.parts.rope import band_frequencies
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}
    rot = {"dims": 12, "base": 4000.0, "scaling": sc}
    f = plain.rotary_frequencies(rot)
    kinds = set()
    for i, got in enumerate(f.tolist()):
        raw = 4000.0 ** (-2.0 * i / 12)
        wave = 2 * math.pi / raw
        if wave < 25.0:
            want, kind = raw, "kept"
        elif wave > 100.0:
            want, kind = raw / 8.0, "divided"
        else:
            s = (100.0 / wave - 1.0) / 3.0
            want, kind = (1 - s) * raw / 8.0 + s * raw, "blended"
        kinds.add(kind)
        assert math.isclose(got, want, rel_tol=1e-12)
    assert kinds == {"kept", "divided", "blended"}
    raw = 4000.0 ** (-2.0 * torch.arange(6, dtype=F) / 12)
    assert torch.allclose(band_frequencies(raw, 8.0, 1.0, 4.0, 100.0), f, rtol=1e-12)
    from lucciola_b200.parts.base import Runtime
    from lucciola_b200.parts.rope import NeighbourRotary
    table, dims = NeighbourRotary(Runtime("cpu", torch.float32), 16, 4000.0, 12, bands=(8.0, 1.0, 4.0, 100)).pair_table()
    assert dims == 12 and torch.equal(table, f.to(torch.float32))


def test_window_and_cap_by_hand():
    """A scale of zero and a window of 2: the mean of the last two values.  A cap: scores c tanh(s / c)."""
    D = 2
    eye = torch.eye(D, dtype=F)
    w = {"q": eye, "k": eye, "v": eye, "o": eye}
    m = {"heads": 1, "kv_heads": 1, "dim": D, "vdim": D, "scale": 0.0, "softcap": 5.0, "mask": {"size": 2}}
    h = torch.arange(1, 9, dtype=F).reshape(4, 2)
    out, _ = plain.attention(h, w, m, 1e-9, None)
    for i in range(4):
        assert torch.allclose(out[i], h[max(0, i - 1):i + 1].mean(0))
    # unit heads: q . k of a vector with itself is dim whatever its length
    m = dict(m, scale=1.5, mask={"size": 9})
    h = torch.tensor([[3.0, 0.0], [0.0, 0.5]], dtype=F)
    out, _ = plain.attention(h, w, m, 1e-12, None)
    e = math.exp(5.0 * math.tanh(2 * 1.5 / 5.0))
    assert torch.allclose(out[1], (1.0 * h[0] + e * h[1]) / (1.0 + e), atol=1e-9)


def test_experts_by_hand():
    """Identity experts times 1, 2, 3: a token gets the mean factor of the experts its id names, plus the gated shared one."""
    one = torch.ones(1, 1, dtype=F)
    w = {"table": torch.tensor([[0, 2], [1, 0]], dtype=torch.int32), "shared.up": one, "shared.down": one * 10, "shared.sg": one * 0.0}
    for j in range(3):
        w[f"e{j}.up"], w[f"e{j}.down"] = one, one * (j + 1)
    mlp = {"router": {"experts": 3, "top": 2}, "shared": {"ff": 1}}
    h = torch.tensor([[2.0], [2.0]], dtype=F)
    g = plain.gelu(torch.tensor(2.0, dtype=F)).item()
    out = plain.expert_feed_forward(h, [0, 1], w, mlp)
    assert torch.allclose(out, torch.tensor([[g * 2.0 + 0.5 * 10 * g], [g * 1.5 + 0.5 * 10 * g]], dtype=F))


def test_the_order_of_layer_runs():
    cfg = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 3}}
    assert plain.layer_runs(cfg) == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1), (1, 2), (2, -1), (3, -1)]
    assert plain.layer_runs({"layers": [0, 1], "loop": {"start": 2, "stop": 2, "times": 4}}) == [(0, -1), (1, -1)]
    assert plain.layer_runs({"layers": [0, 1], "loop": {"start": 0, "stop": 2, "times": 1}}) == [(0, 0), (1, -1)]
    assert plain.layer_runs({"layers": [0, 1]}) == [(0, -1), (1, -1)]


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions_and_single_tokens_equal_the_whole(name):
    cfg = nz.CONFIGS[name]
    w = nz.make_weights(cfg, 11)
    ids = nz.tokens(cfg, 50, salt=3)
    model = plain.PlainNulalorn(cfg, w)
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
    tensors a checkpoint of this design has, in their shapes, and runs the layers in their order."""
    from lucciola_b200.config.registry import resolve_architecture
    from lucciola_b200.parts.base import Runtime
    cfg = nz.CONFIGS[name]
    arch = resolve_architecture(cfg)
    typed = arch.config_from_dict(cfg)
    assert typed.to_dict() == json.loads(json.dumps(cfg))
    w = nz.make_weights(cfg, 5)
    model = arch.build(typed, Runtime("cpu", torch.float32))
    specs = {s.name: tuple(s.shape) for s in model.all_param_specs()}
    assert specs == {k: tuple(v.shape) for k, v in w.items()}
    runs = plain.layer_runs(cfg)
    assert [(c.block, c.entry) for c in model.calls] == runs and [c.cache for c in model.calls] == list(range(len(runs)))


def test_configurations_that_are_refused():
    from lucciola_b200.config.model_config import ConfigError
    from lucciola_b200.config.nulalorn_config import NulalornConfig
    good = nz.CONFIGS["A"]
    def broken(change):
        d = json.loads(json.dumps(good))
        change(d)
        with pytest.raises(ConfigError):
            NulalornConfig.from_dict(d)
    broken(lambda d: d["layers"][0].update(type="hyena"))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda d: d["loop"].update(stop=9))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][1]["mlp"]["shared"].update(ff=0))
    broken(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=5))
    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=3))
    broken(lambda d: d.pop("norm"))


def test_random_tables_name_distinct_experts():
    from lucciola_b200.parts.base import ParamSpec
    from lucciola_b200.weights.random_init import random_tensor
    t = random_tensor(ParamSpec("t", (200, 3), integer=True, below=5), 1, 0.02, 0.0, torch.bfloat16)
    assert t.dtype == torch.int32 and tuple(t.shape) == (200, 3) and int(t.min()) == 0 and int(t.max()) == 4
    assert all(len(set(row)) == 3 for row in t.tolist())


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random_build(seed):
    from lucciola_b200.config.registry import resolve_architecture
    from lucciola_b200.parts.base import Runtime
    cfg = nz.random_config(seed)
    arch = resolve_architecture(cfg)
    model = arch.build(arch.config_from_dict(cfg), Runtime("cpu", torch.float32))
    w = nz.make_weights(cfg, seed)
    assert {s.name: tuple(s.shape) for s in model.all_param_specs()} == {k: tuple(v.shape) for k, v in w.items()}
    ids = nz.tokens(cfg, 12, salt=seed)
    assert torch.isfinite(plain.PlainNulalorn(cfg, w).forward(ids)).all()
