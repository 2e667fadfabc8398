"""The Tekarax configuration on the CPU: registry, the model's description and tensor names, the size only a tensor gives,
the order in which looped layers run, refused configurations, cache groups and state, and the plain implementation's own
consistency (the recurrence in closed form, the shift, the window, the sink, values that count by their distance)."""
import copy
import math

import pytest
import torch

import plain_tekarax as plain
import tekarax_cases as cases
from torchlet_b200.config import TekaraxConfig, config_from_dict, known_architectures
from torchlet_b200.parts import LayeredModel, expected_tensors


def test_registered_and_chosen_by_name():
    assert "Tekarax" in known_architectures()
    for name in ("P", "Q", "R", "S"):
        config = config_from_dict(cases.CASES[name])
        assert isinstance(config, TekaraxConfig)
        assert TekaraxConfig.from_dict(config.to_dict()) == config


def test_description_and_tensor_names():
    spec = cases.config_for("P").model_spec()
    assert [layer.block for layer in spec.layers] == ["sandwich"] * 5
    assert [layer.mixer.kind for layer in spec.layers] == ["time_mixing", "gated_attention", "latent_attention", "latent_attention", "time_mixing"]
    assert [layer.feed_forward.kind if layer.feed_forward else None for layer in spec.layers] == \
        ["routed_clamped_glu", "mlp", "routed_clamped_glu", None, None]
    assert all(layer.block_params["gates"] == ("rg1", "rg2") for layer in spec.layers)
    attention = spec.layers[1].mixer.params
    assert (attention["sink"], attention["gate"], attention["value_rotation"].params["dims"]) == ("learned", "head_sigmoid", 16)
    assert attention["positions"].params["scaling"]["factor"] == 8.0 and "scaling" not in attention["value_rotation"].params
    routed = spec.layers[0].feed_forward.params
    assert (routed["score"], routed["renormalize"], routed["weight_on"], routed["limit"]) == ("sigmoid", False, "input", None)
    names = {t.name: t.shape for t in expected_tensors(spec)}
    for name, shape in {"embed": (101, 96), "head": (101, 96), "final.norm": (96,), "loop.step": (3, 96), "l0.norm1": (96,),
                        "l0.norm1b": (96,), "l0.norm2": (96,), "l0.norm2b": (96,), "l0.rg1": (96, 96), "l0.rg1.b": (96,),
                        "l0.rg2": (96, 96), "l0.rg2.b": (96,), "l0.mix.mu.r": (96,), "l0.mix.mu.w": (96,), "l0.mix.r": (36, 96),
                        "l0.mix.g": (36, 96), "l0.mix.w1": (7, 96), "l0.mix.w2": (36, 7), "l0.mix.w0": (36,), "l0.mix.u": (3, 12),
                        "l0.mix.norm": (36,), "l0.mix.o": (96, 36), "l0.mlp.router": (6, 96), "l0.mlp.e5.gate": (24, 96),
                        "l0.mlp.shared.up": (40, 96), "l1.mix.q": (96, 96), "l1.mix.k": (48, 96), "l1.mix.v": (32, 96),
                        "l1.mix.sink": (4,), "l1.mix.g": (4, 96), "l1.mix.o": (96, 64), "l1.mlp.up": (40, 96), "l1.mlp.up.b": (40,),
                        "l1.mlp.down": (96, 40), "l1.mlp.down.b": (96,), "l2.mix.q": (60, 96), "l2.mix.dkv": (40, 96),
                        "l2.mix.dkv.norm": (40,), "l2.mix.uk": (60, 40), "l2.mix.uv": (84, 40), "l2.mix.o": (96, 84)}.items():
        assert names[name] == shape, name
    for absent in ("l0.mlp.e6.gate", "l2.mlp.shared.gate", "l3.norm2", "l3.rg2", "l1.mlp.gate", "l2.mix.g", "l2.mix.dq", "l0.norm1.b"):
        assert absent not in names
    assert "loop.step" not in {t.name for t in expected_tensors(cases.config_for("R").model_spec())}


def test_the_decay_rank_comes_from_a_tensor():
    raw = cases.config_json("P")
    config = TekaraxConfig.from_dict(raw)
    with pytest.raises(ValueError, match="decay rank is not known"):
        config.model_spec()
    shapes = {t.name: t.shape for t in expected_tensors(cases.config_for("P").model_spec())}
    assert config.with_tensor_shapes(shapes) == cases.config_for("P")


def test_the_order_in_which_looped_layers_run():
    runs = lambda name: [(e.layer, e.add_row) for e in cases.config_for(name).model_spec().schedule]
    assert runs("P") == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]
    assert runs("Q") == [(0, None), (1, 0), (2, None)]  # a loop that runs once still adds its row
    assert runs("R") == [(i, None) for i in range(5)]
    assert runs("S") == [(0, 0), (1, None), (0, 1), (1, None), (2, None)]
    for name in ("P", "Q", "R", "S"):
        assert plain.layer_runs(cases.CASES[name]) == runs(name)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=15), "pairs"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "at most"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "lacks low"),
    (lambda c: c["layers"][2]["mixer"].pop("mask"), "lacks mask"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "lacks dim"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "does not fit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "unknown kind"),
    (lambda c: c["loop"].update(stop=9), "do not lie within"),
    (lambda c: c["loop"].update(times=0), "positive"),
    (lambda c: c.pop("width"), "lacks required keys"),
])
def test_refused_configurations(change, message):
    raw = copy.deepcopy(cases.CASES["P"])
    change(raw)
    with pytest.raises(ValueError, match=message):
        TekaraxConfig.from_dict(raw)


def test_cache_groups_and_state():
    needs = LayeredModel(cases.config_for("P").model_spec()).cache_needs()
    assert len(needs) == 9 and [n.owner for n in needs] == list(range(9))  # every run of a looped layer keeps its own
    mixing = needs[0]
    assert mixing.kv is None and {k: tuple(s.shape) for k, s in mixing.state.items()} == {"shift": (96,), "matrix": (3, 12, 12)}
    attention = needs[1]  # keys of 24 and values of 16 are laid out in rows of 24
    assert (attention.kv.num_kv_heads, attention.kv.head_dim, attention.kv.window, attention.kv.planes) == (2, 24, None, 2)
    latent = needs[2]
    assert (latent.kv.num_kv_heads, latent.kv.head_dim, latent.kv.window, latent.kv.planes) == (1, 40, 13, 1)
    assert needs[7].kv.window == 5 and needs[7].state is None


def test_a_row_outside_the_table_is_refused():
    import dataclasses

    from torchlet_b200.config import ScheduleEntry

    spec = cases.config_for("P").model_spec()
    broken = dataclasses.replace(spec, schedule=(ScheduleEntry(0, add_row=3),))
    with pytest.raises(ValueError, match="row 3 of a table of 3"):
        broken.validate()


def test_plain_recurrence_in_closed_form():
    g = torch.Generator().manual_seed(5)
    T, H, D = 7, 2, 3
    r, k, v = (torch.randn(T, H, D, generator=g, dtype=torch.float64) for _ in range(3))
    decay = torch.rand(T, H, D, generator=g, dtype=torch.float64)
    u = torch.randn(H, D, generator=g, dtype=torch.float64)
    o = plain.wkv_scan(r, k, v, decay, u)
    t, h = 5, 1
    # o_t = sum_(s < t) (prod_(s < q < t) a_q * k_s . r_t) v_s + (u k_t . r_t) v_t: the decay of a step meets the tokens
    # before it only, and never the newest of them
    want = (u[h] * k[t, h] * r[t, h]).sum() * v[t, h]
    for s in range(t):
        a = torch.prod(decay[s + 1:t, h], dim=0)
        want = want + (a * k[s, h] * r[t, h]).sum() * v[s, h]
    assert torch.allclose(o[t, h], want, rtol=1e-12)
    assert torch.allclose(o[0, h], (u[h] * k[0, h] * r[0, h]).sum() * v[0, h], rtol=1e-12)
    x = torch.randn(4, 5, generator=g, dtype=torch.float64)
    mu = torch.rand(5, generator=g, dtype=torch.float64)
    shifted = plain.token_shift(x, mu)
    assert torch.allclose(shifted[0], x[0] * (1 - mu)) and torch.allclose(shifted[3], x[3] + (x[2] - x[3]) * mu)


def test_plain_attention_window_sink_and_turned_values():
    T = 12
    v = torch.eye(T, dtype=torch.float64).view(T, 1, T)
    zero = torch.zeros(T, 1, 2, dtype=torch.float64)
    out = plain.softmax_attention(zero, zero, v, 1.0, window=3)[:, 0]
    want = torch.zeros(T, dtype=torch.float64)
    want[7:10] = 1.0 / 3.0
    assert torch.allclose(out[9], want) and torch.allclose(out[0], torch.eye(T, dtype=torch.float64)[0])
    # a sink of score ln 5 beside four keys of score 0: each key gets 1 / 9
    out = plain.softmax_attention(zero, zero, v, 7.0, sink=torch.tensor([math.log(5.0)], dtype=torch.float64))[:, 0]
    assert torch.allclose(out[3, :4], torch.full((4,), 1.0 / 9.0, dtype=torch.float64))
    # values turned by their position and turned back by the query's: only the distance counts
    freq = plain.plain_frequencies(100.0, 4)
    one = torch.randn(1, 1, 4, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    near = plain.rotate_halves(plain.rotate_halves(one, torch.tensor([5]), freq), torch.tensor([-9]), freq)
    far = plain.rotate_halves(plain.rotate_halves(one, torch.tensor([105]), freq), torch.tensor([-109]), freq)
    assert torch.allclose(near, far, rtol=1e-10)
    f = plain.key_frequencies({"base": 100.0, "dims": 4, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 16}})
    s = (16 / (2 * math.pi) - 1.0) / 3.0  # wavelengths 2 pi (blended) and 20 pi (slowed down by the factor)
    assert math.isclose(float(f[0]), (1 - s) / 4.0 + s) and math.isclose(float(f[1]), 0.1 / 4.0)


def test_plain_units_and_router():
    assert plain.relu_squared(torch.tensor([-3.0, 0.0, 2.0])).tolist() == [0.0, 0.0, 4.0]
    w = {"m.router": torch.tensor([[1.0], [3.0], [2.0]], dtype=torch.float64)}
    chosen, weight = plain.route({"router": {"experts": 3, "top": 2}}, w, "m.", torch.ones(1, 1, dtype=torch.float64))
    assert chosen.tolist() == [[1, 2]]
    assert torch.allclose(weight, torch.sigmoid(torch.tensor([[3.0, 2.0]], dtype=torch.float64)))  # not renormalized
