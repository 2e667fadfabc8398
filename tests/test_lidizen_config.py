"""The Lidizen configuration on the CPU: registry, the model's description and tensor names, refused configurations, cache
groups with kept first tokens and the model's own state, the page manager's kept pages, and the plain functions against
closed forms."""
import copy

import pytest
import torch

import lidizen_cases as cases
import plain_lidizen as plain
from torchlet_b200.cache.manager import CacheManager, GroupSpec
from torchlet_b200.config import LidizenConfig, config_from_dict, known_architectures
from torchlet_b200.parts import LayeredModel, expected_tensors

NAMES = ["P", "Q", "R", "S", "T"]


def test_registered_and_chosen_by_name():
    assert "Lidizen" in known_architectures()
    for name in NAMES:
        config = config_from_dict(cases.CASES[name])
        assert isinstance(config, LidizenConfig)
        assert LidizenConfig.from_dict(config.to_dict()) == config


def test_description_and_tensor_names():
    spec = cases.config_for("P").model_spec()
    assert all(layer.block == "hyper_connected" and layer.block_params["taps"] is None for layer in spec.layers)
    assert [layer.mixer.params["value_mix"] for layer in spec.layers] == [None, "first", None, "later"]
    assert [layer.mixer.params["keep_first"] for layer in spec.layers] == [5, 1, 18, 0]
    assert [layer.feed_forward.kind if layer.feed_forward else None for layer in spec.layers] == \
        ["gated_mlp", "routed_clamped_glu", None, "routed_clamped_glu"]
    assert (spec.token_pairs.buckets, spec.token_pairs.mul_prev, spec.token_pairs.mul_cur) == (37, 5, 3)
    tensors = {t.name: t for t in expected_tensors(spec)}
    for name, shape in {"embed": (101, 96), "bigram": (38, 96), "embed.norm": (96,), "final.norm": (96,), "l0.norm1": (96,),
                        "l0.norm2": (96,), "l0.hc1.in": (3,), "l0.hc2.out": (3,), "l0.hc1.mix": (3, 3), "l0.mix.q": (96, 96),
                        "l0.mix.q.b": (96,), "l0.mix.k": (48, 96), "l0.mix.k.b": (48,), "l0.mix.v": (32, 96), "l0.mix.v.b": (32,),
                        "l0.mix.q.norm": (96,), "l0.mix.k.norm": (48,), "l0.mix.talk": (4, 4), "l0.mix.o": (96, 64),
                        "l1.mix.vmix": (), "l0.mlp.gate.b": (40,), "l0.mlp.down.b": (96,), "l1.mlp.router": (6, 96),
                        "l1.mlp.router.b": (6,), "l1.mlp.e5.up": (24, 96), "l1.mlp.e5.down": (96, 24)}.items():
        assert tensors[name].shape == shape and not tensors[name].optional, name
    for absent in ("l1.mlp.e0.gate", "l1.mlp.e0.up.b", "l0.mix.o.b", "l0.norm1.b", "l0.canon1", "head"):
        assert absent not in tensors
    for unread in ("l2.norm2", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"):  # a layer without a feed-forward may carry them
        assert tensors[unread].optional and not tensors[unread.replace("l2", "l1")].optional
    assert tensors["l0.mix.vmix"].optional and tensors["lm_head"].optional
    assert "bigram" not in {t.name for t in expected_tensors(cases.config_for("S").model_spec())}


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "lacks scale"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=22), "at most"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "negative"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=16), "cannot be mixed"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "exceeds"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown kind"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "lacks mul_cur"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "positive"),
    (lambda c: c.pop("width"), "lacks required keys"),
])
def test_refused_configurations(change, message):
    raw = copy.deepcopy(cases.CASES["P"])
    change(raw)
    with pytest.raises(ValueError, match=message):
        LidizenConfig.from_dict(raw)


def test_options_that_do_not_go_together_are_refused():
    from torchlet_b200.config.spec import PartSpec
    from torchlet_b200.parts import FEED_FORWARDS, MIXERS, build_part

    base = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "score_mix": True}
    for extra in ({"softcap": 3.0}, {"sink": True}, {"gate": "sigmoid"}, {"values_from_keys": True}, {"chunk": 8}):
        with pytest.raises(ValueError, match="not built together"):
            build_part(MIXERS, PartSpec("gated_attention", {**base, **extra}))
    with pytest.raises(ValueError, match="unknown value_mix"):
        build_part(MIXERS, PartSpec("gated_attention", {**base, "value_mix": "last"}))
    with pytest.raises(ValueError, match="unknown expert unit"):
        build_part(FEED_FORWARDS, PartSpec("routed_clamped_glu", {"hidden_size": 8, "intermediate_size": 8, "num_experts": 2,
                                                                  "top_k": 1, "limit": None, "unit": "tanh"}))


def test_cache_groups_and_state():
    from torchlet_b200.cache.storage import CacheStorage

    model = LayeredModel(cases.config_for("P").model_spec())
    needs = model.cache_needs()
    assert [(n.kv.num_kv_heads, n.kv.window, n.kv.keep_first) for n in needs] == [(2, 13, 5), (2, 37, 1), (3, 7, 18), (2, 20, 0)]
    storage = CacheStorage(needs, 8, 3, 20, 128, "cpu", torch.float32, model.state_specs())
    assert [(g.window, g.keep_first) for g in storage.groups] == [(13, 5), (37, 1), (7, 18), (20, 0)]
    assert storage.model_states["last_token"].shape == (3, 1) and storage.model_states["last_token"].dtype == torch.int32
    storage.model_states["last_token"][:] = 9
    storage.clear_slot(1)
    assert storage.model_states["last_token"].flatten().tolist() == [9, 0, 9]
    assert LayeredModel(cases.config_for("S").model_spec()).state_specs() == {}


@pytest.mark.parametrize("window,keep,page", [(13, 5, 8), (13, 8, 8), (13, 9, 8), (1, 17, 4), (40, 0, 8), (3, 60, 8), (16, 16, 16)])
def test_pages_of_kept_tokens_are_never_given_back(window, keep, page):
    manager = CacheManager([GroupSpec(1, 8, window, (0,), 60, keep_first=keep)], page, 2, 200)
    for rid, cuts in (("a", [37, 1, 1, 50, 3, 1, 1, 1, 1, 40]), ("b", [1] * 90)):
        manager.admit(rid)
        length = 0
        for n in cuts:
            length += n
            assert manager.extend(rid, length)
            manager.advance(rid, length)
            manager.check()
            visible = plain.visible(length + 1, window, keep)[length]  # what the next token sees
            needed = {j // page for j in range(length) if visible[j]}
            table = manager.table(rid, 0)
            held = {i for i, p in enumerate(table) if p}
            assert needed <= held, "every page the next token sees is held"
            assert all(i < -(-keep // page) or (i + 1) * page > length - window + 1 for i in held), "no other page is"
        manager.finish(rid)
        manager.check()
    assert manager.pools[0].num_free == 59


def test_plain_functions_in_closed_form():
    assert plain.bigram_rows([3, 5, 5], 7, 2, 3) == [7, (3 * 2 + 5 * 3) % 7, (5 * 2 + 5 * 3) % 7]
    seen = plain.visible(6, 2, 1)
    assert [row.nonzero().flatten().tolist() for row in seen] == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5]]
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    assert torch.allclose(plain.layer_norm(x, torch.tensor([2.0, 1.0]).double(), 0.0), torch.tensor([[-2.0, 1.0]]).double())
    # pairs turn by the same angle: the dot product of two rotated vectors depends on the distance alone
    q, k = torch.randn(1, 1, 6, dtype=torch.float64), torch.randn(1, 1, 6, dtype=torch.float64)
    at = lambda v, p: plain.rotate_pairs(v, torch.tensor([float(p)], dtype=torch.float64), 50.0, 4)
    assert torch.allclose((at(q, 9) * at(k, 4)).sum(), (at(q, 25) * at(k, 20)).sum())
    chosen, weight = plain.route(torch.tensor([[0.0, 2.0, 1.0]], dtype=torch.float64), 2)
    assert chosen.tolist() == [[1, 2]] and torch.allclose(weight, torch.softmax(torch.tensor([[2.0, 1.0]]).double(), -1))


def test_plain_prefix_property():
    """A position's logits do not depend on what follows it."""
    ids, whole = cases.plain_logits("P", 40, 3)
    part = plain.forward(cases.weights_for("P"), cases.CASES["P"], ids[:25]).float()
    assert torch.allclose(whole[:25], part, atol=1e-6)
