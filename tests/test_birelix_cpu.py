"""Birelix without a GPU: the configuration reader and its faults, the plan's tensor names, what every layer keeps in the
cache, random-model folders, parts that refuse what they cannot do, and the plain mechanisms on cases worked out by hand."""
import copy
import math

import numpy as np
import pytest

import plain_birelix as P
from birelix_helpers import CONFIGS, drawn_config, lively_weights, tensor_shapes


def plan_of(raw):
    from velox_b200.config import resolve_architecture
    arch = resolve_architecture(raw)
    cfg = arch.config_class.from_dict(raw)
    return cfg, arch.plan(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS) + ["drawn 0", "drawn 3", "drawn 6"])
def test_the_plan_asks_for_the_tensors_of_the_design(name):
    from velox_b200.models.decoder import DecoderModel
    raw = CONFIGS[name] if name in CONFIGS else drawn_config(int(name.split()[1]))
    cfg, plan = plan_of(raw)
    assert type(cfg).__name__ == "BirelixConfig" and cfg.to_dict()["layers"] == raw["layers"]
    assert plan_of(cfg.to_dict())[0] == cfg
    assert {s.name: tuple(s.shape) for s in DecoderModel(plan).tensor_specs()} == tensor_shapes(raw)


def test_what_the_layers_keep():
    from velox_b200.models.decoder import DecoderModel
    from velox_b200.parts import CacheParts, FixedState, PagedKV, PagedLatent
    specs = DecoderModel(plan_of(CONFIGS["even"])[1]).cache_specs()
    assert specs[0] == PagedLatent(96, 0) and specs[5] == PagedLatent(72, 0)
    assert specs[1] == PagedKV(2, 64, 40) and specs[3] == PagedKV(1, 128, 16, 64)
    # (the ring of the convolutions' inputs holds a row per tap: q [2, 64], k [2, 64], v [4, 64]; the state is kept transposed)
    assert specs[2] == CacheParts((FixedState((4, 512)), FixedState((4, 64, 64))))
    assert specs[4] == CacheParts((FixedState((4, 576)), FixedState((2, 32, 128))))


def test_a_slot_that_is_handed_out_again_is_cleared():
    import torch
    from velox_b200.cache.manager import CacheManager
    from velox_b200.models.decoder import DecoderModel
    model = DecoderModel(plan_of(CONFIGS["deltas"])[1])
    cache = CacheManager(model.cache_specs(), model.cache_sources(), page_size=16, num_pages=4, max_requests=2, max_blocks=4,
                         device=torch.device("cpu"))
    slot = cache.add_request("a")
    states = [part.state for place in range(3) for part in cache.layer(place).parts]
    assert tuple(states[0].shape) == (2, 7, 540) and tuple(states[1].shape) == (2, 2, 140, 130)
    for st in states:
        st[slot] = 3.0
    cache.release("a")
    assert cache.add_request("b") == slot and all(float(st[slot].abs().max()) == 0.0 for st in states)


@pytest.mark.parametrize("change,fault", [
    (lambda c: c.pop("vocab"), "missing key 'vocab'"),
    (lambda c: c["norm"].pop("eps"), "missing key 'norm.eps'"),
    (lambda c: c.update(layers=[]), "key 'layers': expected a list"),
    (lambda c: c["layers"][0].update(type="conv"), "layers[0].type 'conv'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "heads (6) is not a multiple of kv_heads (4)"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "mixer.conv must be a positive integer"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=5), "rot_dim (5) must be even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), "rot.dims must equal rot_dim"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "mixer.rot.base must be a number"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "mixer.q_rank must be a positive integer"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "mixer.scale must be a number"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "mask.size must be a positive integer"),
    (lambda c: c["layers"][2]["mixer"].update(mask=7), "mask must hold a size"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top (6) exceeds the experts of the kept groups (5)"),
    (lambda c: c["layers"][4]["mlp"]["router"]["groups"].update(keep=1), "top (4) exceeds the experts of the kept groups (2)"),
    (lambda c: c["layers"][4]["mlp"]["router"]["groups"].update(count=3), "4 experts do not form 3 equal groups"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "expert.limit must be a number above 0"),
    (lambda c: c["layers"][0]["mlp"].pop("expert"), "mlp.expert.ff must be a positive integer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "mlp.kind 'gated' is not 'dense' or 'moe'"),
])
def test_faults_of_a_configuration_are_named(change, fault):
    from velox_b200.config import ConfigError
    raw = copy.deepcopy(CONFIGS["odd"])
    change(raw)
    with pytest.raises(ConfigError) as e:
        plan_of(raw)
    assert fault in str(e.value)


def test_absent_keys_mean_not_there():
    raw = copy.deepcopy(CONFIGS["odd"])
    del raw["layers"][2]["mixer"]["mask"], raw["embedding"]
    cfg, plan = plan_of(raw)
    assert plan.layers[2].mixer.params["window"] == 0 and plan.layers[2].feed_forward is None and set(plan.layers[2].norms) == {"mixer"}
    assert plan.layers[0].feed_forward.params["groups"] == 1 and plan.embedding.params["scale"] == 1.0
    assert "l2.norm2" in plan.ignored_tensors


def test_a_random_model_folder_can_be_written_and_read_back(tmp_path):
    from velox_b200.config import load_config
    from velox_b200.weights.random_init import write_random_model
    from velox_b200.weights.safetensors_io import SafetensorsFile
    cfg, _ = plan_of(CONFIGS["routed"])
    folder = write_random_model(str(tmp_path / "m"), cfg, seed=4)
    arch, back = load_config(folder)
    assert arch.name == "Birelix" and back == cfg
    f = SafetensorsFile(str(tmp_path / "m" / "model.safetensors"))
    assert set(f.keys()) == set(tensor_shapes(CONFIGS["routed"]))
    assert 0.3 < f.tensor("l0.mix.v.conv").float().numpy().std() < 0.7
    f.close()


def test_parts_refuse_what_they_cannot_do():
    from velox_b200.parts import GatedDeltaRule, LatentAttention, PartSpec, PreNormBlock, RoutedExperts
    sizes = dict(hidden_size=64, num_heads=4, num_kv_heads=2, head_dim=32, v_head_dim=32, conv_taps=4)
    GatedDeltaRule("x.", **sizes)
    for change in (dict(num_kv_heads=3), dict(head_dim=257), dict(v_head_dim=0), dict(conv_taps=65)):
        with pytest.raises(ValueError):
            GatedDeltaRule("x.", **dict(sizes, **change))
    with pytest.raises(ValueError, match="not both"):
        LatentAttention("x.", 64, 2, 16, 8, 16, 32, 0.2, PartSpec("rotary", "", dict(head_dim=8, theta=100.0)), output_gate=True, head_gate=True)
    with pytest.raises(ValueError, match="bounded gate"):
        RoutedExperts("x.", 64, 4, 2, 32, scores="sigmoid", gated=False, names=("up", "down"), capped=(1.0, 1.7))
    with pytest.raises(ValueError, match="needs a feed-forward"):
        PreNormBlock(GatedDeltaRule("x.", **sizes), None, {"mixer": None, "feed_forward": None})
    with pytest.raises(ValueError, match="renormalised"):
        RoutedExperts("x.", 64, 4, 2, 32, renormalise=True)


# -- the plain mechanisms on cases worked out by hand ----------------------------------------------------------------------

def test_windows_hold_the_token_itself_and_those_right_before_it():
    m = P.window_mask(5, 2)
    assert m[0].tolist() == [True] + [False] * 4 and m[3].tolist() == [False, False, True, True, False]
    assert np.array_equal(P.window_mask(4, 1), np.eye(4, dtype=bool)) and P.window_mask(4, 0)[3].all()


def test_one_is_added_to_the_denominator():
    s, m = np.array([[0.0, 5.0], [math.log(3.0), 0.0]]), np.array([[True, False], [True, True]])
    assert np.allclose(P.softmax(s, m, plus_one=True), [[0.5, 0.0], [0.6, 0.2]])
    assert np.allclose(P.softmax(s, m), [[1.0, 0.0], [0.75, 0.25]])
    assert np.allclose(P.softmax(np.array([[-800.0]]), np.array([[True]]), plus_one=True), 0.0)


def test_neighbours_are_turned_together():
    x = np.zeros((2, 1, 4))
    x[:, 0, 0] = x[:, 0, 2] = 1.0
    y = P.rotate_neighbours(x, [0, 3], 100.0)
    assert np.allclose(y[0], x[0])
    assert np.allclose(y[1, 0], [math.cos(3.0), math.sin(3.0), math.cos(0.3), math.sin(0.3)])


def test_the_last_tap_is_the_current_tokens_and_zeros_come_before_the_first():
    x, w = np.array([[1.0], [2.0], [4.0]]), np.array([[0.5, -1.0, 3.0]])
    assert np.allclose(P.short_convolution(x, w), P.silu(np.array([[3.0], [5.0], [0.5 - 2.0 + 12.0]])))
    assert np.allclose(P.short_convolution(x[:1], w), P.silu(np.array([[3.0]])))


def test_the_delta_rule_replaces_what_a_key_held():
    k = np.zeros((2, 1, 3))
    k[:, 0, 1] = 1.0
    v = np.array([[[2.0, 5.0]], [[7.0, -1.0]]])
    one = np.ones((2, 1))
    o, S = P.delta_walk(k, k, v, one, one)       # a full step: the second value takes the first one's place
    assert np.allclose(o[:, 0], v[:, 0]) and np.allclose(S[0], [[0, 0], [7, -1], [0, 0]])
    o, _ = P.delta_walk(k, k, v, 0.5 * one, 0.25 * one)
    first = 0.25 * v[0, 0]
    assert np.allclose(o[1, 0], 0.5 * first + 0.25 * (v[1, 0] - 0.5 * first))


def test_groups_are_judged_by_their_two_best_scores():
    z = np.array([[3.0, -3.0, 1.0, 0.9, 0.0, 0.0]])          # the largest score lies in a group whose second is small
    E = np.eye(6)
    chosen, w = P.route(z, E, {"top": 2, "groups": {"count": 3, "keep": 1}})
    s = P.sigmoid(z[0])
    assert chosen.tolist() == [[2, 3]] and np.allclose(w, [s[[2, 3]] / (s[2] + s[3])])
    assert P.route(z, E, {"top": 2})[0].tolist() == [[0, 2]]
    # groups of one are judged by that one
    assert P.route(z, E, {"top": 1, "groups": {"count": 6, "keep": 2}})[0].tolist() == [[0]]


def test_experts_have_bounds():
    h = np.array([[1.0, 10.0]])
    eye = np.eye(2)
    g = np.array([1.0, 2.0])
    assert np.allclose(P.expert(h, eye, -eye, eye, 2.0), g * P.sigmoid(1.702 * g) * (np.array([-1.0, -2.0]) + 1.0))


def test_a_sequence_and_its_beginning_agree():
    cfg = CONFIGS["odd"]
    w = lively_weights(cfg, 3)
    toks = [int(t) for t in np.random.default_rng(4).integers(0, cfg["vocab"], 25)]
    assert np.allclose(P.forward(cfg, w, toks)[:9], P.forward(cfg, w, toks[:9]))
    assert P.greedy_generate(cfg, w, toks[:5], 2)[0] == int(np.argmax(P.forward(cfg, w, toks[:5])[-1]))
