"""Negilorn without a GPU: the configuration reader and its faults, the plan's tensor names, what every layer keeps in the
cache and whose keys it reads, pages given back at the end of a chunk, random-model folders, and the plain mechanisms on
cases worked out by hand."""
import copy
import math

import numpy as np
import pytest

import plain_negilorn as N
from negilorn_helpers import CONFIGS, drawn_config, lively_weights, tensor_shapes


def plan_of(raw):
    from velox_b200.config import resolve_architecture
    arch = resolve_architecture(raw)
    cfg = arch.config_class.from_dict(raw)
    return cfg, arch.plan(cfg)


def without_ranks(raw):
    raw = copy.deepcopy(raw)
    for lay in raw["layers"]:
        lay["mixer"].pop("rank", None)
    return raw


@pytest.mark.parametrize("name", sorted(CONFIGS) + ["drawn 0", "drawn 3", "drawn 6"])
def test_the_plan_asks_for_the_tensors_of_the_design(name):
    from velox_b200.models.decoder import DecoderModel
    raw = CONFIGS[name] if name in CONFIGS else drawn_config(int(name.split()[1]))
    cfg, plan = plan_of(raw)
    assert type(cfg).__name__ == "NegilornConfig" and cfg.to_dict()["layers"] == raw["layers"]
    assert plan_of(cfg.to_dict())[0] == cfg
    want = tensor_shapes(raw)
    assert {s.name: tuple(s.shape) for s in DecoderModel(plan).tensor_specs()} == want
    # without the middle width of the decays in the configuration, the file's tensor decides it
    open_ended = {s.name: tuple(s.shape) for s in DecoderModel(plan_of(without_ranks(raw))[1]).tensor_specs()}
    assert set(open_ended) == set(want)
    for n, shape in open_ended.items():
        assert len(shape) == len(want[n]) and all(a in (b, -1) for a, b in zip(shape, want[n]))


def test_what_the_layers_keep_and_whose_keys_they_read():
    from velox_b200.cache.kinds import flat_specs
    from velox_b200.models.decoder import DecoderModel
    from velox_b200.parts import BorrowedCache, CacheParts, FixedState, PagedKV
    model = DecoderModel(plan_of(CONFIGS["even"])[1])
    specs = model.cache_specs()
    row = FixedState((128,))
    # layer 0's keys are read with chunks of 40 and of 16: kept as a window of the longer; layer 2's by chunks of 50 alone
    assert specs[0] == CacheParts((row, PagedKV(2, 64, 40, 0, 0, 0, 0)))
    assert specs[1] == CacheParts((row, CacheParts((row, FixedState((4, 32, 32))))))
    assert specs[2] == CacheParts((row, PagedKV(1, 128, 0, 64, 0, 0, 50)))
    assert specs[4] == specs[5] == CacheParts((row, BorrowedCache()))
    assert specs[6] == CacheParts((row, PagedKV(2, 32, 0, 0, 0, 0, 96)))
    assert model.cache_sources() == [None, None, None, None, 2, 0, None]
    assert flat_specs(specs[4]) == [row] and len(flat_specs(specs[1])) == 3
    # an owner whose borrower sees everything keeps everything
    raw = copy.deepcopy(CONFIGS["even"])
    del raw["layers"][5]["mixer"]["mask"]
    assert DecoderModel(plan_of(raw)[1]).cache_specs()[0].parts[1] == PagedKV(2, 64, 0, 0, 0, 0, 0)


def test_pages_before_the_next_tokens_chunk_are_given_back():
    from velox_b200.cache.manager import CacheManager
    from velox_b200.parts import PagedKV
    cache = CacheManager([PagedKV(2, 8, chunk=40), PagedKV(2, 8, 40), PagedKV(2, 8)], [None] * 3, page_size=16, num_pages=12, max_requests=2,
                         max_blocks=12)
    held = lambda: [sum(1 for p in t if p >= 0) for t in cache.requests["a"].tables]
    cache.add_request("a")

    def go(n):
        assert cache.reserve("a", n)
        cache.commit("a", n)
        cache.check()
        return held()
    assert go(39) == [3, 3, 3]          # the next token, 39, still belongs to the first chunk
    assert go(1) == [1, 3, 3]           # the next one opens chunk 2: of its page (32 .. 47) only positions from 40 on are read
    assert go(25) == [3, 4, 5]          # 65: pages 2, 3, 4; the window still reads 26
    assert go(14) == [3, 3, 5]          # 79
    assert go(1) == [0, 3, 5]           # 80, a chunk's and a page's edge: nothing of the past is read
    assert go(40) == [1, 3, 8]          # 120: page 7 (112 .. 127)
    cache.release("a")
    assert cache.free_pages() == [12, 12, 12]


def test_a_borrowing_place_gets_the_lenders_pages_and_a_state_of_its_own():
    import torch
    from velox_b200.cache.manager import CacheManager
    from velox_b200.models.decoder import DecoderModel
    model = DecoderModel(plan_of(CONFIGS["even"])[1])
    cache = CacheManager(model.cache_specs(), model.cache_sources(), page_size=16, num_pages=4, max_requests=2, max_blocks=4,
                         device=torch.device("cpu"))
    own, lent = cache.layer(2), cache.layer(4)
    assert lent.parts[1].k_pool.data_ptr() == own.parts[1].k_pool.data_ptr() and lent.parts[1].group == own.parts[1].group
    assert own.parts[1].writes and not lent.parts[1].writes
    assert lent.parts[0].state.data_ptr() != own.parts[0].state.data_ptr() and lent.parts[0].writes
    mix = cache.layer(1)
    assert tuple(mix.parts[1].parts[0].state.shape) == (2, 128) and tuple(mix.parts[1].parts[1].state.shape) == (2, 4, 32, 32)
    assert len(cache.groups) == 3 and [g.layers for g in cache.groups] == [[0], [2], [6]]
    # a slot that is handed out again starts from zeros in every one of these
    slot = cache.add_request("a")
    for st in (own.parts[0].state, lent.parts[0].state, mix.parts[1].parts[1].state):
        st[slot] = 3.0
    cache.release("a")
    assert cache.add_request("b") == slot
    for st in (own.parts[0].state, lent.parts[0].state, mix.parts[1].parts[1].state):
        assert float(st[slot].abs().max()) == 0.0
    with pytest.raises(ValueError):
        CacheManager([model.cache_specs()[4]], [None], 16, 4, 2, 4)


@pytest.mark.parametrize("change,fault", [
    (lambda c: c.pop("vocab"), "missing key 'vocab'"),
    (lambda c: c["norm"].pop("eps"), "missing key 'norm.eps'"),
    (lambda c: c.update(layers=[]), "key 'layers': expected a list"),
    (lambda c: c["layers"][0].update(type="conv"), "layers[0].type 'conv'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "heads (4) is not a multiple of kv_heads (3)"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale must be a number"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "softcap must be a number above 0"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims (7) must be even"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "rot.scaling.low must be a number"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size must be a positive integer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=4), "kv_from 4 must name an earlier attention layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from 1 must name an earlier attention layer"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=10), "kv_heads, dim and vdim must equal that layer's"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "mixer.dim must be a positive integer"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top (6) exceeds experts (5)"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "mlp.expert.ff must be a positive integer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "mlp.kind 'gated' is not 'dense' or 'moe'"),
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
    cfg, plan = plan_of(raw)
    last = plan.layers[4]
    assert last.mixer.params["chunk"] == 0 and last.mixer.params["score_softcap"] == 0.0 and last.mixer.params["position"] is None
    assert last.feed_forward.params["shared"] is None and plan.layers[2].feed_forward is None and set(plan.layers[2].norms) == {"mixer"}
    assert plan.layers[2].cache_of == 0 and not plan.layers[2].mixer.params["own_kv"]
    del raw["logit_scale"]
    assert plan_of(raw)[1].head.params["logit_scale"] == 1.0


def test_a_random_model_folder_can_be_written_and_read_back(tmp_path):
    from velox_b200.config import load_config
    from velox_b200.weights.random_init import write_random_model
    from velox_b200.weights.safetensors_io import SafetensorsFile
    cfg, _ = plan_of(CONFIGS["routed"])
    folder = write_random_model(str(tmp_path / "m"), cfg, seed=4)
    arch, back = load_config(folder)
    assert arch.name == "Negilorn" and back == cfg
    f = SafetensorsFile(str(tmp_path / "m" / "model.safetensors"))
    assert set(f.keys()) == set(tensor_shapes(CONFIGS["routed"]))
    assert tuple(f.tensor("l0.norm1").shape) == ()
    share = f.tensor("l1.shift").float().numpy()
    assert share.min() >= 0.0 and share.max() <= 1.0 and 0.3 < share.mean() < 0.7
    f.close()


def test_the_frequencies_are_those_of_the_plain_implementation():
    from velox_b200.parts.position import RotaryPosition
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}
    part = RotaryPosition("", head_dim=32, theta=5000.0, rotary_dim=24, scaling=sc)
    want = N.rotary_frequencies({"base": 5000.0, "dims": 24, "scaling": sc})
    assert part.magnitude == 1.0 and np.abs(part.inverse_frequencies() / want - 1.0).max() < 1e-6
    with pytest.raises(ValueError):
        RotaryPosition("", head_dim=32, scaling={"factor": 8.0, "low": 1.0, "original": 256})


# -- the plain mechanisms on cases worked out by hand ----------------------------------------------------------------------

def test_the_norm_has_one_multiplier_and_the_shift_takes_zeros_before_the_first_row():
    x = np.array([[3.0, 4.0], [6.0, 8.0]])
    assert np.allclose(N.scalar_norm(x, 2.0, 0.0), 2.0 * x / np.array([[math.sqrt(12.5)], [math.sqrt(50.0)]]))
    h = np.array([[1.0, 10.0], [3.0, 30.0]])
    assert np.allclose(N.token_shift(h, np.array([0.25, 1.0])), [[0.75, 0.0], [2.5, 10.0]])


def test_chunks_are_counted_from_the_first_position():
    m = N.chunk_mask(7, 3)
    assert m[2].tolist() == [True, True, True, False, False, False, False]
    assert m[3].tolist() == [False, False, False, True, False, False, False]
    assert m[5].tolist() == [False, False, False, True, True, True, False] and m[6].sum() == 1
    assert np.array_equal(N.chunk_mask(4, 1), np.eye(4, dtype=bool)) and N.chunk_mask(4, 0)[3].all()


def test_one_is_added_to_the_denominator():
    p = N.softmax_plus_one(np.array([[0.0, 5.0], [math.log(3.0), 0.0]]), np.array([[True, False], [True, True]]))
    assert np.allclose(p, [[0.5, 0.0], [0.6, 0.2]])
    assert np.allclose(N.softmax_plus_one(np.array([[800.0]]), np.array([[True]])), 1.0)
    assert np.allclose(N.softmax_plus_one(np.array([[-800.0]]), np.array([[True]])), 0.0)


def test_frequencies_are_stretched_by_wavelength():
    rot = {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}}
    f, plain = N.rotary_frequencies(rot), N.rotary_frequencies({"base": 10000.0, "dims": 8})
    # wavelengths 6.28 (below 25: kept), 62.8 (between), 628 and 6,283 (above 100: four times slower)
    assert np.allclose(plain, [1.0, 0.1, 0.01, 0.001]) and f[0] == 1.0 and np.allclose(f[2:], plain[2:] / 4.0)
    s = (100.0 / (2.0 * math.pi / 0.1) - 1.0) / 3.0
    assert abs(f[1] - ((1.0 - s) * 0.025 + s * 0.1)) < 1e-15


def test_the_recurrence_sees_the_current_token_through_the_bonus_only():
    r, k, v = np.array([[[1.0, 2.0]], [[3.0, 1.0]]]), np.array([[[1.0, 1.0]], [[0.5, 2.0]]]), np.array([[[1.0, 0.0]], [[0.0, 1.0]]])
    w, u = np.full((2, 1, 2), 0.5), np.array([[2.0, 0.0]])
    o, S = N.wkv_walk(r, k, v, w, u)
    assert np.allclose(o[0, 0], [2.0, 0.0])                         # r . (u k) v with u = (2, 0): 1 * 2 * 1
    assert np.allclose(o[1, 0], [4.0, 3.0])                         # the first token undecayed: (3 + 1) v_0; own: 3 * 2 * 0.5
    assert np.allclose(S[0], [[0.5, 0.5], [0.5, 2.0]])
    # in two pieces, the second from the first one's state
    o1, S1 = N.wkv_walk(r[:1], k[:1], v[:1], w[:1], u)
    o2, S2 = N.wkv_walk(r[1:], k[1:], v[1:], w[1:], u, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)


def test_the_weight_enters_an_expert_before_its_square():
    rng = np.random.default_rng(0)
    h, W = rng.normal(size=(5, 6)), rng.normal(size=(3, 6))
    P = {"router": W}
    for e in range(3):
        P["e%d.up" % e], P["e%d.down" % e] = rng.normal(size=(4, 6)), rng.normal(size=(6, 4))
    y = N.routed_feed_forward(h, P, {"router": {"experts": 3, "top": 2}})
    chosen, weight = N.route(h, W, 2)
    s = N.sigmoid(h @ W.T)
    for t in range(5):
        assert list(chosen[t]) == list(np.argsort(-s[t])[:2]) and np.allclose(weight[t], np.sort(s[t])[::-1][:2])
        # the activation is homogeneous of degree two: the weight comes out squared
        want = sum(s[t, e] ** 2 * N.expert(h[t:t + 1], P["e%d.up" % e], P["e%d.down" % e])[0] for e in chosen[t])
        assert np.allclose(y[t], want)


def test_borrowed_keys_are_the_owners_and_the_mask_is_the_borrowers():
    cfg = copy.deepcopy(CONFIGS["odd"])
    w = lively_weights(cfg, 6)
    toks = list(range(40))
    base = N.forward(cfg, w, toks)
    w2 = dict(w)
    w2["l0.mix.k"] = w["l0.mix.k"][::-1].copy()
    layers, layers2 = [], []
    N.forward(cfg, w, toks, layers_out=layers)
    N.forward(cfg, w2, toks, layers_out=layers2)
    assert np.abs(layers2[2] - layers[2]).max() > 1e-3
    cfg2 = copy.deepcopy(cfg)
    cfg2["layers"][2]["mixer"]["mask"] = {"size": 20}
    got = N.forward(cfg2, w, toks)
    assert np.allclose(got[:19], base[:19]) and np.abs(got[19] - base[19]).max() > 1e-4


def test_the_state_reaches_across_chunks():
    cfg = CONFIGS["odd"]
    w = lively_weights(cfg, 7)
    a, b = [5] + list(range(1, 30)), [6] + list(range(1, 30))
    assert np.abs(N.forward(cfg, w, a)[-1] - N.forward(cfg, w, b)[-1]).max() > 1e-5


def test_greedy_generation_appends_the_most_likely_token():
    cfg = CONFIGS["ones"]
    w = lively_weights(cfg, 2)
    out = N.greedy_generate(cfg, w, [5, 6, 7], 3)
    assert out[0] == int(np.argmax(N.forward(cfg, w, [5, 6, 7])[-1])) and len(out) == 3
    assert out[1] == int(np.argmax(N.forward(cfg, w, [5, 6, 7, out[0]])[-1]))
