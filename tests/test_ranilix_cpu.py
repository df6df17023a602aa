"""Ranilix without a GPU: the configuration reader, the spec, the tensor names, the order of a rotated head's numbers, a
cache that keeps keys and a state for one layer, and the plain implementation against itself."""
import copy

import pytest
import torch

import plain_ranilix as plain
from ranilix_util import CONFIGS, attention, config, doubles, parallel, position_errors, prompts, random_weights
from trapetum_b200.config import ConfigError, PartSpec, RanilixConfig, load_config
from trapetum_b200.engine.model import tensor_specs_for_config
from trapetum_b200.parts import KVNeed, Runtime, StateNeed, build_part

CPU = Runtime(torch.float32, torch.device("cpu"))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_spec_names_the_tensors_of_a_model_folder(name):
    cfg = CONFIGS[name]
    w = random_weights(cfg, 1)
    specs = tensor_specs_for_config(cfg)
    optional = {n for n, s in specs.items() if s.optional}
    assert set(specs) - optional <= set(w) <= set(specs)
    for n in w:
        assert tuple(specs[n].shape) == tuple(w[n].shape), n
    # what may be absent: the norm that nothing follows, and the first mixing layer's number, which nothing reads
    for n in optional:
        i = int(n[1:n.index(".")])
        assert (n.endswith("norm2") and cfg["layers"][i]["mlp"] is None) or \
            (n.endswith("vmix") and not any(L["mixer"].get("v_mix") for L in cfg["layers"][:i])), n


def test_every_constant_comes_from_the_configuration():
    cfg = RanilixConfig.from_dict(CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.embedding_scale, cfg.norm_eps) == (150, 48, 3.0, 1e-5)
    a = cfg.layers[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.rot.dims, a.rot.base, a.v_mix) == (4, 2, 12, 8, 0.4, 33, 12, 1000.0, True)
    p = cfg.layers[1].mixer
    assert (p.left_scale, p.right_scale, p.right.decay, p.right.vdim, p.left.window) == (0.6, 1.3, (0.5, 0.9, 0.99), 10, None)
    assert cfg.layers[2].ff is None and cfg.layers[3].ff == 56 and cfg.layers[5].mixer.window is None
    assert RanilixConfig.from_dict(CONFIGS["C"]).embedding_scale == 1.0
    _, spec = load_config(CONFIGS["A"])
    mixes = [L.mixer.params.get("v_mix") for L in spec.layers]
    assert [None if m is None else m["first"] for m in mixes] == [None, None, True, False, None, False]
    assert spec.layers[0].block.params.keys() == {"norm", "ffn_norm"}


@pytest.mark.parametrize("change, says", [
    (lambda c: c["layers"][0].__setitem__("type", "attention_2"), "known mixers"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "layers[1].mixer.left_scale"),
    (lambda c: c["layers"][1]["mixer"]["right"]["decay"].pop(), "2 numbers for 3 heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].__setitem__("decay", 0.5), "right.decay"),
    (lambda c: c["layers"][1]["mixer"]["left"].__setitem__("v_mix", True), "left.v_mix"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "layers[0].mixer.rot.base"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 2), "kv_heads"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 16), "cannot be mixed"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "known kinds: dense"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "layers[0].mlp.ff"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_a_wrong_configuration_is_refused_with_the_keys_name(change, says):
    c = copy.deepcopy(CONFIGS["A"])
    change(c)
    with pytest.raises(ConfigError) as e:
        RanilixConfig.from_dict(c)
    assert says in str(e.value)


@pytest.mark.parametrize("dims, head", [(2, 6), (8, 8), (6, 10)])
def test_a_rotation_of_neighbours_is_a_rotation_of_halves_in_another_order(dims, head):
    rope = build_part("position", PartSpec("rope", {"head_dim": head, "rotary_dim": dims, "theta": 77.0, "pairing": "neighbours",
                                                    "table": "float64"}), "", CPU)
    order = torch.tensor(rope.head_order())
    assert sorted(order.tolist()) == list(range(head))
    x = torch.randn(9, 2, head, dtype=plain.F)
    pos = torch.arange(9) * 5
    assert torch.allclose(plain.turn(x, pos, dims, 77.0, True)[..., order], plain.turn(x[..., order], pos, dims, 77.0, False))
    rope.bind({})
    assert torch.equal(rope.rotary_table()[0].cpu(), plain.frequencies(dims, 77.0).float())
    assert build_part("position", PartSpec("rope", {"head_dim": head, "theta": 10.0}), "", CPU).head_order() is None


def test_a_layer_may_keep_keys_and_a_state():
    from trapetum_b200.cache import BothView, Cache
    cache = Cache({0: (KVNeed(2, 8), StateNeed((6,))), 1: KVNeed(2, 8), 2: StateNeed((3,))}, {}, 256, torch.float32, "cpu", max_slots=2)
    s = cache.claim()
    cache.grow({s: 70})
    v = cache.view(0, 0)
    assert isinstance(v, BothView) and v.kv.k.shape[1:] == (2, 64, 8) and v.state.data.shape == (2, 6)
    assert not isinstance(cache.view(1, 1), BothView) and cache.view(2, 2).data.shape == (2, 3)
    v.state.data[s] = 5.0
    cache.release(s)
    assert cache.claim() == s and float(cache.view(0, 0).state.data[s].abs().max()) == 0.0        # zero when a sequence starts
    cache.check()
    with pytest.raises(TypeError):
        Cache({0: (KVNeed(2, 8), KVNeed(1, 8))}, {}, 256, torch.float32, "cpu")


def test_mixers_side_by_side_hold_one_line_and_one_state():
    _, spec = load_config(CONFIGS["A"])
    pair = build_part("mixer", spec.layers[1].mixer, "l1.", CPU)
    kv, state = pair.cache_need()
    assert (kv.n_kv_heads, kv.head_dim, kv.window) == (2, 12, None) and state.shape == (3 * 12 * 10,)
    right = spec.layers[1].mixer.params["right"]
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("side_by_side", {"left": right, "right": right, "left_scale": 1, "right_scale": 1}), "l1.", CPU)


def test_argument_blocks_have_one_size_on_both_sides():
    """A Python structure that has drifted from its C struct would hand a kernel garbage pointers."""
    import ctypes
    from trapetum_b200.csrc import build, ops
    for library, function, mirror in ops.args_mirrors():
        assert getattr(build.load(library), function)() == ctypes.sizeof(mirror), mirror.__name__


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_plain_implementation_fed_in_pieces_equals_itself(name):
    cfg = CONFIGS[name]
    w = doubles(random_weights(cfg, 2))
    ids = prompts(cfg["vocab"], [130], seed=1)[0]
    whole = plain.forward(cfg, w, ids)
    for pieces in ([129, 1], [1] + [1] * 129, [64, 1, 2, 63], [5, 5, 5, 115]):
        assert float(position_errors(plain.logits(cfg, w, ids, pieces), whole).max()) < 1e-9


def test_the_plain_mechanisms_by_hand():
    pos = torch.arange(12)
    window = plain.seen(pos, pos, 5)
    assert window[4, 0] and not window[5, 0] and window[5, 1] and not window[3, 4]
    p = plain.weights(torch.zeros(1, 3, dtype=plain.F), torch.ones(1, 3, dtype=torch.bool), sink=0.0)
    assert torch.allclose(p, torch.full((1, 3), 0.25, dtype=plain.F))
    # retention as the sum it is: o_t = sum_j decay^(t - j) (q_t . k_j) v_j
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(7, 2, n, generator=g, dtype=plain.F) for n in (3, 3, 4))
    o, S = plain.retain(q, k, v, [0.5, 0.9], torch.zeros(2, 3, 4, dtype=plain.F))
    for h, d in enumerate((0.5, 0.9)):
        want = sum(d ** (6 - j) * (q[6, h] @ k[j, h]) * v[j, h] for j in range(7))
        assert torch.allclose(o[6, h], want)
        assert torch.allclose(S[h], sum(d ** (6 - j) * k[j, h][:, None] * v[j, h] for j in range(7)))


def test_a_single_layer_model_of_every_mixer_builds():
    for layer in (attention(2, 1, 16, 24, 0.25, size=9, rot=(8, 100.0)), parallel((2, 1, 16, 24, 0.25, None), (8, 16, (8, 10.0), (0.5, 1.0)))):
        specs = tensor_specs_for_config(config(50, 32, [(layer, None), (layer, 24)]))
        assert specs["l0.norm2"].optional and not specs["l1.norm2"].optional
