"""Sezanex without a GPU: the configuration reader, the spec and its schedule, the tensor names, the blended rotation, what
attention and experts refuse to combine, and the plain implementation against itself and by hand."""
import copy
import math

import pytest
import torch

import plain_sezanex as plain
from sezanex_util import CONFIGS, attention, config, dense, doubles, mamba2, moe, position_errors, prompts, random_weights
from trapetum_b200.config import ConfigError, PartSpec, SezanexConfig, load_config
from trapetum_b200.engine.model import Model, tensor_specs_for_config
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
    for n in optional:                               # the norms that nothing follows
        assert ".norm2" in n and cfg["layers"][int(n[1:n.index(".")])]["mlp"] is None, n
    assert ("loop.in" in specs) == bool(cfg.get("loop"))


def test_every_constant_comes_from_the_configuration():
    cfg = SezanexConfig.from_dict(CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (150, 48, 1e-5, 1, 3, 3)
    a = cfg.layers[3].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.rot.dims, a.rot.base) == (4, 2, 12, 8, 0.4, 33, 12, 1000.0)
    assert a.rot.scaling == {"factor": 3.0, "original": 128.0, "fast": 8.0, "slow": 1.0}
    m = cfg.layers[2].mixer
    assert (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (4, 15, 16, 4, 5, 3)
    assert cfg.layers[2].mlp is None and cfg.layers[1].mlp.ff == 40
    assert (cfg.layers[0].mlp.experts, cfg.layers[0].mlp.top, cfg.layers[0].mlp.ff) == (5, 2, 24)
    bare = SezanexConfig.from_dict(CONFIGS["C"])
    assert bare.loop is None and bare.layers[2].mixer.window is None and bare.layers[2].mixer.rot.dims == 0
    assert SezanexConfig.from_dict(CONFIGS["B"]).layers[2].mixer.rot.scaling is None


def test_a_repeated_span_is_a_schedule_in_which_every_call_owns_its_cache():
    _, spec = load_config(CONFIGS["A"])
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [e.before is not None for e in spec.schedule] == [False, True, False, True, False, True, False, False]
    assert all(e.cache_of is None for e in spec.schedule)
    needs, readers = Model(spec, CPU).cache_needs()
    assert readers == {} and [type(needs[e]) for e in range(8)] == [KVNeed] + [StateNeed] * 6 + [KVNeed]
    assert (needs[0].window, needs[7].window, needs[7].n_kv_heads) == (5, 33, 2)
    assert [(e.layer, e.before is not None) for e in spec.schedule] == plain.calls(CONFIGS["A"])
    for name in "BC":
        assert [(e.layer, e.before is not None) for e in load_config(CONFIGS[name])[1].schedule] == plain.calls(CONFIGS[name])


@pytest.mark.parametrize("change, says", [
    (lambda c: c["layers"][0].__setitem__("type", "gla"), "known mixers"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "rot.scaling.slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), "scaling.factor"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "layers[1].mixer.state"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("groups", 3), "groups=3"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("norm_groups", 7), "norm_groups=7"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "glu"), "known kinds: dense, moe"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top=6 of experts=5"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "layers[1].mlp.ff"),
    (lambda c: c["loop"].__setitem__("stop", 5), "loop start=1 stop=5"),
    (lambda c: c["loop"].pop("times"), "loop.times"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_a_wrong_configuration_is_refused_with_the_keys_name(change, says):
    c = copy.deepcopy(CONFIGS["A"])
    change(c)
    with pytest.raises(ConfigError) as e:
        SezanexConfig.from_dict(c)
    assert says in str(e.value)


@pytest.mark.parametrize("rot", [
    {"dims": 16, "base": 500.0, "scaling": {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}},
    {"dims": 2, "base": 20.0, "scaling": {"factor": 8.0, "original": 16, "fast": 4.0, "slow": 0.5}},
    {"dims": 64, "base": 10000.0, "scaling": {"factor": 0.5, "original": 4096, "fast": 32.0, "slow": 1.0}},
    {"dims": 8, "base": 100.0, "scaling": {"factor": 2.0, "original": 64, "fast": 1.0, "slow": 1.0}},       # a ramp of no width
    {"dims": 12, "base": 1000.0},
])
def test_the_blended_rotation_and_its_factor(rot):
    rope = build_part("position", PartSpec("rope", {"head_dim": rot["dims"] + 4, "rotary_dim": rot["dims"], "theta": rot["base"],
                                                    "scaling": rot.get("scaling"), "table": "float64"}), "", CPU)
    rope.bind({})
    f, mult = plain.frequencies(rot)
    assert torch.equal(rope.rotary_table()[0], f.float()) and rope.rotary_table()[1] == rot["dims"]
    assert abs(rope.amplitude - mult) < 1e-12


def test_a_factor_on_the_rotation_goes_through_the_path_that_has_it_or_is_refused():
    rot = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    pos = PartSpec("rope", {"head_dim": 8, "theta": 10.0, "scaling": rot})
    plain_attention = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "scale": 0.5, "position": pos,
                       "q": "q", "k": "k", "v": "v", "o": "o"}
    assert build_part("mixer", PartSpec("attention", plain_attention), "", CPU).projected
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("retention", {"hidden_size": 16, "heads": 1, "key_dim": 8, "value_dim": 8, "decay": [0.9], "k_scale": None,
                                                   "eps": 1e-5, "position": pos, "q": "q", "k": "k", "v": "v", "g": "g", "o": "o"}), "", CPU)
    with pytest.raises(ValueError):
        build_part("position", PartSpec("rope", {"head_dim": 8, "theta": 10.0, "scaling": rot, "scaling_factor": 2.0}), "", CPU)


def test_what_attention_experts_and_blocks_refuse_to_combine():
    base = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "scale": 0.5, "position": PartSpec("none", {"head_dim": 8}),
            "q": "q", "k": "k", "v": "v", "o": "o"}
    for more in ({"sink": "s", "unit_sink": True}, {"sink": "s", "talk": "t"}, {"value_gate": "g", "block": 4},
                 {"head_norm": {"q": "a", "k": "b", "eps": 1e-5}, "proj_norm": {"q": "a", "k": "b", "eps": 1e-5}}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("attention", dict(base, **more)), "", CPU)
    norms = {"q": "a", "k": "b", "eps": 1e-5}
    assert not build_part("mixer", PartSpec("attention", dict(base, unit_sink=True, proj_norm=norms)), "", CPU).mixed
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("routed_experts", {"hidden_size": 16, "experts": 2, "top": 1, "intermediate_size": 8,
                                                               "weight_on": "both", "router": "r", "expert": "e{}.", "gate": "g", "up": "u",
                                                               "down": "d"}), "", CPU)
    ffn = build_part("feed_forward", PartSpec("mlp", {"hidden_size": 16, "intermediate_size": 8, "activation": "gelu", "up": "u", "down": "d"}), "", CPU)
    mixer = build_part("mixer", PartSpec("attention", base), "", CPU)
    norm = PartSpec("dynamic_tanh", {"size": 16, "weight": "w", "bias": "b", "alpha": "a"})
    with pytest.raises(ValueError):
        build_part("block", PartSpec("sandwich", {"pre_mixer_norm": norm, "post_mixer_norm": norm, "pre_ffn_norm": norm}), "", CPU,
                   mixer=mixer, feed_forward=ffn)


def test_a_stream_is_not_replaced_while_an_addition_waits():
    from trapetum_b200.parts import ResidualStream
    s = ResidualStream(torch.zeros(2, 4))
    s.replace(torch.ones(1, 2, 4))
    assert float(s.h.sum()) == 8.0                     # one part: its memory is the stream
    s.add(torch.ones(2, 4))
    with pytest.raises(RuntimeError):
        s.replace(torch.ones(3, 2, 4))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_plain_implementation_fed_in_pieces_equals_itself(name):
    cfg = CONFIGS[name]
    w = doubles(random_weights(cfg, 2))
    ids = prompts(cfg["vocab"], [130], seed=1)[0]
    whole = plain.forward(cfg, w, ids)
    for pieces in ([129, 1], [1] * 130, [64, 2, 1, 63], [2] * 65, [5, 5, 5, 115]):
        assert float(position_errors(plain.logits(cfg, w, ids, pieces), whole).max()) < 1e-9


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_test_models_route_without_close_calls(name):
    """What the comparisons in 16 bits rest on: no winner changes for a rounding; and the scores are neither all one nor all
    zero, so that a missing or doubled weight shows."""
    cfg = CONFIGS[name]
    for seed in (23 + ord(name), 3):
        w = doubles(random_weights(cfg, seed))
        ids = prompts(cfg["vocab"], [200], seed=seed)[0]
        assert plain.routing_margin(cfg, w, ids) > 0.3
        i = next(j for j, L in enumerate(cfg["layers"]) if (L["mlp"] or {}).get("kind") == "moe")
        x = w["embed"][ids]
        h = plain.named_norm(x, w, f"l{i}.norm2")
        s = plain.route(h, w[f"l{i}.mlp.router"], cfg["layers"][i]["mlp"]["router"]["top"])[1][:, 0]
        assert float(((s > 0.05) & (s < 0.98)).double().mean()) > 0.4 and float(s.std()) > 0.05


def test_the_plain_mechanisms_by_hand():
    pos = torch.arange(12)
    window = plain.seen(pos, pos, 5)
    assert window[4, 0] and not window[5, 0] and window[5, 1] and not window[3, 4]
    p = plain.weights(torch.zeros(1, 3, dtype=plain.F), torch.ones(1, 3, dtype=torch.bool))
    assert torch.allclose(p, torch.full((1, 3), 0.25, dtype=plain.F))          # exp(0) / (1 + 3 exp(0))
    p = plain.weights(torch.full((1, 2), -800.0, dtype=plain.F), torch.ones(1, 2, dtype=torch.bool))
    assert float(p.abs().max()) == 0.0
    x = torch.tensor([-2.0, 0.0, 0.5], dtype=plain.F)
    assert torch.allclose(plain.dyt(x, 0.5, torch.tensor(2.0), torch.tensor(1.0)), torch.tanh(0.5 * x) * 2 + 1)
    assert abs(float(plain.gelu(torch.tensor(1.0, dtype=plain.F))) - 0.5 * (1 + math.erf(1 / math.sqrt(2)))) < 1e-12
    # the weight goes in, not out: an expert is not linear
    g = torch.Generator().manual_seed(0)
    t = {f"e0.{k}": torch.randn(*s, generator=g) for k, s in (("gate", (4, 3)), ("up", (4, 3)), ("down", (3, 4)))}
    t["router"] = torch.randn(1, 3, generator=g)
    h = torch.randn(2, 3, generator=g, dtype=plain.F)
    y = plain.routed(h, moe(1, 1, 4), t, "")
    s = torch.sigmoid(h @ t["router"].double().T)
    assert torch.allclose(y, plain.expert(s * h, t, "e0."))
    assert not torch.allclose(y, s * plain.expert(h, t, "e0."), rtol=1e-2)
    # the recurrence as the sum it is
    T, H, P, N = 6, 2, 3, 4
    xs, B, C = (torch.randn(T, n, k, generator=g, dtype=plain.F) for n, k in ((H, P), (1, N), (1, N)))
    dt, A, D = torch.rand(T, H, generator=g, dtype=plain.F), torch.randn(H, generator=g, dtype=plain.F), torch.randn(H, generator=g, dtype=plain.F)
    y, S = plain.recur(xs, B, C, dt, A, D, torch.zeros(H, N, P, dtype=plain.F))
    for hh in range(H):
        want = D[hh] * xs[5, hh] + sum(torch.exp(-torch.exp(A[hh]) * dt[j + 1:, hh].sum()) * dt[j, hh] * (B[j, 0] @ C[5, 0]) * xs[j, hh] for j in range(T))
        assert torch.allclose(y[5, hh], want)


def test_a_single_layer_model_of_every_kind_builds():
    for mixer in (attention(2, 1, 16, 24, 0.25, size=9, rot=(8, 100.0)), mamba2(2, 8, 16, groups=2, norm_groups=4)):
        for ff in (None, dense(24), moe(3, 2, 8)):
            for loop in (None, (0, 1, 1), (0, 1, 4)):
                specs = tensor_specs_for_config(config(50, 32, [(mixer, ff)], loop))
                assert ("loop.in" in specs) == bool(loop) and specs["l0.norm1.alpha"].shape == ()
                assert specs["l0.norm2b.alpha"].optional == (ff is None)
