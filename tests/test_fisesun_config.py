"""Fisesun on the CPU: the configuration reader, the parts it picks, tensor names, the caches, and the plain implementation's
own mechanisms."""
import copy
import math

import pytest
import torch

import plain_fisesun as plain
from fisesun_cases import ALL, CONFIG_A, CONFIG_B, CONFIG_ODD, MOE, ONLY_EXPERTS, attention, mlstm, model
from mlx_lm_b200.cache import CacheManager
from mlx_lm_b200.config import ConfigError, get_architecture
from mlx_lm_b200.parts import (ExpertsMLP, GatedMLP, MLSTMMixer, OutputNormBlock, PagedKVSpec, RMSNorm, StateSpec,
                               TalkingHeadsAttention, rotation_frequencies)
from mlx_lm_b200.weights.loader import WeightError, check_tensors, random_tensors


def describe(config):
    arch = get_architecture(config)
    return arch.build(arch.args_class.from_dict(copy.deepcopy(config)))


def test_found_by_its_architecture_key_and_parts_follow_the_layer_list():
    d = describe(CONFIG_A)
    assert d.model_type == "fisesun" and d.position is None and d.head.tied_to is None and d.head.softcap == 25.0
    assert d.embedding.scale == 2.0 and isinstance(d.final_norm, RMSNorm)
    assert all(isinstance(b, OutputNormBlock) and isinstance(b.norm_1, RMSNorm) for b in d.blocks)
    assert [type(b.mixer) for b in d.blocks] == [MLSTMMixer, TalkingHeadsAttention, TalkingHeadsAttention, MLSTMMixer, TalkingHeadsAttention]
    assert [type(b.feed_forward) for b in d.blocks] == [ExpertsMLP, GatedMLP, ExpertsMLP, type(None), ExpertsMLP]
    m = d.blocks[0].mixer
    assert (m.n_heads, m.dim, m.vdim, m.gate_cap) == (3, 16, 24, 10.0)
    a = d.blocks[2].mixer
    assert (a.n_heads, a.n_kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.window, a.keep_first, a.rot_dims, a.rot_base) == \
        (4, 2, 16, 24, 0.3, 15.0, 37, 5, 16, 500.0)
    assert a.qk_norm and not a.has_talk and not a.has_bias and not a.interleaved and a.rot_scaling["original"] == 96
    # the first layer that mixes values gives its own, the others take them
    assert [b.mixer.value_mix for b in d.blocks if isinstance(b.mixer, TalkingHeadsAttention)] == [None, "first", "mix"]
    e = d.blocks[0].feed_forward
    assert (e.inner, e.n_experts, e.top, e.table_vocab, e.router, e.shared.inner) == (24, 5, 2, 96, None, 40)
    assert d.blocks[2].feed_forward.shared is None
    b = describe(CONFIG_B)
    assert b.head.softcap == 0.0 and b.blocks[0].mixer.window is None and b.blocks[0].mixer.softcap == 0.0
    assert b.blocks[0].mixer.rot_dims == 0 and b.blocks[2].mixer.keep_first == 21
    assert all(p.all_replayable() for p in d.parts())


def test_tensor_names_and_shapes():
    d = describe(CONFIG_A)
    specs = {s.name: tuple(s.shape) for s in d.param_specs()}
    D = 64
    assert specs["embed"] == specs["head"] == (96, D) and specs["final.norm"] == specs["l0.norm1"] == specs["l0.norm2"] == (D,)
    assert specs["l0.mix.q"] == specs["l0.mix.k"] == (48, D) and specs["l0.mix.v"] == specs["l0.mix.g"] == (72, D)
    assert specs["l0.mix.i"] == specs["l0.mix.f"] == (3, D) and specs["l0.mix.i.b"] == specs["l0.mix.f.b"] == (3,)
    assert specs["l0.mix.norm"] == (72,) and specs["l0.mix.o"] == (D, 72)
    assert specs["l1.mix.q"] == (64, D) and specs["l1.mix.k"] == (32, D) and specs["l1.mix.v"] == (80, D) and specs["l1.mix.o"] == (D, 160)
    assert specs["l1.mix.q.norm"] == (64,) and specs["l1.mix.k.norm"] == (32,) and "l1.mix.vmix" not in specs
    assert specs["l2.mix.vmix"] == specs["l4.mix.vmix"] == ()
    assert specs["l0.mlp.table"] == (96, 2) and specs["l0.mlp.e4.gate"] == specs["l0.mlp.e0.up"] == (24, D) and specs["l0.mlp.e2.down"] == (D, 24)
    assert specs["l0.mlp.shared.gate"] == specs["l0.mlp.shared.up"] == (40, D) and specs["l0.mlp.shared.down"] == (D, 40)
    assert specs["l1.mlp.gate"] == (72, D) and "l2.mlp.shared.gate" not in specs and "l3.norm2" not in specs and "l0.mlp.router" not in specs
    w = random_tensors(d, 3)
    check_tensors(d, w)
    assert w["l4.mlp.table"].dtype == torch.int32
    for k, n in (("l0.mlp.table", 5), ("l4.mlp.table", 4)):         # rows of different experts
        t = w[k].long()
        assert 0 <= int(t.min()) and int(t.max()) < n and all(len(set(r)) == t.shape[1] for r in t.tolist())
    with pytest.raises(WeightError, match="l3.norm2"):
        check_tensors(d, dict(w, **{"l3.norm2": torch.ones(D)}))


def test_caches():
    d = describe(CONFIG_A)
    specs = d.cache_specs()
    assert specs[(0, "memory")] == StateSpec((3, 25, 16)) and specs[(0, "max")] == StateSpec((3,))
    assert specs[(3, "memory")] == StateSpec((2, 17, 40)) and specs[(3, "max")] == StateSpec((2,))
    assert specs[1] == PagedKVSpec(2, 16, 37, value_dim=40, keep_first=5) and specs[2] == PagedKVSpec(2, 16, 37, value_dim=24, keep_first=5)
    assert specs[4] == PagedKVSpec(2, 16, 50, value_dim=24, keep_first=2)
    m = CacheManager(specs, page_size=16, n_pages=9, max_requests=2, max_len=128, dtype=torch.float32, device="cpu")
    slot = m.add_request("a")
    for grp in m.state_groups:
        grp.data[:, slot] = 7.0
    m.reserve("a", 120)
    m.commit("a")
    # the page of the kept positions, and what the window of 37 (or 50) before position 120 touches: pages 5 .. 7, or 4 .. 7
    assert sorted(m.pages_in_use()) == [4, 4, 5]
    m.check()
    m.release("a")
    assert m.add_request("b") == slot and all(float(grp.data[:, slot].abs().max()) == 0.0 for grp in m.state_groups)
    b = describe(CONFIG_B).cache_specs()
    assert b[0].window is None and b[2] == PagedKVSpec(6, 32, 3, value_dim=8, keep_first=21)


def test_configuration_errors():
    bad = lambda edit: (lambda c: (edit(c), c)[1])(copy.deepcopy(CONFIG_A))
    cases = [
        lambda c: c["layers"][0].update(type="retention"),
        lambda c: c["layers"][0]["mixer"].pop("gate_cap"),
        lambda c: c["layers"][0]["mixer"].update(gate_cap=0),
        lambda c: c["layers"][0]["mixer"].update(dim=600),
        lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
        lambda c: c["layers"][1]["mixer"].pop("scale"),
        lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
        lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18),
        lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("low"),
        lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
        lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1),
        lambda c: c["layers"][4]["mixer"].update(vdim=32),
        lambda c: c["layers"][0]["mlp"].update(kind="mixture"),
        lambda c: c["layers"][0]["mlp"]["router"].update(top=6),
        lambda c: c["layers"][0]["mlp"].pop("expert"),
        lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"),
        lambda c: c["layers"][1]["mlp"].update(ff=0),
        lambda c: c["embedding"].pop("scale"),
        lambda c: c.pop("norm"),
        lambda c: c.update(width=0),
        lambda c: c.update(layers=[]),
    ]
    for i, edit in enumerate(cases):
        with pytest.raises(ConfigError):
            describe(bad(edit))
            pytest.fail(f"case {i} was accepted")
    for config in ALL.values():
        describe(config)


def test_a_table_that_names_no_expert_is_refused():
    d = describe(ONLY_EXPERTS)
    w = random_tensors(d, 1)
    ff = d.blocks[0].feed_forward
    w["l0.mlp.table"][3, 0] = 6
    with pytest.raises(ValueError, match="outside 0 .. 5"):
        ff.bind(w, torch.float32, "cpu")


def test_random_weights_give_a_working_plain_model():
    for config in (CONFIG_A, CONFIG_B, CONFIG_ODD):
        w = random_tensors(describe(config), 3, torch.bfloat16)
        toks = list(range(20))
        after, logits = plain.layers(config, w, toks)
        assert after.shape == (len(config["layers"]), 20, config["width"]) and torch.isfinite(logits).all()
        # causal: a later token does not move earlier logits
        again_ = plain.forward(config, w, toks[:12] + [7] * 8)
        assert float((again_[:12] - logits[:12]).abs().max()) < 1e-9


def test_frequencies_by_wavelength():
    """Short wavelengths keep their frequency, long ones are stretched, those between are blended; the framework's table and
    the plain one agree."""
    rot = {"dims": 64, "base": 10000.0, "scaling": {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 700}}
    f = plain.frequencies(dict(rot, scaling=None))
    got = plain.frequencies(rot)
    length = 2 * math.pi / f
    short, long_ = length < 700 / 5.0, length > 700 / 1.5
    assert bool(short.any()) and bool(long_.any()) and bool((~short & ~long_).any())
    assert torch.equal(got[short], f[short]) and torch.allclose(got[long_], f[long_] / 6.0)
    mid = ~short & ~long_
    assert bool((got[mid] < f[mid]).all()) and bool((got[mid] > f[mid] / 6.0).all())
    for r in (rot, {"dims": 10, "base": 50.0, "scaling": {"factor": 3.0, "low": 2.0, "high": 2.0, "original": 40}},
              {"dims": 6, "base": 1e6, "scaling": {"factor": 1.0, "low": 0.5, "high": 7.0, "original": 1000}}):
        mine, factor = rotation_frequencies(r["dims"], r["base"], r["scaling"])
        assert factor == 1.0
        if r["scaling"]["low"] != r["scaling"]["high"]:
            assert torch.allclose(torch.tensor(mine, dtype=torch.float64), plain.frequencies(r), rtol=1e-12)
    plain_, one = rotation_frequencies(64, 10000.0)
    assert one == 1.0 and torch.allclose(torch.tensor(plain_, dtype=torch.float64), f)


def test_plain_mechanisms():
    """The plain functions on inputs whose results can be written down."""
    # a memory of one number: m starts at 0, not at minus infinity, so a weak first input is divided by exp(-0) = 1
    q = k = torch.ones(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([5.0, 7.0], dtype=torch.float64).view(2, 1, 1)
    i = torch.tensor([[-2.0], [1.0]], dtype=torch.float64)
    f = torch.tensor([[-0.5], [-0.25]], dtype=torch.float64)
    o = plain.matrix_memory(q, k, v, i, f)[:, 0, 0]
    m1 = max(-0.5, -2.0)
    take = math.exp(-2.0 - m1)
    S, n = take * 5.0, take
    want = [S / (max(n, math.exp(-m1)) + 1e-6)]
    m2 = max(-0.25 + m1, 1.0)
    keep, take = math.exp(-0.25 + m1 - m2), math.exp(1.0 - m2)
    S, n = keep * S + take * 7.0, keep * n + take
    want.append(S / (max(n, math.exp(-m2)) + 1e-6))
    assert torch.allclose(o, torch.tensor(want, dtype=torch.float64), atol=1e-12)
    # windows and kept first positions
    seen = plain.visible(6, {"size": 2, "keep_first": 1})
    assert seen.int().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0],
                                   [1, 0, 0, 0, 1, 1]]
    # a rotation of pairs (i, i + 1) of a head of three by one radian at position 1
    x = torch.tensor([[[1.0, 2.0, 9.0]], [[1.0, 2.0, 9.0]]], dtype=torch.float64)
    t = plain.turn(x, {"dims": 2, "base": 10.0})
    assert t[0, 0].tolist() == [1.0, 2.0, 9.0]
    assert torch.allclose(t[1, 0], torch.tensor([math.cos(1) - 2 * math.sin(1), 2 * math.cos(1) + math.sin(1), 9.0], dtype=torch.float64))
    assert plain.mix_values(1.0, 3.0, 0.25) == 1.5
    assert float(plain.soft_cap(torch.tensor(1e9), 4.0)) == 4.0 and float(plain.soft_cap(torch.tensor(3.0), None)) == 3.0
    # experts out of a table, each with weight 1 / top
    w = {"n.table": torch.tensor([[1, 0], [2, 1]], dtype=torch.int32)}
    for e in range(3):
        w.update({f"n.e{e}.gate": torch.full((1, 1), 1.0), f"n.e{e}.up": torch.full((1, 1), 10.0 ** e), f"n.e{e}.down": torch.ones(1, 1)})
    h = torch.ones(2, 1, dtype=torch.float64)
    y = plain.experts_by_token(h, torch.tensor([1, 0]), w, "n", 2)[:, 0] / float(plain.silu(torch.tensor(1.0, dtype=torch.float64)))
    assert torch.allclose(y, torch.tensor([55.0, 5.5], dtype=torch.float64))
