"""Vobusun on the CPU: the configuration reader, the parts it picks, tensor names, the caches (also the embedding's, and
those of layers that run another layer's weights), and the plain implementation's own mechanisms."""
import copy
import math

import pytest
import torch

import plain_vobusun as plain
from vobusun_cases import ALL, CONFIG_A, CONFIG_B, CONFIG_ODD, FF, PLAIN_RESIDUAL, latent, model, retention, rglru
from mlx_lm_b200.cache import CacheManager
from mlx_lm_b200.config import ConfigError, get_architecture
from mlx_lm_b200.parts import (EMBEDDING_CACHE, GatedMLP, HyperBlock, LatentAttention, PagedKVSpec, RetentionMixer, RGLRUMixer,
                               RMSNorm, StateSpec, StreamsNorm, TokenPairEmbedding)
from mlx_lm_b200.weights.loader import WeightError, check_tensors, random_tensors


def describe(config):
    arch = get_architecture(config)
    return arch.build(arch.args_class.from_dict(copy.deepcopy(config)))


def test_found_by_its_architecture_key_and_parts_follow_the_layer_list():
    d = describe(CONFIG_A)
    assert d.model_type == "vobusun" and d.position is None and d.head.tied_to is None
    assert all(isinstance(b, HyperBlock) and isinstance(b.norm_1, RMSNorm) and b.n_streams == 3 and b.learned for b in d.blocks)
    assert [type(b.mixer) for b in d.blocks] == [RetentionMixer, LatentAttention, RGLRUMixer, RetentionMixer]
    assert [type(b.feed_forward) for b in d.blocks] == [GatedMLP, GatedMLP, GatedMLP, type(None)]
    assert all(b.residual_scale == 0.35 for b in d.blocks)
    f = d.blocks[1].feed_forward
    assert (f.inner, f.unit, f.limit) == (72, "bounded", 0.7)
    e = d.embedding
    assert isinstance(e, TokenPairEmbedding) and (e.scale, e.buckets, e.mul_prev, e.mul_cur, e.n_streams) == (4.0, 211, 17, 5, 3)
    assert isinstance(d.final_norm, StreamsNorm) and d.final_norm.n_streams == 3
    r = d.blocks[0].mixer
    assert (r.n_heads, r.dim, r.vdim, r.rot_dims, r.rot_base) == (3, 16, 24, 8, 1000.0) and r.decay_list == [0.75, 0.9375, 0.984375]
    m = d.blocks[1].mixer
    assert (m.n_heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.rank, m.window, m.head_gate, m.interleaved) == (4, 16, 8, 24, 40, 32, 37, True, True)
    u = d.blocks[2].mixer
    assert (u.inner, u.blocks, u.block, u.taps) == (48, 3, 16, 4)
    # the last two layers run blocks 1 and 2 again with caches of their own
    assert [(x.block, x.write) for x in d.runs()] == [(0, True), (1, True), (2, True), (3, True), (1, True), (2, True)]
    assert len({x.cache_id for x in d.runs()}) == 6
    # in B the layer with the tensors comes after one of its copies
    assert [x.block for x in describe(CONFIG_B).runs()] == [1, 0, 1, 2, 1]


def test_tensor_names_and_shapes():
    d = describe(CONFIG_A)
    specs = {s.name: tuple(s.shape) for s in d.param_specs()}
    D = 64
    assert specs["embed"] == (96, D) and specs["bigram"] == (212, D) and specs["embed.norm"] == specs["final.norm"] == (D,)
    assert specs["head"] == (96, D)
    assert specs["l0.mix.q"] == specs["l0.mix.k"] == (48, D) and specs["l0.mix.v"] == specs["l0.mix.g"] == (72, D)
    assert specs["l0.mix.o"] == (D, 72) and "l0.mix.decay" not in specs
    assert specs["l1.mix.dq"] == (40, D) and specs["l1.mix.dq.norm"] == (40,) and specs["l1.mix.uq"] == (4 * 24, 40)
    assert specs["l1.mix.dkv"] == (40, D) and specs["l1.mix.dkv.norm"] == (32,) and specs["l1.mix.g"] == (4, D)
    assert specs["l1.mix.uk"] == (64, 32) and specs["l1.mix.uv"] == (96, 32) and specs["l1.mix.o"] == (D, 96)
    assert "l1.mix.q" not in specs
    assert specs["l2.mix.y"] == specs["l2.mix.x"] == (48, D) and specs["l2.mix.y.b"] == specs["l2.mix.x.b"] == (48,)
    assert specs["l2.mix.conv"] == (48, 4) and specs["l2.mix.conv.b"] == specs["l2.mix.lam"] == (48,)
    assert specs["l2.mix.ra"] == specs["l2.mix.ri"] == (3, 16, 16) and specs["l2.mix.ra.b"] == specs["l2.mix.ri.b"] == (3, 16)
    assert specs["l2.mix.o"] == (D, 48)
    assert specs["l0.mlp.gate"] == specs["l0.mlp.up"] == (40, D) and specs["l0.mlp.down"] == (D, 40)
    assert specs["l0.hc1.in"] == specs["l0.hc2.out"] == (3,) and specs["l0.hc2.mix"] == (3, 3)
    assert "l3.norm2" not in specs and "l3.hc2.in" not in specs and "l3.hc1.mix" in specs
    assert not any(k.startswith(("l4.", "l5.")) for k in specs)
    w = random_tensors(d, 3)
    check_tensors(d, w)
    with pytest.raises(WeightError, match="l4.norm1"):
        check_tensors(d, dict(w, **{"l4.norm1": torch.ones(D)}))
    none = {s.name for s in describe(PLAIN_RESIDUAL).param_specs()}
    assert not any(".hc" in k for k in none) and "bigram" not in none and "embed.norm" in none


def test_caches():
    d = describe(CONFIG_A)
    specs = d.cache_specs()
    ids = [x.cache_id for x in d.runs()]
    assert specs[EMBEDDING_CACHE] == StateSpec((1,))
    assert specs[ids[0]] == StateSpec((3, 24, 16)) and specs[ids[3]] == StateSpec((2, 16, 40))
    kv = PagedKVSpec(1, 40, 37, value_dim=0)
    assert specs[ids[1]] == specs[ids[4]] == kv
    assert specs[(ids[2], "unit")] == specs[(ids[5], "unit")] == StateSpec((48,))
    assert specs[(ids[2], "conv")] == specs[(ids[5], "conv")] == StateSpec((3, 48))
    m = CacheManager(specs, page_size=16, n_pages=6, max_requests=2, max_len=64, dtype=torch.float32, device="cpu")
    g = m.kv_groups[m.where(ids[1])[1]]
    assert g.k.shape == (2, 6, 1, 16, 40) and g.v is g.k
    assert m.state_groups[m.where(EMBEDDING_CACHE)[1]].data.shape == (1, 2, 1)
    # a window's pages are given back, a new request finds its state slot empty
    slot = m.add_request("a")
    for grp in m.state_groups:
        grp.data[:, slot] = 7.0
    m.reserve("a", 60)
    m.commit("a")
    assert m.pages_in_use() == [3]                   # positions 24 .. 59 stay readable: pages 1 .. 3
    m.check()
    m.release("a")
    assert m.add_request("b") == slot and all(float(grp.data[:, slot].abs().max()) == 0.0 for grp in m.state_groups)
    # a convolution of one tap keeps nothing, and an embedding without pairs has no state
    one = describe(PLAIN_RESIDUAL).cache_specs()
    assert EMBEDDING_CACHE not in one and (0, "conv") not in one and one[(0, "unit")] == StateSpec((32,))


def test_configuration_errors():
    bad = lambda edit: (lambda c: (edit(c), c)[1])(copy.deepcopy(CONFIG_A))
    cases = [
        lambda c: c["layers"][0].update(type="wkv"),
        lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5]),
        lambda c: c["layers"][0]["mixer"].pop("decay"),
        lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
        lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
        lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6),
        lambda c: c["layers"][1]["mixer"].pop("q_rank"),
        lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
        lambda c: c["layers"][2]["mixer"].update(blocks=5),
        lambda c: c["layers"][2]["mixer"].update(conv=0),
        lambda c: c["layers"][4].update(weights_of=4),
        lambda c: c["layers"][4].update(weights_of=9),
        lambda c: c["layers"][3].update(weights_of=5),
        lambda c: c["layers"][4]["mixer"].update(scale=0.5),
        lambda c: c["layers"][0]["mlp"].update(kind="moe"),
        lambda c: c["layers"][0]["mlp"].pop("limit"),
        lambda c: c["embedding"]["bigram"].pop("mul_cur"),
        lambda c: c["embedding"]["bigram"].update(buckets=0),
        lambda c: c["embedding"].pop("scale"),
        lambda c: c.update(streams=0),
        lambda c: c.pop("norm"),
        lambda c: c.update(width=0),
    ]
    for i, edit in enumerate(cases):
        with pytest.raises(ConfigError):
            describe(bad(edit))
            pytest.fail(f"case {i} was accepted")
    for config in ALL.values():
        describe(config)


def test_random_weights_give_a_working_plain_model():
    for config in (CONFIG_A, CONFIG_B, CONFIG_ODD):
        w = {k: v.float() for k, v in random_tensors(describe(config), 3, torch.bfloat16).items()}
        toks = list(range(20))
        after, logits = plain.layers(config, w, toks)
        assert after.shape == (len(config["layers"]), 20, config["width"]) and torch.isfinite(logits).all()
        # causal: a later token does not move earlier logits
        again_ = plain.forward(config, w, toks[:12] + [7] * 8)
        assert float((again_[:12] - logits[:12]).abs().max()) < 1e-9


def test_plain_mechanisms():
    """The plain functions on inputs whose results can be written down."""
    # two streams: each new one from both old ones, indexed [from, to]
    x = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]])
    y = torch.tensor([[100.0, 0.0]])
    new = plain.mix_streams(x, torch.tensor([[1.0, 3.0], [0.0, 2.0]]), torch.tensor([1.0, -1.0]), y, 0.5)
    assert new[0].tolist() == [[51.0, 2.0]] and new[1].tolist() == [[3.0 + 20.0 - 50.0, 6.0 + 40.0]]
    assert plain.read_streams(x, torch.tensor([2.0, 0.5])).tolist() == [[7.0, 14.0]]
    # pairs of tokens: the row of the pair, and the last row at the start
    cfg = {"embedding": {"scale": 0.0, "bigram": {"buckets": 7, "mul_prev": 3, "mul_cur": 5}}, "norm": {"eps": 0.0}}
    w = {"embed": torch.zeros(9, 1), "bigram": torch.arange(1.0, 9.0)[:, None], "embed.norm": torch.ones(1)}
    rows = plain.embedding(torch.tensor([4, 8, 8]), dict(w, bigram=torch.stack([torch.arange(8.0) + 1, torch.ones(8)], 1),
                                                         embed=torch.zeros(9, 2), **{"embed.norm": torch.ones(2)}), cfg, torch.float64)
    ratio = (rows[:, 0] / rows[:, 1]).round().long().tolist()
    assert ratio == [8, (4 * 3 + 8 * 5) % 7 + 1, (8 * 3 + 8 * 5) % 7 + 1]
    # a rotation of pairs (i, i + 1) of a head of three by a quarter turn at position 1
    cos, sin = torch.tensor([[1.0], [0.0]]), torch.tensor([[0.0], [1.0]])
    v = torch.tensor([[[1.0, 2.0, 9.0]], [[1.0, 2.0, 9.0]]])
    assert plain.turn_halves(v, cos, sin, 2)[1].tolist() == [[-2.0, 1.0, 9.0]]
    # a recurrence written out: one channel, gates fixed by their biases
    name, big = "u", 50.0
    ident = {f"{name}.y": torch.ones(1, 1), f"{name}.y.b": torch.zeros(1), f"{name}.x": torch.ones(1, 1), f"{name}.x.b": torch.zeros(1),
             f"{name}.conv": torch.tensor([[0.0, 1.0]]), f"{name}.conv.b": torch.zeros(1), f"{name}.ra": torch.zeros(1, 1, 1),
             f"{name}.ri": torch.zeros(1, 1, 1), f"{name}.ra.b": torch.full((1, 1), big), f"{name}.ri.b": torch.full((1, 1), big),
             f"{name}.lam": torch.tensor([math.log(math.expm1(0.01))]), f"{name}.o": torch.ones(1, 1)}
    h = torch.tensor([[1.0], [2.0]], dtype=torch.float64)
    out = plain.rglru(h, ident, name, {"width": 1}, 1e-5)
    a = math.exp(-0.08)
    b = math.sqrt(1 - a * a)
    gelu = plain.gelu_tanh(torch.tensor([1.0, 2.0], dtype=torch.float64))
    want = torch.tensor([b * 1.0, a * b * 1.0 + b * 2.0], dtype=torch.float64) * gelu
    assert torch.allclose(out[:, 0], want, atol=1e-6)
