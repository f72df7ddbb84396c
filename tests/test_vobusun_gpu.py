"""Vobusun through the engine against the plain implementation (tests/plain_vobusun.py): whole prompts, prefill against
token-by-token decoding, portions down to two tokens, mixed batches with pages and slots that are used again, each mechanism
alone, weights made so that a lost key, a window that is one token off, a lost state or a wrong pair of tokens would show,
layers that run another layer's weights, long decoding, sizes that differ in every place, and greedy generation through
the entry points."""
import copy

import pytest
import torch

import plain_vobusun as plain
from helpers import Trace, max_live_tokens, mixed_schedule, run_trace
from lelatar_cases import run_engine, tokens, worst
from vobusun_cases import (ALL, CONFIG_A, CONFIG_B, FF, ONLY_RETENTION, ONLY_RGLRU, again, latent, loud_layers, make_dir, model,
                           retention, rglru, sharpen)

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
# Largest |difference| as a fraction of max(1, largest |logit| of the row).  float32: sums in another order.
# bfloat16: the rounding of every product's inputs, through up to six layers (measured: 0.003 to 0.06); a window that is
# one position off moves the sharpened models' logits by 0.15 of that scale and more.
TOL = {"float32": 2e-5, "bfloat16": 0.08}


def reference(config, weights, requests):
    return {name: plain.forward(config, weights, toks, dtype=torch.float64).float() for name, toks in requests.items()}


def load(path, dtype):
    from mlx_lm_b200.weights import load_model
    return load_model(str(path), dtype=dtype)[0]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALL))
def test_whole_prompts(name, dtype, tmp_path):
    """One step per prompt, all logits: also the first tokens of a sequence (lengths 1, 2, 3: shorter than the convolutions'
    taps, no token before the first), and runs of more than one tile of 128 rows."""
    config = ALL[name]
    weights = make_dir(tmp_path, config, seed=11)
    reqs = {f"r{n}": tokens(n, config["vocab"], n) for n in (1, 2, 3, 37, 150, 260)}
    tr = Trace()
    for rid, toks in reqs.items():
        tr.whole(rid, toks)
    got = run_engine(load(tmp_path, dtype), tr)
    w = worst(got, reference(config, weights, reqs))
    print(f"whole {name} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALL))
def test_every_cutting_gives_the_same_logits(name, dtype, tmp_path):
    """Prefill then 40 tokens one by one; portions of many sizes (two tokens, one, sizes around 16, 32, 64 and 128 rows: cuts
    inside the convolutions' taps, inside pages and tiles); mixed batches of unequal requests in a pool with three slots and
    few pages, so that both are used again by later requests."""
    config = ALL[name]
    weights = make_dir(tmp_path, config, seed=5)
    V = config["vocab"]
    reqs = {"a": tokens(70, V, 1), "b": tokens(131, V, 2), "c": tokens(23, V, 3), "d": tokens(300, V, 4), "e": tokens(5, V, 5)}
    tr = Trace()
    for rid, toks in reqs.items():
        tr.bulk_then_single(f"{rid}:tail", toks, tail=40)
    for rid, toks in reqs.items():
        tr.portions(f"{rid}:portions", toks, sizes=(2, 1, 15, 2, 16, 17, 3, 33, 2, 37, 64, 2, 130, 1, 31))
    mixed_schedule(tr, [(f"{rid}:mixed", toks) for rid, toks in reqs.items()], seed=1, max_live=3)
    mixed_schedule(tr, [(f"{rid}:mixed2", toks) for rid, toks in reversed(list(reqs.items()))], seed=2, max_live=3,
                   sizes=(2, 1, 1, 48, 1, 16, 1, 2, 37, 1, 1, 9, 130, 1))
    pool = max_live_tokens(tr, round_to=16)
    got = run_engine(load(tmp_path, dtype), tr, page_size=16, n_pages=pool // 16, max_requests=3, max_len=512)
    assert len(got) == 4 * sum(len(t) for t in reqs.values())
    w = worst(got, reference(config, weights, reqs))
    print(f"cuttings {name} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 16, 40, 63, 64, 65, 130])
def test_window_edges(window, dtype, tmp_path):
    """Sharp attention: the plain model with a window one position longer or shorter gives other logits, the engine gives
    those of the window itself, in whole prompts, in portions that end at and next to the edges, and in decoding."""
    config = model(64, 48, [latent(dim=16, heads=4, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scale=0.25, window=window)], streams=2)
    weights = make_dir(tmp_path, config, seed=22, edit=lambda w: sharpen(w, 6.0))
    reqs = {"a": tokens(300, 64, 31), "b": tokens(200, 64, 32)}
    ref = reference(config, weights, reqs)
    for other in (window - 1, window + 1):
        if other > 0:
            wrong = copy.deepcopy(config)
            wrong["layers"][0]["mixer"]["mask"]["size"] = other
            assert float((plain.forward(wrong, weights, reqs["a"]).float() - ref["a"]).abs().max()) > 0.3
    tr = Trace()
    tr.whole("a:0", reqs["a"])
    tr.portions("a:1", reqs["a"], sizes=(window, 1, 2, 126, 16, 15, 1, 112))
    tr.portions("b:1", reqs["b"], sizes=(window + 1, max(window - 1, 1), 2, 2))
    tr.bulk_then_single("b:2", reqs["b"], tail=2 * window + 3 if window < 64 else 80)
    got = run_engine(load(tmp_path, dtype), tr)
    w = worst(got, ref)
    print(f"window {window} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["retention", "rglru"])
def test_far_tokens_stay_in_the_state(case, dtype, tmp_path):
    """Heads and channels that hardly forget: one loud token at the start moves the logits hundreds of positions later; a
    state that is lost between portions, at a tile's border or between prefill and decoding would show."""
    config = {"retention": ONLY_RETENTION, "rglru": ONLY_RGLRU}[case]
    V = config["vocab"]

    def edit(w):
        w["embed"][0] *= 30.0                         # token 0 stands out ...
        w["bigram"] *= 0.0
        for k in w:
            if k.endswith(".lam"):
                w[k] = torch.full_like(w[k], -7.5)    # ... and is remembered
            elif k.endswith(".mix.v") or k.endswith(".mix.x"):
                w[k] += 8.0 * torch.outer(torch.sign(torch.randn(w[k].shape[0], generator=torch.Generator().manual_seed(1))),
                                          w["embed"][0] / w["embed"][0].norm() / w[k].shape[1] ** 0.5)
    weights = make_dir(tmp_path, config, seed=4, edit=edit)
    body = [t or 1 for t in tokens(420, V, 5)]
    reqs = {"with": [0] + body, "without": [1] + body}
    ref = reference(config, weights, reqs)
    assert float((ref["with"][-20:] - ref["without"][-20:]).abs().max()) > 0.1
    tr = Trace()
    for rid, toks in reqs.items():
        tr.whole(f"{rid}:0", toks)
        tr.portions(f"{rid}:1", toks, sizes=(127, 1, 2, 126, 16, 15, 1, 112))
        tr.bulk_then_single(f"{rid}:2", toks, tail=200)
    got = run_engine(load(tmp_path, dtype), tr)
    w = worst(got, ref)
    print(f"far tokens {case} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


def test_each_mechanism_matters_and_is_there(tmp_path):
    """The plain model without a mechanism, or with one of its constants changed, gives other logits; the engine gives those
    of the full one."""
    config = CONFIG_A
    weights = make_dir(tmp_path, config, seed=3, edit=lambda w: sharpen(w, 4.0))
    toks = tokens(60, config["vocab"], 1)
    ref = reference(config, weights, {"a": toks})
    differs = lambda logits: float((logits.float() - ref["a"]).abs().max())
    w64 = {k: v.double() for k, v in weights.items()}
    for name, value in (("bigram", 0.0), ("embed.norm", 1.0), ("l1.mix.dq.norm", 1.0), ("l1.mix.dkv.norm", 1.0), ("l1.mix.g", 0.0),
                        ("l2.mix.conv", 0.25), ("l2.mix.conv.b", 0.0), ("l2.mix.y.b", 0.0), ("l2.mix.x.b", 0.0), ("l2.mix.ra", 0.0),
                        ("l2.mix.ra.b", 0.0), ("l2.mix.ri", 0.0), ("l2.mix.ri.b", 0.0), ("l2.mix.lam", 0.0), ("l0.mix.g", 1.0),
                        ("l1.hc1.in", 0.4), ("l0.hc2.out", 0.5), ("final.norm", 1.0)):
        changed = dict(w64)
        changed[name] = torch.full_like(w64[name], value)
        assert differs(plain.forward(config, changed, toks)) > 0.005, name
    turned = dict(w64)
    turned["l1.hc1.mix"] = w64["l1.hc1.mix"].T.contiguous()
    assert differs(plain.forward(config, turned, toks)) > 0.01

    def edited(path, value):
        c = copy.deepcopy(config)
        node = c
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        return c
    for path, value in ((("layers", 0, "mixer", "decay"), [0.7, 0.9375, 0.984375]), (("layers", 0, "mixer", "rot"), {"dims": 0, "base": 1.0}),
                        (("layers", 0, "mixer", "rot", "base"), 100.0), (("layers", 3, "mixer", "rot", "dims"), 38),
                        (("layers", 1, "mixer", "scale"), 0.1), (("layers", 1, "mixer", "mask", "size"), 36),
                        (("layers", 1, "mixer", "rot", "base"), 100.0), (("layers", 0, "mlp", "limit"), 100.0), (("layers", 2, "mlp", "limit"), 0.5),
                        (("embedding", "scale"), 1.0), (("embedding", "bigram", "mul_prev"), 18), (("embedding", "bigram", "mul_cur"), 4),
                        (("residual_mult",), 1.0), (("norm", "eps"), 0.1)):
        assert differs(plain.forward(edited(path, value), w64, toks)) > 0.005, path
    # the layers that run an earlier layer's weights have caches of their own
    once = copy.deepcopy(config)
    once["layers"] = once["layers"][:-1]
    assert differs(plain.forward(once, w64, toks)) > 0.01
    tr = Trace()
    tr.whole("a:w", toks)
    tr.bulk_then_single("a:t", toks, tail=25)
    w = worst(run_engine(load(tmp_path, "float32"), tr), ref)
    assert w < TOL["float32"], w


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_that_are_used_again(dtype, tmp_path):
    """One slot and few pages: every request runs in the slot and the pages the one before left behind (its states, its
    convolutions' inputs and its last token are gone), and gives what it gives alone."""
    config = CONFIG_B
    weights = make_dir(tmp_path, config, seed=2)
    V = config["vocab"]
    a, b = tokens(120, V, 1), tokens(9, V, 2)
    ref = reference(config, weights, {"a": a, "b": b, "c": [3] + a})
    assert float((ref["c"][1:] - ref["a"]).abs().max()) > 0.05
    tr = Trace()
    tr.whole("a:1", a)
    tr.portions("b:1", b, sizes=(2, 1, 3))
    tr.whole("c:1", [3] + a)
    tr.bulk_then_single("a:2", a, tail=30)
    tr.bulk_then_single("b:2", b, tail=8)
    got = run_engine(load(tmp_path, dtype), tr, max_requests=1, n_pages=16)
    assert worst(got, ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype, tmp_path):
    """A short prompt and then 500 tokens one by one beside a second request that comes and goes."""
    config = CONFIG_A
    weights = make_dir(tmp_path, config, seed=8)
    V = config["vocab"]
    reqs = {"a": tokens(510, V, 1), "b": tokens(200, V, 2)}
    ref = reference(config, weights, reqs)
    tr = Trace()
    tr.step([("a", reqs["a"][:10], "all"), ("b", reqs["b"][:3], "all")])
    for t in range(10, 510):
        e = [("a", reqs["a"][t:t + 1], "all")]
        tb = t - 7
        if tb < 200:
            e.append(("b", reqs["b"][tb:tb + 1], "all"))
        tr.step(e, end=(["b"] if tb == 199 else []) + (["a"] if t == 509 else []))
    got = run_engine(load(tmp_path, dtype), tr, n_pages=48, max_requests=2, max_len=640)
    w = worst(got, ref)
    print(f"long decoding {dtype}: {w:.3g}")
    assert w < TOL[dtype]


def test_trace_replay_with_few_slots_and_pages(tmp_path):
    """The command-line replay on this design: mixed steps in a pool that forces pages and slots to be used again."""
    config = CONFIG_B
    weights = make_dir(tmp_path / "m", config, seed=13)
    V = config["vocab"]
    reqs = {f"r{i}": tokens(n, V, 40 + i) for i, n in enumerate((50, 3, 129, 64, 18, 77))}
    ref = reference(config, weights, reqs)
    tr = Trace()
    mixed_schedule(tr, list(reqs.items()), seed=5, max_live=4)
    for dtype in DTYPES:
        got = run_trace(str(tmp_path / "m"), tr, dtype, str(tmp_path / f"out-{dtype}"), extra=("--max-requests", "4"))
        w = worst(got, ref)
        print(f"replay {dtype}: {w:.3g}")
        assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_points(dtype, tmp_path):
    """``generate``, ``stream_generate`` and ``batch_generate`` (scheduler, decode graphs, device sampler; tokens handed from
    step to step on the device, the token before among them) give the plain model's greedy tokens."""
    from mlx_lm_b200 import batch_generate, generate, load, stream_generate
    config = CONFIG_A
    weights = make_dir(tmp_path, config, seed=24, edit=loud_layers)
    V = config["vocab"]
    prompts = [tokens(9, V, 1), tokens(21, V, 1), tokens(2, V, 2), tokens(1, V, 7)]

    def greedy(prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(plain.forward(config, weights, seq)[-1].argmax()))
        return seq[len(prompt):]

    def agrees(got, ref, prompt):
        for i, (a, b) in enumerate(zip(got, ref)):
            if a != b:
                lg = plain.forward(config, weights, prompt + ref[:i])[-1]
                top = torch.topk(lg, 2).values
                return dtype == "bfloat16" and float(top[0] - top[1]) < 0.05 * float(lg.abs().max())
        return len(got) == len(ref)

    want = [greedy(p, 40) for p in prompts]
    assert all(len(set(w)) >= 4 for w in want), want          # the model does not just repeat itself
    model_, tokenizer = load(str(tmp_path), dtype=dtype)
    for p, w in zip(prompts, want):
        got = [int(t) for t in generate(model_, tokenizer, p, max_tokens=40).split()]
        assert agrees(got, w, p), (got, w)
        streamed = [r.token for r in stream_generate(model_, tokenizer, p, max_tokens=40, prefill_step_size=5)]
        assert agrees(streamed, w, p), (streamed, w)
    out = batch_generate(model_, tokenizer, prompts, max_tokens=40, return_token_ids=True)
    for got, w, p in zip(out.token_ids, want, prompts):
        assert agrees(got, w, p), (got, w)


def test_command_line_and_sampling(tmp_path):
    """`python -m mlx_lm_b200 generate` on a model folder gives the Python entry point's tokens; the random-weights mode builds
    the design from a config.json alone; and what is drawn with a temperature does not depend on what else is in the batch."""
    import json
    import subprocess
    import sys
    from helpers import ROOT
    from mlx_lm_b200 import generate, load
    from mlx_lm_b200.generate import BatchGenerator
    from mlx_lm_b200.sampling import make_sampler
    config = CONFIG_B
    make_dir(tmp_path / "m", config, seed=31)
    model_, tokenizer = load(str(tmp_path / "m"), dtype="float32")
    want = generate(model_, tokenizer, [5, 17, 3], max_tokens=12)
    run = lambda *a: subprocess.run([sys.executable, "-m", "mlx_lm_b200", "generate", *a], cwd=ROOT, capture_output=True,
                                    text=True, timeout=300)
    r = run("--model", str(tmp_path / "m"), "--prompt", "5 17 3", "-m", "12", "--dtype", "float32", "--verbose", "F")
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == want.split()
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(config))
    r = run("--random-weights", "11", "--config", str(cfg), "--prompt", "5 17 3", "-m", "12", "--temp", "0.7",
            "--top-p", "0.9", "--min-p", "0.01", "--top-k", "20", "--seed", "4", "--verbose", "F")
    assert r.returncode == 0 and len(r.stdout.split()) == 12, r.stderr
    prompts = [tokens(n, config["vocab"], n) for n in (5, 31, 64)]

    def drawn(**kw):
        gen = BatchGenerator(model_, max_tokens=20, sampler=make_sampler(0.8, top_p=0.95), seed=1, **kw)
        uids = gen.insert(prompts)
        out = {u: [] for u in uids}
        while gen.scheduler.has_work():
            for resp in gen.next_generated():
                out[resp.uid].append(resp.token)
        return [out[u] for u in uids]
    together = drawn(completion_batch_size=8, prefill_batch_size=8)
    assert all(len(t) == 20 for t in together)
    assert drawn(completion_batch_size=1, prefill_batch_size=1) == together
    assert drawn(completion_batch_size=2, prefill_batch_size=1, prefill_step_size=7, max_tokens_per_step=9) == together


def drawn_config(seed):
    """A configuration drawn from sizes a small model might have: every layer with a mixer of its own sizes, some layers on
    another layer's weights, feed-forwards or none, any number of streams."""
    import random
    rng = random.Random(seed)
    width = rng.choice([64, 96, 128, 192])
    layers = []
    for i in range(rng.choice([2, 3, 4, 5])):
        own = [j for j, l in enumerate(layers) if "weights_of" not in l]
        if own and rng.random() < 0.3:
            layers.append(again(layers, rng.choice(own)))
            continue
        mlp = FF(rng.choice([16, 64, 96, 160]), rng.choice([0.8, 1.5, 7.0])) if rng.random() < 0.8 else None
        kind = rng.choice(["retention", "latent", "rglru"])
        heads = rng.choice([1, 2, 3, 4, 6, 8])
        if kind == "retention":
            dim = rng.choice([8, 16, 32, 48, 64, 96, 128])
            layers.append(retention(dim=dim, heads=heads, vdim=rng.choice([16, 32, 48, 64, 96, 128, 160]),
                                    decay=[round(1.0 - 0.5 ** rng.uniform(2.0, 10.0), 6) for _ in range(heads)],
                                    rot=(rng.choice([d for d in (2, 8, 16, 32, 48, 64, 128) if d <= dim]), rng.choice([100.0, 10000.0, 1e6])), mlp=mlp))
        elif kind == "latent":
            layers.append(latent(dim=rng.choice([16, 32, 64]), heads=heads, rot_dim=rng.choice([8, 16, 32]), vdim=rng.choice([16, 32, 80]),
                                 q_rank=rng.choice([24, 64, 136]), kv_rank=rng.choice([24, 64, 96, 160]), scale=rng.choice([0.09, 0.125, 0.25]),
                                 base=rng.choice([100.0, 10000.0, 250000.0]), window=rng.choice([5, 33, 100, 1000]), mlp=mlp))
        else:
            blocks = rng.choice([1, 2, 4])
            layers.append(rglru(width=blocks * rng.choice([16, 24, 48, 64]), blocks=blocks, conv=rng.choice([1, 2, 3, 4, 7]), mlp=mlp))
    return model(rng.choice([100, 256, 576]), width, layers, streams=rng.choice([1, 2, 3, 4, 6, 8]), mult=rng.choice([0.3, 0.5, 1.0]),
                 scale=rng.choice([0.5, 1.0, 8.0]), bigram=rng.choice([(31, 7, 3), (1009, 131, 17), (257, 1, 1)]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_drawn_configurations(seed, dtype, tmp_path):
    """Whole prompts (one of several tiles), prefill and decoding, portions and a mixed batch, for configurations nobody
    picked by hand."""
    config = drawn_config(seed)
    weights = make_dir(tmp_path, config, seed=seed)
    V = config["vocab"]
    reqs = {"a": tokens(600, V, 1), "b": tokens(131, V, 2), "c": tokens(1, V, 3), "d": tokens(77, V, 4)}
    tr = Trace()
    for rid, toks in reqs.items():
        tr.whole(f"{rid}:whole", toks)
    tr.bulk_then_single("b:tail", reqs["b"], tail=40)
    tr.portions("a:portions", reqs["a"], sizes=(2, 129, 1, 64, 3, 200, 17))
    mixed_schedule(tr, [(f"{rid}:mixed", toks) for rid, toks in reqs.items()], seed=seed, max_live=3)
    pool = max_live_tokens(tr, round_to=64)
    got = run_engine(load(tmp_path, dtype), tr, page_size=16, n_pages=pool // 16, max_requests=3, max_len=1024)
    w = worst(got, reference(config, weights, reqs))
    print(f"drawn {seed} {dtype}: {w:.3g}")
    assert w < TOL[dtype]
