"""Fisesun through the engine against the plain implementation (tests/plain_fisesun.py): whole prompts, prefill against
token-by-token decoding, portions down to two tokens, mixed batches with pages and slots that are used again, each mechanism
alone, weights made so that a lost key, a window or a kept position that is one off, a lost state or a wrong expert would show,
long decoding, sizes that differ in every place, and greedy generation through the entry points."""
import copy

import pytest
import torch

import plain_fisesun as plain
from fisesun_cases import (ALL, CONFIG_A, CONFIG_B, FF, MOE, ONLY_MLSTM, attention, loud_layers, make_dir, mlstm, model, sharpen)
from helpers import Trace, max_live_tokens, mixed_schedule, run_trace
from lelatar_cases import run_engine, tokens, worst

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
# Largest |difference| as a fraction of max(1, largest |logit| of the row).  float32: sums in another order.
# bfloat16: the rounding of every product's inputs, through up to five layers (measured: 0.004 to 0.031); a window that is one position off moves the
# sharpened models' logits several times as far.
TOL = {"float32": 2e-5, "bfloat16": 0.05}


def reference(config, weights, requests):
    return {name: plain.forward(config, weights, toks, dtype=torch.float64).float() for name, toks in requests.items()}


def load(path, dtype):
    from mlx_lm_b200.weights import load_model
    return load_model(str(path), dtype=dtype)[0]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALL))
def test_whole_prompts(name, dtype, tmp_path):
    """One step per prompt, all logits: also the first tokens of a sequence (lengths 1, 2, 3), and runs of more than one tile of
    128 rows."""
    config = ALL[name]
    weights = make_dir(tmp_path, config, seed=11)
    reqs = {f"r{n}": tokens(n, config["vocab"], n) for n in (1, 2, 3, 37, 150, 260)}
    tr = Trace()
    for rid, toks in reqs.items():
        tr.whole(rid, toks)
    w = worst(run_engine(load(tmp_path, dtype), tr), reference(config, weights, reqs))
    print(f"whole {name} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALL))
def test_every_cutting_gives_the_same_logits(name, dtype, tmp_path):
    """Prefill then 40 tokens one by one; portions of many sizes (two tokens, one, sizes around 16, 32, 64 and 128 rows: cuts
    inside pages, windows and tiles); mixed batches of unequal requests in a pool with three slots and few pages, so that both
    are used again by later requests."""
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
@pytest.mark.parametrize("window,keep", [(1, 0), (2, 3), (16, 16), (40, 17), (63, 1), (64, 64), (65, 5), (130, 33), (20, 120)])
@pytest.mark.parametrize("heads", ["small", "64"])
def test_edges_of_windows_and_kept_positions(heads, window, keep, dtype, tmp_path):
    """Sharp attention: the plain model with a window one position longer or shorter, or one kept position more or fewer, gives
    other logits; the engine gives those of the design itself, in whole prompts, in portions that end at and next to the edges,
    and in decoding.  Heads of 64 over values of 64 take other kernels for portions."""
    size = dict(dim=16, heads=4, kv_heads=2, vdim=16, scale=0.25, rot=(8, 1000.0)) if heads == "small" \
        else dict(dim=64, heads=2, kv_heads=1, vdim=64, scale=0.125, rot=(32, 1000.0))
    config = model(64, 48, [attention(window=window, keep=keep, softcap=40.0, v_mix=False, **size)])
    # the layer speaks loudly, its rotation is slow enough for far keys to matter
    weights = make_dir(tmp_path, config, seed=22, edit=lambda w: (sharpen(w, 6.0), loud_layers(w, 8.0)))
    reqs = {"a": tokens(300, 64, 31), "b": tokens(240, 64, 32)}
    ref = reference(config, weights, reqs)
    for key, other in (("size", window - 1), ("size", window + 1), ("keep_first", keep - 1), ("keep_first", keep + 1)):
        if other > 0 or (other == 0 and key == "keep_first"):
            wrong = copy.deepcopy(config)
            wrong["layers"][0]["mixer"]["mask"][key] = other
            assert float((plain.forward(wrong, weights, reqs["a"]).float() - ref["a"]).abs().max()) > 0.3, (key, other)
    tr = Trace()
    tr.whole("a:0", reqs["a"])
    tr.portions("a:1", reqs["a"], sizes=(window, 1, 2, 126, 16, 15, 1, 112))
    tr.portions("b:1", reqs["b"], sizes=(window + 1, max(window - 1, 1), 2, 2, max(keep, 1), 2))
    tr.bulk_then_single("b:2", reqs["b"], tail=2 * window + 3 if window < 64 else 80)
    tr.bulk_then_single("b:3", reqs["b"], tail=239)
    w = worst(run_engine(load(tmp_path, dtype), tr), ref)
    print(f"window {window} keep {keep} {heads} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["memory", "kept"])
def test_far_tokens_are_remembered(case, dtype, tmp_path):
    """One loud token at the start moves the logits hundreds of positions later, through a memory that hardly forgets or through
    a kept first position far outside the window; a state that is lost between portions, at a tile's border or between prefill
    and decoding, or a kept page given back, would show."""
    config = ONLY_MLSTM if case == "memory" else model(64, 48, [attention(window=24, keep=1, softcap=30.0, v_mix=False, rot=None)])
    V = config["vocab"]

    def edit(w):
        loud_layers(w, 6.0)
        sharpen(w, 5.0)
        for k in w:
            if k.endswith(".mix.f.b"):
                w[k] = torch.full_like(w[k], 30.0)     # capped: the memory keeps nearly everything
            elif k.endswith(".mix.i") or k.endswith(".mix.f"):
                w[k] *= 0.3
        if case == "memory":
            w["embed"][0] *= 8.0
    weights = make_dir(tmp_path, config, seed=4, edit=edit)
    body = [t or 1 for t in tokens(420, V, 5)]
    reqs = {"with": [0] + body, "without": [1] + body}
    ref = reference(config, weights, reqs)
    assert float((ref["with"][-20:] - ref["without"][-20:]).abs().max()) > 0.3
    tr = Trace()
    for rid, toks in reqs.items():
        tr.whole(f"{rid}:0", toks)
        tr.portions(f"{rid}:1", toks, sizes=(127, 1, 2, 126, 16, 15, 1, 112))
        tr.bulk_then_single(f"{rid}:2", toks, tail=200)
    w = worst(run_engine(load(tmp_path, dtype), tr), ref)
    print(f"far tokens {case} {dtype}: {w:.3g}")
    assert w < TOL[dtype]


def test_each_mechanism_matters_and_is_there(tmp_path):
    """The plain model without a mechanism, or with one of its constants changed, gives other logits; the engine gives those
    of the full one."""
    config = CONFIG_A
    weights = make_dir(tmp_path, config, seed=3, edit=lambda w: (sharpen(w, 3.0), loud_layers(w, 2.0)))
    toks = tokens(60, config["vocab"], 1)
    ref = reference(config, weights, {"a": toks})
    differs = lambda logits: float((logits.float() - ref["a"]).abs().max())
    for name, value in (("l0.norm1", 0.5), ("l2.norm2", 0.5), ("final.norm", 1.0), ("l0.mix.i", 0.0), ("l0.mix.i.b", 0.0), ("l0.mix.f", 0.0),
                        ("l0.mix.f.b", 0.0), ("l0.mix.g", 0.0), ("l0.mix.norm", 1.0), ("l1.mix.q.norm", 1.0), ("l2.mix.k.norm", 1.0),
                        ("l4.mix.vmix", 0.0), ("l0.mlp.shared.down", 0.0), ("l4.mlp.shared.up", 0.0), ("l2.mlp.table", 1)):
        assert differs(plain.forward(config, dict(weights, **{name: torch.full_like(weights[name], value)}), toks)) > 0.01, name
    # the first layer that mixes values does not use its own number; an unmixed layer before it is not where they come from
    assert differs(plain.forward(config, dict(weights, **{"l2.mix.vmix": torch.tensor(0.9)}), toks)) < 1e-6
    rolled = dict(weights, **{"l0.mlp.table": weights["l0.mlp.table"].roll(1, dims=0)})
    assert differs(plain.forward(config, rolled, toks)) > 0.02

    def edited(path, value):
        c = copy.deepcopy(config)
        node = c
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        return c
    at = lambda i, *path: ("layers", i, "mixer") + path
    for path, value in ((at(0, "gate_cap"), 2.0), (at(3, "gate_cap"), 100.0), (at(1, "scale"), 0.2), (at(2, "softcap"), 5.0), (at(4, "softcap"), None),
                        (at(2, "mask", "size"), 36), (at(2, "mask", "keep_first"), 4), (at(1, "mask", "keep_first"), 0), (at(2, "rot", "scaling"), None),
                        (at(2, "rot", "scaling", "factor"), 2.0), (at(2, "rot", "scaling", "original"), 48), (at(2, "rot", "base"), 100.0),
                        (at(4, "rot", "dims"), 8), (at(4, "v_mix"), False), (at(1, "v_mix"), True), (("embedding", "scale"), 1.0),
                        (("logit_softcap",), None), (("norm", "eps"), 0.1)):
        w = dict(weights)
        if path == at(1, "v_mix"):       # (its values would be the ones that are mixed in: another width, so only their source moves)
            continue
        assert differs(plain.forward(edited(path, value), w, toks)) > 0.005, path
    tr = Trace()
    tr.whole("a:w", toks)
    tr.bulk_then_single("a:t", toks, tail=25)
    w = worst(run_engine(load(tmp_path, "float32"), tr), ref)
    assert w < TOL["float32"], w


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_that_are_used_again(dtype, tmp_path):
    """One slot and few pages: every request runs in the slot and the pages the one before left behind (its memories and maxima
    are gone), and gives what it gives alone."""
    config = CONFIG_B
    weights = make_dir(tmp_path, config, seed=2, edit=lambda w: loud_layers(w, 2.0))
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
    w = worst(got, ref)
    print(f"used again {dtype}: {w:.3g}")
    assert w < TOL[dtype]


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
    step to step on the device, where the tables of experts read them) give the plain model's greedy tokens."""
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
    """A configuration drawn from sizes a small model might have: every layer with a mixer and a feed-forward of its own sizes."""
    import random
    rng = random.Random(seed)
    width = rng.choice([64, 96, 128, 192])
    G, vdim = rng.choice([1, 2, 4]), rng.choice([16, 32, 48, 64, 128])
    layers = []
    for _ in range(rng.choice([2, 3, 4, 5])):
        r = rng.random()
        mlp = None if r < 0.15 else FF(rng.choice([16, 64, 96, 160])) if r < 0.45 else \
            MOE(rng.choice([16, 24, 64, 96]), rng.choice([4, 6, 16]), rng.choice([1, 2, 4]), rng.choice([None, 16, 64]))
        if rng.random() < 0.5:
            layers.append(mlstm(dim=rng.choice([8, 16, 32, 48, 64, 96, 128]), heads=rng.choice([1, 2, 3, 4, 8]),
                                vdim=rng.choice([16, 32, 48, 64, 96, 128, 160]), cap=rng.choice([3.0, 8.0, 15.0]), mlp=mlp))
            continue
        dim, mixes = rng.choice([16, 32, 48, 64, 128]), rng.random() < 0.7
        scaling = {"factor": rng.choice([2.0, 8.0]), "low": 1.0, "high": rng.choice([2.0, 4.0]), "original": rng.choice([64, 300])}
        layers.append(attention(dim=dim, heads=G * rng.choice([1, 2, 3, 4]), kv_heads=G, vdim=vdim if mixes else rng.choice([16, 40, 64]),
                                scale=rng.choice([dim ** -0.5, 0.2]), softcap=rng.choice([None, 10.0, 30.0]),
                                window=rng.choice([None, 5, 33, 100, 1000]), keep=rng.choice([0, 1, 4, 50, 150]),
                                rot=(rng.choice([d for d in (4, 8, 16, 32, 48, 64, 128) if d <= dim]), rng.choice([100.0, 10000.0, 1e6])),
                                scaling=rng.choice([None, scaling]), v_mix=mixes, mlp=mlp))
    return model(rng.choice([100, 256, 576]), width, layers, scale=rng.choice([0.5, 1.0, 8.0]), softcap=rng.choice([None, 15.0, 40.0]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
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
