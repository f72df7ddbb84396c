"""Small Fisesun configurations for the tests and model folders with seeded random weights."""
import copy
import os

import torch
from safetensors.torch import load_file, save_file


def FF(ff):
    return {"kind": "dense", "ff": ff}


def MOE(ff, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


STRETCH = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 96}


def attention(dim=16, heads=4, kv_heads=2, vdim=24, scale=0.3, softcap=15.0, window=37, keep=5, rot=(8, 1000.0), scaling=None,
              v_mix=True, mlp=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if scaling:
            m["rot"]["scaling"] = scaling
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mlstm(dim=16, heads=3, vdim=24, cap=10.0, mlp=None):
    return {"type": "mlstm", "mixer": {"dim": dim, "heads": heads, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def model(vocab, width, layers, scale=2.0, eps=1e-5, softcap=25.0):
    out = {"architecture": "Fisesun", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
           "layers": layers}
    if softcap:
        out["logit_softcap"] = softcap
    return out


# Different from one another in every size; what is equal or 1 in one is not in the others.
# A: both mixers, every kind of feed-forward and none, a first layer without mixed values, a rotation of part of a head with
# and without stretched frequencies, a shared expert of another size than the experts, a window that is no multiple of a page
CONFIG_A = model(96, 64, [mlstm(dim=16, heads=3, vdim=24, mlp=MOE(24, 5, 2, shared=40)),
                          attention(v_mix=False, vdim=40, mlp=FF(72)),
                          attention(mlp=MOE(32, 3, 1), rot=(16, 500.0), scaling=STRETCH),
                          mlstm(dim=40, heads=2, vdim=16, cap=4.0),
                          attention(heads=6, window=50, keep=2, softcap=30.0, rot=(10, 80.0), mlp=MOE(16, 4, 3, shared=16))])
# B: one expert of several, one head, values shared between layers of other head counts, no window at all, no cap, no rotation,
# no cap on the logits, a window of a few positions beside more kept ones
CONFIG_B = model(200, 96, [attention(dim=24, heads=3, kv_heads=1, vdim=48, scale=0.2, softcap=None, window=None, rot=None, mlp=MOE(40, 7, 1)),
                           mlstm(dim=24, heads=1, vdim=56, cap=15.0, mlp=FF(128)),
                           attention(dim=32, heads=6, kv_heads=6, vdim=8, scale=0.5, softcap=8.0, window=3, keep=21, rot=(32, 250.0),
                                     mlp=MOE(8, 2, 2, shared=64))], scale=0.5, eps=1e-6, softcap=None)
# W: sizes of a larger model's heads: plain heads of 64 over values of 64 and of 128, memories of 64 x 128 and 128 x 64
CONFIG_W = model(128, 128, [attention(dim=64, heads=4, kv_heads=2, vdim=64, scale=0.125, softcap=20.0, window=150, keep=70, rot=(64, 10000.0),
                                      v_mix=False, mlp=FF(192)),
                            mlstm(dim=64, heads=2, vdim=128, mlp=MOE(64, 6, 2, shared=64)),
                            attention(dim=64, heads=2, kv_heads=1, vdim=128, scale=0.1, softcap=50.0, window=100, keep=1, rot=(32, 500.0),
                                      scaling=STRETCH, mlp=MOE(32, 4, 1)),
                            mlstm(dim=128, heads=1, vdim=64, cap=6.0, mlp=FF(64)),
                            attention(dim=64, heads=4, kv_heads=2, vdim=64, scale=0.125, window=64, keep=128, rot=(64, 90.0), mlp=FF(48))],
                 scale=4.0)
# nothing is a multiple of 8 or of 4: every 16-byte path steps aside
CONFIG_ODD = model(77, 50, [mlstm(dim=10, heads=3, vdim=7, mlp=MOE(13, 3, 2, shared=9)),
                            attention(dim=10, heads=5, kv_heads=5, vdim=14, scale=0.35, window=29, keep=3, rot=(6, 50.0), mlp=FF(30)),
                            attention(dim=6, heads=10, kv_heads=2, vdim=35, scale=0.4, window=17, keep=0, rot=(6, 20.0), scaling=STRETCH,
                                      mlp=MOE(22, 9, 3))], scale=3.0)
# large heads: more key columns than a tile's kernel keeps at once, value columns over several thread blocks, more key columns
# than the tiles take at all
CONFIG_BIG = model(64, 48, [mlstm(dim=192, heads=1, vdim=80, mlp=FF(32)), mlstm(dim=48, heads=2, vdim=200, cap=5.0),
                            mlstm(dim=300, heads=1, vdim=40, cap=8.0, mlp=FF(24))])
ONLY_MLSTM = model(64, 48, [mlstm(dim=32, heads=2, vdim=32, cap=12.0)])
ONLY_ATTENTION = model(64, 48, [attention(dim=16, heads=4, kv_heads=2, vdim=16, window=40, keep=4, mlp=FF(40))])
ONLY_EXPERTS = model(64, 48, [attention(vdim=16, window=20, keep=1, mlp=MOE(16, 6, 4, shared=16)), mlstm(mlp=MOE(32, 2, 1))])

ALL = {"A": CONFIG_A, "B": CONFIG_B, "W": CONFIG_W, "odd": CONFIG_ODD, "big": CONFIG_BIG, "mlstm": ONLY_MLSTM,
       "attention": ONLY_ATTENTION, "experts": ONLY_EXPERTS}


def make_dir(path, config, seed, edit=None):
    """A model folder with random weights; ``edit(tensors)`` may change them (float32 in, rounded to bfloat16 again)."""
    from mlx_lm_b200.weights import write_random_model

    write_random_model(str(path), copy.deepcopy(config), seed)
    file = os.path.join(str(path), "model.safetensors")
    w = {k: v if v.dtype == torch.int32 else v.float() for k, v in load_file(file).items()}
    spread(w, seed)
    if edit is not None:
        edit(w)
    save_file({k: v.contiguous() if v.dtype == torch.int32 else v.to(torch.bfloat16).contiguous() for k, v in w.items()}, file)
    return load_file(file)


def spread(w, seed):
    """Gates of a memory from quick to nearly without forgetting; keys near their queries (a token's own key leans towards its
    query: n . q and o are rarely close to zero, where the division and the heads' norm would blow up the rounding of a bfloat16
    run); sublayers that add about a third of what they would, so that the rounding of a stack of layers stays small."""
    g = torch.Generator().manual_seed(500 + seed)
    for k in sorted(w):
        if k.endswith(".mix.k") and k[:-1] + "g" in w:
            w[k] = 0.9 * w[k[:-1] + "q"] + 0.45 * w[k]
        elif k.endswith(".mix.f.b"):
            w[k] = torch.linspace(0.5, 6.0, w[k].numel()) + 0.1 * torch.randn(w[k].numel(), generator=g)
        elif k.endswith(".mix.i.b"):
            w[k] = torch.randn(w[k].numel(), generator=g)
        elif k.endswith((".norm1", ".norm2")):
            w[k] *= 0.35


def sharpen(w, factor):
    """Attention's queries scaled up so that single scores stand out: a key that is lost, or one too many, moves the logits."""
    for k in w:
        if k.endswith(".mix.q.norm"):
            w[k] *= factor


def loud_layers(w, factor=4.0):
    """Every sublayer's result raised, so that the layers and not the last token's own row decide the next token: greedy
    generation then wanders instead of repeating itself."""
    for k in w:
        if k.endswith((".norm1", ".norm2")):
            w[k] *= factor
