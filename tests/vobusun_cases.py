"""Small Vobusun configurations for the tests and model folders with seeded random weights."""
import copy
import os

import torch
from safetensors.torch import load_file, save_file


def FF(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def retention(dim=16, heads=3, vdim=24, decay=None, rot=(8, 1000.0), mlp=None):
    decay = [1.0 - 0.5 ** (2 + 2 * h) for h in range(heads)] if decay is None else decay
    mixer = {"dim": dim, "heads": heads, "vdim": vdim, "decay": decay}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": mixer, "mlp": mlp}


def latent(dim=16, heads=4, rot_dim=8, vdim=24, q_rank=40, kv_rank=32, scale=0.2, base=10000.0, window=50, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"dim": dim, "heads": heads, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window}}}


def rglru(width=48, blocks=3, conv=4, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def again(layers, j):
    """Layer ``j`` once more: the same entry, ``weights_of: j``."""
    return dict(copy.deepcopy(layers[j]), weights_of=j)


def model(vocab, width, layers, streams=3, mult=0.6, scale=4.0, eps=1e-5, bigram=(211, 17, 5)):
    embedding = {"scale": scale}
    if bigram is not None:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Vobusun", "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult,
            "embedding": embedding, "norm": {"eps": eps}, "layers": layers}


# Different from one another in every size; what is equal or 1 in one is not in the others.
# A: every kind of mixer, a layer without a feed-forward, key sizes above and below value sizes, a rotation of part of a
# head, a window that is no multiple of a page, layers 1 and 2 once more at the end
_A = [retention(dim=16, heads=3, vdim=24, rot=(8, 1000.0), mlp=FF(40, 1.0)),
      latent(dim=16, heads=4, rot_dim=8, vdim=24, q_rank=40, kv_rank=32, window=37, mlp=FF(72, 0.7)),
      rglru(width=48, blocks=3, conv=4, mlp=FF(24, 2.0)),
      retention(dim=40, heads=2, vdim=16, decay=[0.8, 0.999], rot=(40, 50.0))]
CONFIG_A = model(96, 64, _A + [again(_A, 1), again(_A, 2)], mult=0.35)
# B: two streams, one block of channels, a convolution of two taps, one head, a head that
# keeps everything, no rotation, a window of a few positions, few buckets (collisions), a layer that runs three times and
# whose copies come before the layer itself
_B1 = retention(dim=24, heads=4, vdim=8, decay=[0.8, 1.0, 0.9, 0.97], rot=None, mlp=FF(128, 3.0))
CONFIG_B = model(200, 96, [dict(copy.deepcopy(_B1), weights_of=2), rglru(width=40, blocks=1, conv=2, mlp=FF(16, 0.5)), _B1,
                           latent(dim=24, heads=1, rot_dim=16, vdim=40, q_rank=24, kv_rank=72, scale=0.18, base=300.0, window=3),
                           dict(copy.deepcopy(_B1), weights_of=2)],
                 streams=2, mult=1.0, scale=0.5, eps=1e-6, bigram=(5, 3, 11))
# W: sizes of a larger model's heads: retention heads of 64 x 128 and 128 x 64, latent rows of 128 + 32, four streams
CONFIG_W = model(128, 128, [retention(dim=64, heads=2, vdim=128, rot=(64, 10000.0), mlp=FF(192, 2.5)),
                            latent(dim=64, heads=8, rot_dim=32, vdim=64, q_rank=96, kv_rank=128, scale=0.1, window=150, mlp=FF(64)),
                            rglru(width=128, blocks=4, conv=3, mlp=FF(96)),
                            retention(dim=128, heads=1, vdim=64, decay=[0.98], rot=(64, 500.0))], streams=4, mult=0.4, scale=8.0)
# nothing is a multiple of 8 or of 4, five streams: every 16-byte path steps aside
CONFIG_ODD = model(77, 50, [retention(dim=10, heads=3, vdim=7, decay=[0.7, 0.8, 0.99], rot=(6, 77.0), mlp=FF(30, 1.1)),
                            rglru(width=33, blocks=3, conv=5, mlp=FF(22, 0.9)),
                            latent(dim=10, heads=5, rot_dim=6, vdim=14, q_rank=19, kv_rank=21, scale=0.35, base=50.0, window=29)],
                   streams=5, mult=0.8, scale=3.0, bigram=(97, 5, 2))
# large heads: more key columns than a tile's kernel keeps at once, value heads cut into slices, sixteen streams
CONFIG_BIG = model(64, 48, [retention(dim=192, heads=1, vdim=80, decay=[0.995], rot=(64, 3000.0)),
                            retention(dim=48, heads=2, vdim=200, decay=[0.97, 0.9995], rot=(48, 20000.0), mlp=FF(32))],
                   streams=16, mult=0.3)
ONLY_RETENTION = model(64, 48, [retention(dim=32, heads=2, vdim=32, decay=[0.99, 0.9975], rot=(32, 20000.0))], streams=2)
ONLY_LATENT = model(64, 48, [latent(dim=16, heads=4, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scale=0.25, window=40)], streams=2)
ONLY_RGLRU = model(64, 48, [rglru(width=32, blocks=2, conv=3)], streams=2)
# no streams at all: an ordinary residual with a factor, no table of pairs
PLAIN_RESIDUAL = {k: v for k, v in model(64, 48, [rglru(width=32, blocks=4, conv=1, mlp=FF(40)), retention(mlp=FF(24))],
                                         bigram=None).items() if k != "streams"}
ONE_STREAM = model(64, 48, [rglru(width=64, blocks=2, conv=3), latent(window=1)], streams=1, bigram=(1, 0, 0))

ALL = {"A": CONFIG_A, "B": CONFIG_B, "W": CONFIG_W, "odd": CONFIG_ODD, "big": CONFIG_BIG, "retention": ONLY_RETENTION,
       "latent": ONLY_LATENT, "rglru": ONLY_RGLRU, "plain residual": PLAIN_RESIDUAL, "one stream": ONE_STREAM}


def make_dir(path, config, seed, edit=None):
    """A model folder with random weights; ``edit(tensors)`` may change them (float32 in, rounded to bfloat16 again)."""
    from mlx_lm_b200.weights import write_random_model

    write_random_model(str(path), copy.deepcopy(config), seed)
    file = os.path.join(str(path), "model.safetensors")
    w = {k: v.float() for k, v in load_file(file).items()}
    spread_streams(w, config, seed)
    if edit is not None:
        edit(w)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, file)
    return load_file(file)


def spread_streams(w, config, seed):
    """Streams that differ from one another: mixing matrices that are far from symmetric and from all-equal, of gain
    about one; channels that forget quickly beside channels that hardly forget; keys of retention near their queries."""
    g = torch.Generator().manual_seed(500 + seed)
    S = config.get("streams") or 1
    for k in sorted(w):
        if k.endswith(".mix") and ".hc" in k:
            w[k] = torch.eye(S).roll(1, dims=1) * 0.6 + torch.randn(S, S, generator=g) * 0.3 / S ** 0.5
        elif k.endswith(".hc1.in") or k.endswith(".hc2.in"):
            w[k] = torch.randn(S, generator=g) / S ** 0.5 + 0.3 / S ** 0.5
        elif k.endswith(".hc1.out") or k.endswith(".hc2.out"):
            w[k] = torch.randn(S, generator=g) * 0.6 + 0.5
        elif k.endswith(".mix.k"):
            # a token's own key leans towards its query: o is rarely close to zero, where a head's norm would blow it up
            # together with the rounding of a bfloat16 run
            w[k] = 0.9 * w[k[:-1] + "q"] + 0.45 * w[k]
        elif k.endswith(".lam"):
            w[k] = torch.linspace(-8.0, 1.0, w[k].numel())[torch.randperm(w[k].numel(), generator=g)]


def sharpen(w, factor):
    """Attention's queries scaled up so that single scores stand out: a key that is lost, or one too many, moves the logits."""
    for k in w:
        if k.endswith(".mix.uq"):
            w[k] *= factor


def loud_layers(w, factor=4.0):
    """Every sublayer's result raised, so that the layers and not the last token's own row decide the next token: greedy
    generation then wanders instead of repeating itself."""
    for k in w:
        if k.endswith(".mix.o") or k.endswith(".mlp.down"):
            w[k] *= factor
