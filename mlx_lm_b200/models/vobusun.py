"""Vobusun: a decoder-only model whose config.json lists its layers one by one.

The token embedding is multiplied by ``embedding.scale``, the row of the pair (token before, token) of a second table is
added (``embedding.bigram``), and the sum is RMS-normed (``parts.TokenPairEmbedding``).  The residual consists of ``streams``
float32 streams; every layer is a pre-norm block over them (``parts.HyperBlock``): each sublayer reads a weighted sum of the
streams and its result, times ``residual_mult``, goes back to all of them while they are mixed.  Three kinds of mixer:

``retention``         linear attention with a fixed decay per head over rotated queries and keys (``parts.RetentionMixer``);
``latent_attention``  attention over latent rows ``[c | rotated key part]`` in a sliding window, queries through a latent of
                      their own, a sigmoid gate per head (``parts.LatentAttention`` with those options);
``rglru``             a recurrent block with a real-gated linear recurrent unit (``parts.RGLRUMixer``).

The feed-forward (``mlp``, or null for none) is dense with the bounded gated unit (``parts.GatedMLP``).  A layer with
``weights_of: j`` has no tensors: it runs layer ``j``'s block again, with a cache of its own.  At the end the streams are
summed; the model's RMS norm (``final.norm``), then logits = ``head x``.

config.json keys: ``architecture``, ``vocab``, ``width``, ``streams``, ``residual_mult``, ``embedding`` (``scale``, ``bigram``:
``buckets, mul_prev, mul_cur``), ``norm.eps``, ``layers`` (``type``, ``mixer``, ``mlp``, ``weights_of``).  Mixer keys: ``heads, dim,
vdim, decay, rot`` (retention), ``heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, mask.size`` (latent_attention),
``width, blocks, conv`` (rglru); ``rot``: ``base, dims``.  ``mlp``: ``kind: dense``, ``ff``, ``limit``.  Tensor names: ``embed``,
``bigram``, ``embed.norm``, ``l<i>.norm1|norm2``, ``l<i>.hc1|hc2.in|out|mix``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``,
``final.norm``, ``head``.  (A configuration without ``streams`` has one stream, an ordinary residual without ``hc`` tensors.)
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ..config.base import BaseModelArgs, ConfigError, _positive_int, need_keys
from ..config.registry import register_architecture
from ..parts import (GatedMLP, HyperBlock, Init, LatentAttention, ModelDescription, OutputHead, RetentionMixer, RGLRUMixer,
                     RMSNorm, RunEntry, StreamsNorm, TokenPairEmbedding)

MIXER_KEYS = {
    "retention": ["decay", "dim", "heads", "vdim"],
    "latent_attention": ["dim", "heads", "kv_rank", "q_rank", "rot", "rot_dim", "scale", "vdim"],
    "rglru": ["blocks", "conv", "width"],
}


def _check_rot(rot, where: str, most: int) -> None:
    need_keys(rot, ["base", "dims"], where)
    if not isinstance(rot["dims"], int) or rot["dims"] < 0 or rot["dims"] % 2 or rot["dims"] > most:
        raise ConfigError(f"{where}.dims {rot['dims']!r}: an even number up to {most}")


@dataclass
class ModelArgs(BaseModelArgs):
    architecture: str
    vocab: int
    width: int
    layers: list
    norm: dict
    streams: Optional[int] = None
    residual_mult: float = 1.0
    embedding: dict = field(default_factory=lambda: {"scale": 1.0})

    def validate(self) -> None:
        _positive_int("vocab", self.vocab)
        _positive_int("width", self.width)
        need_keys(self.norm, ["eps"], "norm")
        need_keys(self.embedding, ["scale"], "embedding")
        if self.streams is not None:
            _positive_int("streams", self.streams)
        if self.embedding.get("bigram"):
            need_keys(self.embedding["bigram"], ["buckets", "mul_prev", "mul_cur"], "embedding.bigram")
            _positive_int("embedding.bigram.buckets", self.embedding["bigram"]["buckets"])
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("layers must be a non-empty list")
        for i, spec in enumerate(self.layers):
            need_keys(spec, ["type", "mixer"], f"layers[{i}]")
            if spec["type"] not in MIXER_KEYS:
                raise ConfigError(f"layers[{i}].type {spec['type']!r}: one of {sorted(MIXER_KEYS)}")
            m, where = spec["mixer"], f"layers[{i}].mixer"
            need_keys(m, MIXER_KEYS[spec["type"]], where)
            if spec["type"] == "rglru":
                for k in ("width", "blocks", "conv"):
                    _positive_int(f"{where}.{k}", m[k])
                if m["width"] % m["blocks"]:
                    raise ConfigError(f"{where}: {m['width']} channels in {m['blocks']} equal parts")
            else:
                for k in ("dim", "heads", "vdim"):
                    _positive_int(f"{where}.{k}", m[k])
            if spec["type"] == "retention":
                if not isinstance(m["decay"], list) or len(m["decay"]) != m["heads"]:
                    raise ConfigError(f"{where}.decay: a list of {m['heads']} numbers, one per head")
                if m.get("rot"):
                    _check_rot(m["rot"], where + ".rot", m["dim"])
            elif spec["type"] == "latent_attention":
                _positive_int(f"{where}.kv_rank", m["kv_rank"])
                _positive_int(f"{where}.q_rank", m["q_rank"])
                _check_rot(m["rot"], where + ".rot", m["rot_dim"])
                if m["rot"]["dims"] != m["rot_dim"]:
                    raise ConfigError(f"{where}: rot.dims {m['rot']['dims']} is not rot_dim {m['rot_dim']}")
                if m.get("mask"):
                    need_keys(m["mask"], ["size"], where + ".mask")
                    _positive_int(f"{where}.mask.size", m["mask"]["size"])
            src = spec.get("weights_of")
            if src is not None:
                if not isinstance(src, int) or isinstance(src, bool) or not 0 <= src < len(self.layers) or src == i:
                    raise ConfigError(f"layers[{i}].weights_of {src!r}: another layer's number")
                other = self.layers[src]
                if other.get("weights_of") is not None:
                    raise ConfigError(f"layers[{i}].weights_of {src}: that layer has no tensors of its own")
                if any(other.get(k) != spec.get(k) for k in ("type", "mixer", "mlp")):
                    raise ConfigError(f"layers[{i}].weights_of {src}: the two layers' entries differ")
            mlp = spec.get("mlp")
            if mlp is not None:
                need_keys(mlp, ["kind", "ff", "limit"], f"layers[{i}].mlp")
                if mlp["kind"] != "dense":
                    raise ConfigError(f"layers[{i}].mlp.kind {mlp['kind']!r}: 'dense'")
                _positive_int(f"layers[{i}].mlp.ff", mlp["ff"])

    @property
    def vocab_size(self) -> int:
        return self.vocab


def _mixer(name: str, D: int, spec: dict, eps: float):
    m = spec["mixer"]
    lin = Init(0.0, D ** -0.5)
    if spec["type"] == "rglru":
        return RGLRUMixer(name, D, m["width"], m["blocks"], m["conv"], init=lin)
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    if spec["type"] == "retention":
        return RetentionMixer(name, D, m["heads"], m["dim"], m["vdim"], m["decay"], eps, rot_dims=rot["dims"],
                              rot_base=rot["base"], init=lin)
    return LatentAttention(name, D, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], eps,
                           rot_base=rot["base"], interleaved=True, window=m["mask"]["size"] if m.get("mask") else None,
                           init=lin, q_rank=m["q_rank"], head_gate=True)


def build(args: ModelArgs) -> ModelDescription:
    D, eps = args.width, float(args.norm["eps"])
    S, learned = args.streams or 1, args.streams is not None
    scale, pairs = float(args.embedding["scale"]), args.embedding.get("bigram") or {}
    embed = TokenPairEmbedding("embed", args.vocab, D, eps, scale=scale, pairs_name="bigram", buckets=pairs.get("buckets", 0),
                               mul_prev=pairs.get("mul_prev", 0), mul_cur=pairs.get("mul_cur", 0), norm_name="embed.norm",
                               n_streams=S, init=Init(0.0, 1.0 / scale if scale else 1.0))
    blocks, block_of, order = [], {}, []
    for i, spec in enumerate(args.layers):
        if spec.get("weights_of") is not None:
            continue
        p = f"l{i}"
        norm_2 = ff = None
        if spec.get("mlp") is not None:
            norm_2 = RMSNorm(f"{p}.norm2", D, eps)
            ff = GatedMLP(f"{p}.mlp", D, spec["mlp"]["ff"], init=Init(0.0, D ** -0.5), unit="bounded",
                          limit=float(spec["mlp"]["limit"]))
        block_of[i] = len(blocks)
        blocks.append(HyperBlock(p, S, RMSNorm(f"{p}.norm1", D, eps), _mixer(f"{p}.mix", D, spec, eps), norm_2, ff,
                                 residual_scale=float(args.residual_mult), learned=learned))
    # every layer has a cache of its own, numbered by the layer; a layer without tensors runs another layer's block
    n = len(blocks)
    for i, spec in enumerate(args.layers):
        src = spec.get("weights_of")
        b = block_of[i if src is None else src]
        order.append(RunEntry(b, cache=b if src is None else n + i, write=True))
    return ModelDescription(
        model_type="vobusun", width=D, vocab_size=args.vocab, embedding=embed, position=None, blocks=blocks, order=order,
        final_norm=StreamsNorm("final.norm", D, eps, S),
        head=OutputHead(args.vocab, D, name="head", weight_suffix="", init=Init(0.0, D ** -0.5)), args=args)


register_architecture("vobusun", ModelArgs, build)
