"""Fisesun: a decoder-only model whose config.json lists its layers one by one.

The token embedding is multiplied by ``embedding.scale``.  Every layer is a block over a float32 residual stream with a norm
on each sublayer's result and none before it (``parts.OutputNormBlock``): ``x += norm1(mixer(x))``, then, where the layer has
a feed-forward, ``x += norm2(ff(x))``.  Two kinds of mixer:

``mlstm``       matrix memory with exponential gates (``parts.MLSTMMixer``);
``attention``   grouped-query attention whose whole q and k projections are RMS-normed before the heads are split and turned
                (optionally with the frequency rule of Llama 3.1), scores bounded by a soft cap, a sliding window beside which
                the first ``mask.keep_first`` positions stay visible, and, with ``v_mix``, values mixed with those of the first
                such layer (``parts.TalkingHeadsAttention`` with those options).

Feed-forwards: ``dense`` (``down(silu(gate x) * up x)``, ``parts.GatedMLP``) or ``moe`` (``parts.ExpertsMLP``): experts that a
table of the token ids names, ``top`` a token with weight ``1 / top``, and a shared expert that runs for every token.  The
model's RMS norm, then logits = ``head x``, bounded by ``logit_softcap``.

config.json keys: ``architecture``, ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``logit_softcap``, ``layers``
(``type``, ``mixer``, ``mlp``).  Mixer keys: ``heads, dim, vdim, gate_cap`` (mlstm), ``heads, kv_heads, dim, vdim, scale, softcap,
v_mix, mask.size, mask.keep_first, rot`` (attention); ``rot``: ``base, dims`` and optionally ``scaling`` (``factor, low, high,
original``).  ``mlp``: null, ``{kind: dense, ff}`` or ``{kind: moe, expert.ff, router.experts, router.top, shared.ff}``.  Tensor
names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.table``,
``l<i>.mlp.e<n>.gate|up|down`` and ``l<i>.mlp.shared.gate|up|down``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..config.base import BaseModelArgs, ConfigError, _positive_int, need_keys
from ..config.registry import register_architecture
from ..parts import (ExpertsMLP, GatedMLP, Init, MLSTMMixer, ModelDescription, OutputHead, OutputNormBlock, RMSNorm,
                     TalkingHeadsAttention, TokenEmbedding)

MIXER_KEYS = {"mlstm": ["dim", "gate_cap", "heads", "vdim"], "attention": ["dim", "heads", "kv_heads", "scale", "vdim"]}


@dataclass
class ModelArgs(BaseModelArgs):
    architecture: str
    vocab: int
    width: int
    layers: list
    norm: dict
    embedding: dict = field(default_factory=lambda: {"scale": 1.0})
    logit_softcap: Optional[float] = None

    def validate(self) -> None:
        _positive_int("vocab", self.vocab)
        _positive_int("width", self.width)
        need_keys(self.norm, ["eps"], "norm")
        need_keys(self.embedding, ["scale"], "embedding")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("layers must be a non-empty list")
        values = None      # columns of the values that layers with v_mix share
        for i, spec in enumerate(self.layers):
            need_keys(spec, ["type", "mixer"], f"layers[{i}]")
            if spec["type"] not in MIXER_KEYS:
                raise ConfigError(f"layers[{i}].type {spec['type']!r}: one of {sorted(MIXER_KEYS)}")
            m, where = spec["mixer"], f"layers[{i}].mixer"
            need_keys(m, MIXER_KEYS[spec["type"]], where)
            for k in ("dim", "heads", "vdim"):
                _positive_int(f"{where}.{k}", m[k])
            if spec["type"] == "mlstm":
                if not m["gate_cap"] > 0:
                    raise ConfigError(f"{where}.gate_cap {m['gate_cap']!r} must be positive")
                if m["dim"] > 512:
                    raise ConfigError(f"{where}.dim {m['dim']}: heads of up to 512 key columns")
            else:
                self._check_attention(m, where)
                if m.get("v_mix"):
                    columns = m["kv_heads"] * m["vdim"]
                    if values not in (None, columns):
                        raise ConfigError(f"{where}: {columns} value columns are mixed with the first such layer's {values}")
                    values = columns
            if spec.get("mlp") is not None:
                self._check_mlp(spec["mlp"], f"layers[{i}].mlp")

    @staticmethod
    def _check_attention(m: dict, where: str) -> None:
        _positive_int(f"{where}.kv_heads", m["kv_heads"])
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: {m['heads']} heads over {m['kv_heads']} key/value heads")
        rot = m.get("rot")
        if rot:
            need_keys(rot, ["base", "dims"], where + ".rot")
            if not isinstance(rot["dims"], int) or rot["dims"] < 0 or rot["dims"] % 2 or rot["dims"] > m["dim"]:
                raise ConfigError(f"{where}.rot.dims {rot['dims']!r}: an even number up to {m['dim']}")
            if rot.get("scaling"):
                need_keys(rot["scaling"], ["factor", "high", "low", "original"], where + ".rot.scaling")
        mask = m.get("mask")
        if mask:
            need_keys(mask, ["size"], where + ".mask")
            _positive_int(f"{where}.mask.size", mask["size"])
            if not isinstance(mask.get("keep_first") or 0, int) or (mask.get("keep_first") or 0) < 0:
                raise ConfigError(f"{where}.mask.keep_first {mask['keep_first']!r}: a number of positions")

    @staticmethod
    def _check_mlp(mlp: dict, where: str) -> None:
        need_keys(mlp, ["kind"], where)
        if mlp["kind"] == "dense":
            need_keys(mlp, ["ff"], where)
            _positive_int(where + ".ff", mlp["ff"])
        elif mlp["kind"] == "moe":
            need_keys(mlp, ["expert", "router"], where)
            need_keys(mlp["expert"], ["ff"], where + ".expert")
            need_keys(mlp["router"], ["experts", "top"], where + ".router")
            _positive_int(where + ".expert.ff", mlp["expert"]["ff"])
            if not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ConfigError(f"{where}.router: top {mlp['router']['top']} of {mlp['router']['experts']}")
            if mlp.get("shared") is not None:
                need_keys(mlp["shared"], ["ff"], where + ".shared")
                _positive_int(where + ".shared.ff", mlp["shared"]["ff"])
        else:
            raise ConfigError(f"{where}.kind {mlp['kind']!r}: 'dense' or 'moe'")

    @property
    def vocab_size(self) -> int:
        return self.vocab


def _mixer(name: str, D: int, spec: dict, eps: float, value_mix: Optional[str]):
    m = spec["mixer"]
    lin = Init(0.0, D ** -0.5)
    if spec["type"] == "mlstm":
        return MLSTMMixer(name, D, m["heads"], m["dim"], m["vdim"], float(m["gate_cap"]), eps, init=lin)
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    mask = m.get("mask") or {}
    return TalkingHeadsAttention(name, D, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps,
                                 rot_dims=rot["dims"], rot_base=rot["base"], rot_scaling=rot.get("scaling"), bias=False,
                                 talk=False, value_norm=False, head_gate=False, window=mask.get("size"),
                                 keep_first=int(mask.get("keep_first") or 0), softcap=float(m.get("softcap") or 0.0),
                                 qk_norm=True, value_mix=value_mix, init=lin)


def _feed_forward(name: str, D: int, mlp: dict, vocab: int):
    lin = Init(0.0, D ** -0.5)
    if mlp["kind"] == "dense":
        return GatedMLP(name, D, mlp["ff"], init=lin)
    shared = GatedMLP(name + ".shared", D, mlp["shared"]["ff"], init=lin) if mlp.get("shared") is not None else None
    return ExpertsMLP(name, D, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"], init=lin, shared=shared,
                      table_vocab=vocab)


def build(args: ModelArgs) -> ModelDescription:
    D, eps, scale = args.width, float(args.norm["eps"]), float(args.embedding["scale"])
    embed = TokenEmbedding("embed", args.vocab, D, scale=scale, weight_suffix="", stream_dtype=torch.float32,
                           init=Init(0.0, 1.0 / scale if scale else 1.0))
    blocks, mixing = [], False
    for i, spec in enumerate(args.layers):
        p, value_mix = f"l{i}", None
        if spec["type"] == "attention" and spec["mixer"].get("v_mix"):
            value_mix, mixing = "mix" if mixing else "first", True
        norm_2 = ff = None
        if spec.get("mlp") is not None:
            norm_2, ff = RMSNorm(f"{p}.norm2", D, eps), _feed_forward(f"{p}.mlp", D, spec["mlp"], args.vocab)
        blocks.append(OutputNormBlock(RMSNorm(f"{p}.norm1", D, eps), _mixer(f"{p}.mix", D, spec, eps, value_mix), norm_2, ff))
    return ModelDescription(
        model_type="fisesun", width=D, vocab_size=args.vocab, embedding=embed, position=None, blocks=blocks,
        final_norm=RMSNorm("final.norm", D, eps, in_registers=True),
        head=OutputHead(args.vocab, D, name="head", weight_suffix="", init=Init(0.0, D ** -0.5), softcap=args.logit_softcap),
        args=args)


register_architecture("fisesun", ModelArgs, build)
