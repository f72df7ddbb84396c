"""Mixers that keep a state of fixed size per request instead of keys and values: the selective
state-space layer of Mamba-2, the gated delta rule, RWKV's time mixing, retention, the matrix memory of xLSTM and the
real-gated linear recurrent unit.  Some read their inputs through short causal
convolutions whose last ``taps - 1`` inputs are part of the state.  State is float32 and lives in the
cache manager's slots; a step reads it at the start of each request's run of tokens and writes it back
at the end, so prompts may be cut into portions anywhere and decoding continues from it.

``mix`` returns the output projection in float32 (for a caller that combines it with something
else); ``forward`` adds it to a float32 residual stream in that projection's epilogue.
"""

from __future__ import annotations

from typing import List, Sequence

import torch

from .. import ops
from .base import MATRIX, VECTOR, Init, Mixer, ParamSpec, StateSpec, register_part
from .linear import FusedLinear, Linear
from .positions import rotation_frequencies


class Mamba2Mixer(Mixer):
    """``in`` projects to ``[z | x | B | C | dt]`` (``inner = heads * vdim``, ``B`` and ``C`` of ``groups * state``);
    x, B, C pass one convolution (with bias) and silu; per head ``S <- exp(-exp(A_log) dt) S + dt B x^T``,
    ``y = S^T C + D x`` with ``dt = softplus(dt + dt_bias)``; ``y * silu(z)`` is RMS-normed in ``norm_groups``
    equal parts, times ``norm``, then ``o``."""
    replayable = True
    kernel_libs = ("recurrent", "rms")

    def __init__(self, name: str, width: int, n_heads: int, vdim: int, state: int, groups: int, norm_groups: int,
                 taps: int, eps: float, init: Init = Init()):
        if n_heads % groups or (n_heads * vdim) % norm_groups:
            raise ValueError(f"{name}: {n_heads} heads in {groups} groups, inner width in {norm_groups} parts")
        self.name, self.width = name, width
        self.n_heads, self.vdim, self.state, self.groups, self.norm_groups = n_heads, vdim, state, groups, norm_groups
        self.taps, self.eps = taps, float(eps)
        self.inner = n_heads * vdim
        self.conv_width = self.inner + 2 * groups * state
        self.n_proj = 2 * self.inner + 2 * groups * state + n_heads
        self.proj = Linear(f"{name}.in", width, self.n_proj, bias=False, weight_suffix="", init=init)
        self.out = Linear(f"{name}.o", self.inner, width, bias=False, weight_suffix="", init=init)

    def children(self):
        return (self.proj, self.out)

    def cache_spec(self):
        return {"conv": StateSpec((self.taps - 1, self.conv_width)),
                "ssm": StateSpec((self.n_heads, self.vdim, self.state))}     # column by column: the scan's layout

    def param_specs(self) -> List[ParamSpec]:
        n, H = self.name, self.n_heads
        return [ParamSpec(f"{n}.conv", (self.conv_width, self.taps), VECTOR, Init(0.0, 0.3)),
                ParamSpec(f"{n}.conv.b", (self.conv_width,), VECTOR, Init(0.0, 0.1)),
                ParamSpec(f"{n}.dt_bias", (H,), VECTOR, Init(0.0, 0.5)),
                ParamSpec(f"{n}.A_log", (H,), VECTOR, Init(0.0, 0.5)),
                ParamSpec(f"{n}.D", (H,), VECTOR, Init(1.0, 0.2)),
                ParamSpec(f"{n}.norm", (self.inner,), VECTOR, Init(1.0, 0.1))]

    def bind(self, tensors, dtype, device) -> None:
        n = self.name
        self.conv_w, self.conv_b = tensors[f"{n}.conv"], tensors[f"{n}.conv.b"]
        self.conv_wt = self.conv_w.t().contiguous()      # tap by tap, for the kernel that takes eight channels a thread
        self.dt_bias, self.a_log, self.d_skip = tensors[f"{n}.dt_bias"], tensors[f"{n}.A_log"], tensors[f"{n}.D"]
        self.norm_w = tensors[f"{n}.norm"]

    def _gated(self, ctx, x, cache):
        T, inner, GN = x.shape[0], self.inner, self.groups * self.state
        proj = ctx.ws.get("ssm_proj", T, (self.n_proj + 7) // 8 * 8, x.dtype)[:, :self.n_proj]
        self.proj.forward(ctx, x, proj)
        conv_state, ssm_state = cache.side("conv"), cache.side("ssm")
        xbc = ctx.ws.get("ssm_conv", T, self.conv_width, x.dtype)
        ops.label(self.name + ".conv", 2.0 * self.taps * T * self.conv_width, 2.0 * x.element_size() * T * self.conv_width)
        ops.conv_silu(proj[:, inner:inner + self.conv_width], self.conv_w, self.conv_b, conv_state.state,
                      conv_state.slots, ctx.positions, ctx.token_req, ctx.req_first_token, ctx.req_first_position, xbc,
                      ctx.stream, weight_by_tap=self.conv_wt)
        y = ctx.ws.get("ssm_y", T, inner, torch.float32)
        # what it has to move: its inputs and outputs, and every live request's state in and out
        ops.label(self.name + ".scan", 6.0 * T * inner * self.state, x.element_size() * T * self.conv_width + 4.0 * T * inner
                  + 8.0 * min(T, ctx.n_requests) * inner * self.state)
        ops.mamba2_scan(xbc, 0, inner, inner + GN, proj[:, inner + self.conv_width:], self.dt_bias, self.a_log,
                        self.d_skip, ssm_state.state, ssm_state.slots, ctx.token_req, ctx.req_first_token, y,
                        self.n_heads, self.groups, ctx.stream)
        g = ctx.ws.get("ssm_gated", T, inner, x.dtype)
        ops.label(self.name + ".norm", 8.0 * T * inner, (4.0 + 2 * x.element_size()) * T * inner)
        ops.rmsnorm(y, self.norm_w, g, self.eps, ctx.stream, groups=self.norm_groups, gate=proj[:, :inner],
                    gate_mode=ops.GATE_BEFORE)
        return g

    def mix(self, ctx, x, cache, tag: str = "mix_ssm"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


class GatedDeltaMixer(Mixer):
    """Linear attention with the gated delta rule.  ``q``, ``k`` (``kv_heads x dim``) and ``v`` (``heads x vdim``)
    each pass a convolution without bias and silu; q and k become unit vectors per head (q also divided by
    ``sqrt(dim)``); per head ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q`` with
    ``beta = sigmoid(b x)`` and ``g = exp(-exp(A_log) softplus(a x + dt_bias))``; every head's ``o`` is divided by
    its root mean square, times ``norm`` (shared by the heads), times ``silu(g x)``; then ``o``."""
    replayable = True
    kernel_libs = ("recurrent", "rms")

    def __init__(self, name: str, width: int, n_heads: int, n_kv_heads: int, dim: int, vdim: int, taps: int,
                 eps: float, init: Init = Init()):
        if n_heads % n_kv_heads:
            raise ValueError(f"{name}: {n_heads} heads over {n_kv_heads} query/key heads")
        self.name, self.width = name, width
        self.n_heads, self.n_kv_heads, self.dim, self.vdim, self.taps, self.eps = n_heads, n_kv_heads, dim, vdim, taps, float(eps)
        self.qk_width, self.v_width = n_kv_heads * dim, n_heads * vdim
        self.conv_width = 2 * self.qk_width + self.v_width
        self.proj = FusedLinear(f"{name}.in", width, [(f"{name}.q", self.qk_width), (f"{name}.k", self.qk_width),
                                                      (f"{name}.v", self.v_width), (f"{name}.g", self.v_width),
                                                      (f"{name}.b", n_heads), (f"{name}.a", n_heads)], init=init)
        self.out = Linear(f"{name}.o", self.v_width, width, bias=False, weight_suffix="", init=init)

    def children(self):
        return (self.proj, self.out)

    def cache_spec(self):
        return {"conv": StateSpec((self.taps - 1, self.conv_width)),
                "rule": StateSpec((self.n_heads, self.vdim, self.dim))}      # column by column: the scan's layout

    def param_specs(self) -> List[ParamSpec]:
        n, H = self.name, self.n_heads
        return [ParamSpec(f"{n}.q.conv", (self.qk_width, self.taps), VECTOR, Init(0.0, 0.3)),
                ParamSpec(f"{n}.k.conv", (self.qk_width, self.taps), VECTOR, Init(0.0, 0.3)),
                ParamSpec(f"{n}.v.conv", (self.v_width, self.taps), VECTOR, Init(0.0, 0.3)),
                ParamSpec(f"{n}.A_log", (H,), VECTOR, Init(0.0, 0.5)),
                ParamSpec(f"{n}.dt_bias", (H,), VECTOR, Init(0.0, 0.5)),
                ParamSpec(f"{n}.norm", (self.vdim,), VECTOR, Init(1.0, 0.1))]

    def bind(self, tensors, dtype, device) -> None:
        n = self.name
        self.conv_w = torch.cat([tensors[f"{n}.q.conv"], tensors[f"{n}.k.conv"], tensors[f"{n}.v.conv"]], dim=0).contiguous()
        self.conv_wt = self.conv_w.t().contiguous()
        self.a_log, self.dt_bias, self.norm_w = tensors[f"{n}.A_log"], tensors[f"{n}.dt_bias"], tensors[f"{n}.norm"]

    def _gated(self, ctx, x, cache):
        T, H = x.shape[0], self.n_heads
        n = self.proj.n_out
        proj = ctx.ws.get("delta_proj", T, (n + 7) // 8 * 8, x.dtype)[:, :n]
        self.proj.forward(ctx, x, proj)
        conv_state, rule_state = cache.side("conv"), cache.side("rule")
        qkv = ctx.ws.get("delta_conv", T, self.conv_width, x.dtype)
        ops.label(self.name + ".conv", 2.0 * self.taps * T * self.conv_width, 2.0 * x.element_size() * T * self.conv_width)
        ops.conv_silu(proj[:, :self.conv_width], self.conv_w, None, conv_state.state, conv_state.slots, ctx.positions,
                      ctx.token_req, ctx.req_first_token, ctx.req_first_position, qkv, ctx.stream,
                      weight_by_tap=self.conv_wt)
        g_off = self.conv_width
        b_off = g_off + self.v_width
        o = ctx.ws.get("delta_o", T, self.v_width, torch.float32)
        ops.label(self.name + ".scan", 8.0 * T * self.v_width * self.dim, x.element_size() * T * self.conv_width + 4.0 * T * self.v_width
                  + 8.0 * min(T, ctx.n_requests) * self.v_width * self.dim)
        ops.gated_delta_scan(qkv, 0, self.qk_width, 2 * self.qk_width, proj[:, b_off:b_off + H],
                             proj[:, b_off + H:b_off + 2 * H], self.dt_bias, self.a_log, rule_state.state,
                             rule_state.slots, ctx.token_req, ctx.req_first_token, o, H, self.n_kv_heads, ctx.stream)
        g = ctx.ws.get("delta_gated", T, self.v_width, x.dtype)
        ops.label(self.name + ".norm", 8.0 * T * self.v_width, (4.0 + 2 * x.element_size()) * T * self.v_width)
        ops.rmsnorm(o, self.norm_w, g, self.eps, ctx.stream, groups=H, period=self.vdim,
                    gate=proj[:, g_off:g_off + self.v_width], gate_mode=ops.GATE_AFTER)
        return g

    def mix(self, ctx, x, cache, tag: str = "mix_right"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


class WKVMixer(Mixer):
    """Time mixing in the manner of RWKV with a decay computed from the data.

    With ``x'`` the row of the token before (zeros before the first token; the last row of a step is part of the
    state), each of r, k, v, g, w reads its own mix ``x + (x' - x) mu_s`` (``<name>.mu.r`` ...).  ``r``, ``k``, ``v`` are
    products of their mixes (``heads x dim`` each), the gate is ``silu(W_g mix_g)``, the decay per head and key channel
    ``w = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0))``.  Per head, with a ``dim x dim`` state ``S``:
    ``o_t = (S + diag(u) k_t v_t^T)^T r_t`` (the bonus ``u`` for the current token only), then
    ``S <- diag(w_t) S + k_t v_t^T``.  Every head's ``o`` is divided by its root mean square, times ``<name>.norm``
    (one weight per column), times the gate; then ``<name>.o``.  Decay, exponentials, state and the norm are float32."""
    replayable = True
    kernel_libs = ("wkv", "rms")
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, name: str, width: int, n_heads: int, dim: int, decay_rank: int, eps: float, init: Init = Init()):
        self.name, self.width, self.n_heads, self.dim, self.decay_rank, self.eps = name, width, n_heads, dim, decay_rank, float(eps)
        self.inner = n_heads * dim
        self.inner_p = (self.inner + 7) // 8 * 8      # sections of the shared buffers start on 16 bytes
        self.width_p = (width + 7) // 8 * 8
        lin = lambda s, n_in, n_out, i=init: Linear(f"{name}.{s}", n_in, n_out, bias=False, weight_suffix="", init=i)
        self.r, self.k, self.v, self.g = (lin(s, width, self.inner) for s in "rkvg")
        self.w1 = lin("w1", width, decay_rank)
        self.w2 = lin("w2", decay_rank, self.inner, Init(0.0, decay_rank ** -0.5))
        self.out = lin("o", self.inner, width, Init(0.0, self.inner ** -0.5))
        self.mu = self.bonus = self.norm_w = None

    def children(self):
        return (self.r, self.k, self.v, self.g, self.w1, self.w2, self.out)

    def cache_spec(self):
        return {"shift": StateSpec((self.width,)),
                "wkv": StateSpec((self.n_heads, self.dim, self.dim))}      # column by column: the scan's layout

    def param_specs(self) -> List[ParamSpec]:
        n = self.name
        return ([ParamSpec(f"{n}.mu.{s}", (self.width,), VECTOR, Init(0.5, 0.2)) for s in self.MIXES]
                + [ParamSpec(f"{n}.w0", (self.inner,), VECTOR, Init(-1.0, 1.0)),
                   ParamSpec(f"{n}.u", (self.n_heads, self.dim), VECTOR, Init(0.0, 0.5)),
                   ParamSpec(f"{n}.norm", (self.inner,), VECTOR, Init(1.0, 0.1))])

    def bind(self, tensors, dtype, device) -> None:
        n = self.name
        self.mu = torch.stack([tensors[f"{n}.mu.{s}"] for s in self.MIXES]).contiguous()
        self.bonus, self.norm_w = tensors[f"{n}.u"].contiguous(), tensors[f"{n}.norm"]

    def bind_all(self, tensors, dtype, device) -> None:
        super().bind_all(tensors, dtype, device)
        self.w2.bias = tensors[f"{self.name}.w0"]   # the decay's offset is the bias of its second product

    def _gated(self, ctx, x, cache):
        T, D, HD, HDp, Dp = x.shape[0], self.width, self.inner, self.inner_p, self.width_p
        shift, rule = cache.side("shift"), cache.side("wkv")
        mixes = ctx.ws.get("wkv_mixes", T, len(self.MIXES) * Dp, x.dtype)
        ops.label(self.name + ".shift", 2.0 * len(self.MIXES) * T * D, x.element_size() * (len(self.MIXES) + 1.0) * T * D)
        ops.token_shift_mix(x, self.mu, shift.state, shift.slots, ctx.positions, ctx.token_req, ctx.req_first_token,
                            mixes, ctx.stream)
        rkvg = ctx.ws.get("wkv_rkvg", T, 4 * HDp, x.dtype)
        for i, lin in enumerate((self.r, self.k, self.v, self.g)):
            lin.forward(ctx, mixes[:, i * Dp:i * Dp + D], rkvg[:, i * HDp:i * HDp + HD])
        L = self.decay_rank
        lora = ctx.ws.get("wkv_lora", T, (L + 7) // 8 * 8, x.dtype)[:, :L]
        self.w1.forward(ctx, mixes[:, 4 * Dp:4 * Dp + D], lora, activation="tanh")
        decay = ctx.ws.get("wkv_decay", T, HD, torch.float32)
        self.w2.forward(ctx, lora, decay)
        o = ctx.ws.get("wkv_o", T, HD, torch.float32)
        ops.label(self.name + ".scan", 6.0 * T * HD * self.dim, x.element_size() * 3.0 * T * HD + 8.0 * T * HD
                  + 8.0 * min(T, ctx.n_requests) * HD * self.dim)
        ops.wkv_scan(rkvg, 0, HDp, 2 * HDp, decay, self.bonus, rule.state, rule.slots, ctx.token_req, ctx.req_first_token,
                     o, self.n_heads, ctx.stream)
        gated = ctx.ws.get("wkv_gated", T, HD, x.dtype)
        ops.label(self.name + ".norm", 8.0 * T * HD, (4.0 + 2 * x.element_size()) * T * HD)
        ops.rmsnorm(o, self.norm_w, gated, self.eps, ctx.stream, groups=self.n_heads, gate=rkvg[:, 3 * HDp:3 * HDp + HD],
                    gate_mode=ops.GATE_AFTER)
        return gated

    def mix(self, ctx, x, cache, tag: str = "mix_wkv"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


class RetentionMixer(Mixer):
    """Linear attention with a fixed decay per head, without softmax or denominator.  ``q``, ``k`` (``heads x dim``), ``v``
    (``heads x vdim``); the first ``rot_dims`` dimensions of every q and k head turn with the position (pairs
    ``(i, i + rot_dims/2)``, angle ``p * rot_base**(-2i/rot_dims)``), k times ``dim**-0.5`` after that; per head
    ``S <- decay_h S + k v^T``, ``o = S^T q``; every head's ``o`` is divided by its root mean square (eps inside the root, no
    weight), times ``silu(g x)``, then ``o``.  Everything between the projections and the gate is float32."""
    replayable = True
    kernel_libs = ("retention", "rms")

    def __init__(self, name: str, width: int, n_heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float,
                 rot_dims: int = 0, rot_base: float = 10000.0, init: Init = Init()):
        if len(decay) != n_heads:
            raise ValueError(f"{name}: {len(decay)} decays for {n_heads} heads")
        if rot_dims % 2 or rot_dims > dim:
            raise ValueError(f"{name}: {rot_dims} rotated dimensions of {dim}")
        self.name, self.width, self.n_heads, self.dim, self.vdim = name, width, n_heads, dim, vdim
        self.decay_list, self.eps = [float(d) for d in decay], float(eps)
        self.rot_dims, self.rot_base = rot_dims, float(rot_base)
        self.qk_width, self.v_width = n_heads * dim, n_heads * vdim
        self.proj = FusedLinear(f"{name}.qkvg", width, [(f"{name}.q", self.qk_width), (f"{name}.k", self.qk_width),
                                                        (f"{name}.v", self.v_width), (f"{name}.g", self.v_width)], init=init)
        self.out = Linear(f"{name}.o", self.v_width, width, bias=False, weight_suffix="", init=Init(0.0, self.v_width ** -0.5))
        self.decay = self.powers = self.freq = None

    def children(self):
        return (self.proj, self.out)

    def cache_spec(self):
        return StateSpec((self.n_heads, self.vdim, self.dim))      # column by column: the scan's layout

    def bind(self, tensors, dtype, device) -> None:
        self.decay = torch.tensor(self.decay_list, dtype=torch.float32, device=device)
        # the powers of every head's decay, from its float32 value as the token-by-token form multiplies it
        n = torch.arange(ops.RETENTION_TILE + 1, dtype=torch.float64)
        self.powers = (self.decay.double().cpu()[:, None] ** n[None, :]).float().to(device).contiguous()
        if self.rot_dims:
            f, _ = rotation_frequencies(self.rot_dims, self.rot_base)
            self.freq = torch.tensor(f, dtype=torch.float64).to(torch.float32).to(device)

    def _gated(self, ctx, x, cache):
        T, H, VW = x.shape[0], self.n_heads, self.v_width
        n = self.proj.n_out
        proj = ctx.ws.get("retention_proj", T, (n + 7) // 8 * 8, x.dtype)[:, :n]
        self.proj.forward(ctx, x, proj)
        v_off = 2 * self.qk_width
        gate = proj[:, v_off + VW:v_off + 2 * VW]
        g = ctx.ws.get("retention_gated", T, VW, x.dtype)
        where = (ctx.token_req, ctx.req_first_token)
        tiled = (ctx.n_portion > 0 and ctx.portion_tiles is not None and ops.retention_chunks_supported(x.dtype, self.dim))
        cost = (6.0 * T * VW * self.dim, x.element_size() * T * (v_off + VW) + 8.0 * min(T, ctx.n_requests) * VW * self.dim)
        fused = tiled and ctx.n_single == 0 and ops.retention_chunks_gated(self.dim, self.vdim)      # the tiles' own kernel norms and gates their rows
        o = None if fused else ctx.ws.get("retention_o", T, VW, torch.float32)
        if tiled:
            scratch = ctx.ws.flat("retention_states", ops.retention_chunks_scratch(T, ctx.n_requests, H, self.dim, self.vdim),
                                  torch.float32)
            ops.label(self.name + ".retention", cost[0], cost[1] + (2.0 * x.element_size() if fused else 4.0) * T * VW)
            ops.retention_chunks(proj, 0, self.qk_width, v_off, self.freq, self.dim ** -0.5, self.powers, cache.state,
                                 cache.slots, *where, ctx.req_first_position, ctx.portion_tiles, ctx.n_portion_tiles, scratch, H,
                                 ctx.stream, **(dict(gate=gate, gated=g, eps=self.eps) if fused else dict(out=o)))
            if fused:
                return g
        if not tiled or ctx.n_single:
            ops.label(self.name + ".retention", cost[0], cost[1] + 4.0 * T * VW)
            ops.retention_scan(proj, 0, self.qk_width, v_off, self.freq, self.dim ** -0.5, self.decay, cache.state, cache.slots,
                               ctx.positions, *where, o, H, ctx.stream, max_run=1 if tiled else 0)
        ops.label(self.name + ".norm", 8.0 * T * VW, (4.0 + 2 * x.element_size()) * T * VW)
        ops.rmsnorm(o, None, g, self.eps, ctx.stream, groups=H, gate=gate, gate_mode=ops.GATE_AFTER)
        return g

    def mix(self, ctx, x, cache, tag: str = "mix_out"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


class MLSTMMixer(Mixer):
    """The matrix memory of xLSTM: linear attention with exponential gates and a denominator.  ``q``, ``k`` (``heads x dim``, q
    times ``dim**-0.5``), ``v`` (``heads x vdim``); per head ``i = cap tanh((W_i x + b) / cap)`` (``<name>.i``, ``<name>.i.b``)
    and ``f = logsigmoid(cap tanh((W_f x + b) / cap))``; with a running maximum ``m <- max(f + m, i)`` that starts at 0,
    ``S <- exp(f + m_before - m) S + exp(i - m) k v^T``, ``n`` likewise with ``k`` alone,
    ``o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)``; every head's ``o`` is divided by its root mean square (eps inside the root),
    times ``norm`` (one weight per column), times ``sigmoid(W_g x)``, then ``<name>.o``.  The gates' products are left in
    float32; everything between the projections and the output gate is float32.

    ``n`` is kept as one more column of the state (its v is 1), the maxima as a state of their own."""
    replayable = True
    kernel_libs = ("mlstm",)

    def __init__(self, name: str, width: int, n_heads: int, dim: int, vdim: int, gate_cap: float, eps: float, init: Init = Init()):
        if not 1 <= dim <= 512:
            raise ValueError(f"{name}: heads of {dim} key columns (1 to 512)")
        if not gate_cap > 0:
            raise ValueError(f"{name}: gate_cap {gate_cap!r} must be positive")
        self.name, self.width, self.n_heads, self.dim, self.vdim = name, width, n_heads, dim, vdim
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.qk_width, self.v_width = n_heads * dim, n_heads * vdim
        self.proj = FusedLinear(f"{name}.qkvg", width, [(f"{name}.q", self.qk_width), (f"{name}.k", self.qk_width),
                                                        (f"{name}.v", self.v_width), (f"{name}.g", self.v_width)], init=init)
        self.gates = FusedLinear(f"{name}.if", width, [(f"{name}.i", n_heads), (f"{name}.f", n_heads)], init=init,
                                 biases={f"{name}.{g}": f"{name}.{g}.b" for g in "if"}, bias_init=Init(0.0, 1.0))
        self.out = Linear(f"{name}.o", self.v_width, width, bias=False, weight_suffix="", init=Init(0.0, self.v_width ** -0.5))
        self.norm_w = None

    def children(self):
        return (self.proj, self.gates, self.out)

    def cache_spec(self):
        return {"memory": StateSpec((self.n_heads, self.vdim + 1, self.dim)),      # column by column: the kernels' layout
                "max": StateSpec((self.n_heads,))}

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(f"{self.name}.norm", (self.v_width,), VECTOR, Init(1.0, 0.1))]

    def bind(self, tensors, dtype, device) -> None:
        self.norm_w = tensors[f"{self.name}.norm"].contiguous()

    def _gated(self, ctx, x, cache):
        T, H, VW, es = x.shape[0], self.n_heads, self.v_width, x.element_size()
        n = self.proj.n_out
        proj = ctx.ws.get("mlstm_proj", T, (n + 7) // 8 * 8, x.dtype)[:, :n]
        self.proj.forward(ctx, x, proj)
        v_off = 2 * self.qk_width
        gate = proj[:, v_off + VW:v_off + 2 * VW]
        memory, maxima = cache.side("memory"), cache.side("max")
        where = (memory.slots, ctx.token_req, ctx.req_first_token)
        coef = ctx.ws.flat("mlstm_coef", 4 * T * H, torch.float32)
        tiled = ctx.n_portion > 0 and ctx.portion_tiles is not None and ops.mlstm_chunks_supported(x.dtype, self.dim)
        if ctx.n_portion == 0:       # a row a request: the gates' products and the maximum's step in one launch
            ops.label(self.name + ".gates", 4.0 * T * H * self.width, es * (T + 2 * H) * self.width + 24.0 * T * H)
            ops.mlstm_gates_single(x, self.gates.weight, self.gates.bias, self.gate_cap, maxima.state, *where, coef, H, ctx.stream)
        else:
            raw = ctx.ws.get("mlstm_raw", T, (2 * H + 7) // 8 * 8, torch.float32)[:, :2 * H]
            self.gates.forward(ctx, x, raw)
            ops.label(self.name + ".gates", 60.0 * T * H, 24.0 * T * H)
            ops.mlstm_gates(raw, H, self.gate_cap, maxima.state, *where, coef, H, ctx.stream, tiled=tiled)
        g = ctx.ws.get("mlstm_gated", T, (VW + 7) // 8 * 8, x.dtype)[:, :VW]
        cost = (6.0 * T * (VW + H) * self.dim, es * T * (v_off + VW) + 16.0 * T * H + 8.0 * min(T, ctx.n_requests) * (VW + H) * self.dim)
        fused = tiled and ctx.n_single == 0 and ops.mlstm_chunks_gated(self.dim, self.vdim)      # the tiles' own kernel finishes its rows
        o = None if fused else ctx.ws.get("mlstm_o", T, VW, torch.float32)
        den = None if fused else ctx.ws.flat("mlstm_den", T * H, torch.float32)
        heads = (proj, 0, self.qk_width, v_off, self.dim ** -0.5, coef, memory.state)
        if tiled:
            scratch = ctx.ws.flat("mlstm_states", ops.mlstm_chunks_scratch(T, ctx.n_requests, H, self.dim, self.vdim), torch.float32)
            ops.label(self.name + ".memory", cost[0], cost[1] + (2.0 * es if fused else 4.0) * T * VW)
            ops.mlstm_chunks(*heads, *where, ctx.req_first_position, ctx.portion_tiles, ctx.n_portion_tiles, scratch, H, ctx.stream,
                             **(dict(gate=gate, weight=self.norm_w, gated=g, eps=self.eps) if fused else dict(out=o, den=den)))
            if fused:
                return g
        if not tiled or ctx.n_single:
            ops.label(self.name + ".memory", cost[0], cost[1] + 4.0 * T * VW)
            ops.mlstm_scan(*heads, *where, o, den, H, ctx.stream, max_run=1 if tiled else 0)
        ops.label(self.name + ".norm", 10.0 * T * VW, (4.0 + 2 * es) * T * VW)
        ops.mlstm_finish(o, den, coef, self.norm_w, gate, g, H, self.eps, ctx.token_req, ctx.stream)
        return g

    def mix(self, ctx, x, cache, tag: str = "mix_out"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


class RGLRUMixer(Mixer):
    """A recurrent block of two branches of ``inner`` columns: ``y = gelu_tanh(W_y x + b)`` and ``u``, a short causal
    convolution with bias (``<name>.conv`` ``[inner, taps]``, ``<name>.conv.b``; no activation) of ``W_x x + b``, through a
    real-gated linear recurrent unit.  ``u`` is cut into ``blocks`` equal parts with square matrices of their own:
    ``r = sigmoid(ra_b u_b + ra.b_b)``, ``i = sigmoid(ri_b u_b + ri.b_b)``; per channel ``log a = -8 r softplus(lam)``,
    ``S <- a S + sqrt(1 - a^2) i u``; ``<name>.o`` of ``S * y``.  Gates, decays and the state are float32 (the gates'
    products: float32 sums, left in float32)."""
    replayable = True
    kernel_libs = ("recurrent", "rglru", "latent")

    def __init__(self, name: str, width: int, inner: int, blocks: int, taps: int, init: Init = Init()):
        if blocks < 1 or inner % blocks:
            raise ValueError(f"{name}: {inner} channels in {blocks} equal parts")
        if not 1 <= taps <= 9:
            raise ValueError(f"{name}: a convolution of {taps} taps (1 to 9)")
        self.name, self.width, self.inner, self.blocks, self.taps = name, width, inner, blocks, taps
        self.block = inner // blocks
        self.inner_p = (inner + 7) // 8 * 8
        self.proj = FusedLinear(f"{name}.yx", width, [(f"{name}.y", inner), (f"{name}.x", inner)], init=init,
                                biases={f"{name}.y": f"{name}.y.b", f"{name}.x": f"{name}.x.b"}, bias_init=Init(0.0, 0.1))
        self.out = Linear(f"{name}.o", inner, width, bias=False, weight_suffix="", init=Init(0.0, inner ** -0.5))
        self._no_state = None

    def children(self):
        return (self.proj, self.out)

    def cache_spec(self):
        spec = {"unit": StateSpec((self.inner,))}
        if self.taps > 1:
            spec["conv"] = StateSpec((self.taps - 1, self.inner))
        return spec

    def param_specs(self) -> List[ParamSpec]:
        n, W, B, b = self.name, self.inner, self.blocks, self.block
        gate = Init(0.0, b ** -0.5)
        return [ParamSpec(f"{n}.conv", (W, self.taps), VECTOR, Init(0.0, 0.4)), ParamSpec(f"{n}.conv.b", (W,), VECTOR, Init(0.0, 0.1)),
                ParamSpec(f"{n}.ra", (B, b, b), MATRIX, gate), ParamSpec(f"{n}.ra.b", (B, b), VECTOR, Init(0.0, 0.1)),
                ParamSpec(f"{n}.ri", (B, b, b), MATRIX, gate), ParamSpec(f"{n}.ri.b", (B, b), VECTOR, Init(0.0, 0.1)),
                ParamSpec(f"{n}.lam", (W,), VECTOR, Init(-4.0, 1.0))]

    def bind(self, tensors, dtype, device) -> None:
        n = self.name
        self.conv_w, self.conv_b = tensors[f"{n}.conv"].contiguous(), tensors[f"{n}.conv.b"].contiguous()
        self.conv_wt = self.conv_w.t().contiguous()
        # [blocks, 2 * block, block]: a part's recurrence gate, then its input gate, as one product per part
        self.w_gates = torch.cat([tensors[f"{n}.ra"], tensors[f"{n}.ri"]], dim=1).contiguous()
        self.r_bias, self.i_bias = (tensors[f"{n}.{t}.b"].reshape(-1).contiguous() for t in ("ra", "ri"))
        lam = tensors[f"{n}.lam"].double()
        self.decay = (-8.0 * torch.logaddexp(lam, torch.zeros_like(lam))).float().contiguous()
        self._no_state = torch.zeros((1, 0, self.inner), dtype=torch.float32, device=device)

    def _gated(self, ctx, x, cache):
        T, W, es = x.shape[0], self.inner, x.element_size()
        yx = ctx.ws.get("rglru_yx", T, 2 * self.inner_p, x.dtype)[:, :2 * W]
        self.proj.forward(ctx, x, yx)
        y, xb = yx[:, :W], yx[:, W:]
        u = ctx.ws.get("rglru_u", T, self.inner_p, x.dtype)[:, :W]
        state, slots = (cache.side("conv").state, cache.side("conv").slots) if self.taps > 1 else (self._no_state, ctx._slots)
        ops.label(self.name + ".conv", 2.0 * self.taps * T * W, 2.0 * es * T * W)
        ops.conv_silu(xb, self.conv_w, self.conv_b, state, slots, ctx.positions, ctx.token_req, ctx.req_first_token,
                      ctx.req_first_position, u, ctx.stream, weight_by_tap=self.conv_wt, activation=False)
        gates = ctx.ws.get("rglru_gates", T, 2 * W, torch.float32)
        ops.label(self.name + ".gates", 4.0 * T * W * self.block, es * (T * W + 2 * W * self.block) + 8.0 * T * W)
        ops.head_linear(u, self.block, self.w_gates, gates, 2 * self.block, ctx.stream, token_req=ctx.token_req)
        unit = cache.side("unit")
        out = ctx.ws.get("rglru_out", T, self.inner_p, x.dtype)[:, :W]
        ops.label(self.name + ".unit", 30.0 * T * W, (8.0 + 3 * es) * T * W + 8.0 * min(T, ctx.n_requests) * W)
        ops.rglru_scan(gates, self.r_bias, self.i_bias, self.decay, u, y, unit.state, unit.slots, ctx.token_req,
                       ctx.req_first_token, out, self.block, ctx.stream, singles=ctx.n_single > 0, portions=ctx.n_portion > 0)
        return out

    def mix(self, ctx, x, cache, tag: str = "mix_out"):
        g = self._gated(ctx, x, cache)
        return self.out.forward(ctx, g, ctx.ws.get(tag, x.shape[0], self.width, torch.float32))

    def forward(self, ctx, x, residual, cache):
        return self.out.forward(ctx, self._gated(ctx, x, cache), residual, residual=residual)


register_part("mixer", "mlstm", MLSTMMixer)
register_part("mixer", "retention", RetentionMixer)
register_part("mixer", "rglru", RGLRUMixer)
register_part("mixer", "mamba2", Mamba2Mixer)
register_part("mixer", "wkv", WKVMixer)
register_part("mixer", "gated_delta", GatedDeltaMixer)
