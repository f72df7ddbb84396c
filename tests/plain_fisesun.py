"""A plain, slow Fisesun: whole sequences through straightforward torch code, one function per mechanism, written
from the design's equations and sharing nothing with the package.  ``weights``: tensor name -> tensor as stored."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def frequencies(rot):
    """Angle per position of every pair; with ``scaling`` long wavelengths are stretched by ``factor``, short ones kept, and
    those between blended linearly in (original length / wavelength)."""
    out = []
    s = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        if s:
            length = 2.0 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def turn(x, rot):
    """``x [T, heads, d]``: the first ``dims`` of every head turned by the row's number, pairs ``(i, i + dims / 2)``."""
    n = rot["dims"] // 2
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def visible(T, mask):
    """``[query, key]``: the last ``size`` positions, and the first ``keep_first`` of the sequence."""
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    if not mask:
        return back >= 0
    return (back >= 0) & ((back < mask["size"]) | (i[None, :] < mask.get("keep_first", 0)))


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, name, m, eps, shared):
    """``shared``: a dictionary that lives as long as the pass; the first layer that mixes values leaves its own there."""
    T, dt = h.shape[0], h.dtype
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (rms(h @ w[name + ".q"].to(dt).T, eps) * w[name + ".q.norm"].to(dt)).view(T, H, d)
    k = (rms(h @ w[name + ".k"].to(dt).T, eps) * w[name + ".k.norm"].to(dt)).view(T, G, d)
    v = h @ w[name + ".v"].to(dt).T
    if m.get("v_mix"):
        if "v_first" not in shared:
            shared["v_first"] = v
        else:
            v = mix_values(v, shared["v_first"], w[name + ".vmix"].to(dt))
    v = v.view(T, G, m["vdim"])
    if m.get("rot"):
        q, k = turn(q, m["rot"]), turn(k, m["rot"])
    seen = visible(T, m.get("mask"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = soft_cap((q[:, a] @ k[:, g].T) * m["scale"], m.get("softcap"))
        heads.append(torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g])
    return torch.cat(heads, dim=-1) @ w[name + ".o"].to(dt).T


def matrix_memory(q, k, v, i, f):
    """The recurrence token by token: ``q, k [T, H, K]``, ``v [T, H, V]``, logarithms of the input and forget gates
    ``i, f [T, H]``.  ``S`` and ``n`` are kept divided by ``exp(m)``, m the running maximum (0 at the start)."""
    T, H, K = q.shape
    S, n = torch.zeros(H, K, v.shape[2], dtype=q.dtype), torch.zeros(H, K, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / size[:, None]
    return out


def mlstm(h, w, name, m, eps, shared=None):
    T, dt = h.shape[0], h.dtype
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[name + ".q"].to(dt).T).view(T, H, d) * d ** -0.5
    k = (h @ w[name + ".k"].to(dt).T).view(T, H, d)
    v = (h @ w[name + ".v"].to(dt).T).view(T, H, e)
    i = soft_cap(h @ w[name + ".i"].to(dt).T + w[name + ".i.b"].to(dt), cap)
    f = torch.nn.functional.logsigmoid(soft_cap(h @ w[name + ".f"].to(dt).T + w[name + ".f.b"].to(dt), cap))
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * e)
    return (o * w[name + ".norm"].to(dt) * torch.sigmoid(h @ w[name + ".g"].to(dt).T)) @ w[name + ".o"].to(dt).T


MIXERS = {"attention": attention, "mlstm": mlstm}


def gated_feed_forward(h, w, name):
    dt = h.dtype
    return (silu(h @ w[name + ".gate"].to(dt).T) * (h @ w[name + ".up"].to(dt).T)) @ w[name + ".down"].to(dt).T


def experts_by_token(h, tokens, w, name, top):
    """Every token's experts from the table's row of its id, each with weight ``1 / top``."""
    out = torch.zeros_like(h)
    table = w[name + ".table"].long()
    for t, tok in enumerate(tokens.tolist()):
        for c in range(top):
            out[t] += gated_feed_forward(h[t:t + 1], w, f"{name}.e{int(table[tok, c])}")[0] / top
    return out


def feed_forward(h, tokens, w, name, mlp):
    if mlp["kind"] == "dense":
        return gated_feed_forward(h, w, name)
    y = experts_by_token(h, tokens, w, name, mlp["router"]["top"])
    if mlp.get("shared"):
        y = y + gated_feed_forward(h, w, name + ".shared")
    return y


def layers(config, w, tokens, dtype=torch.float64):
    """The residual stream after every layer, [layers, T, width], and the logits [T, vocab]."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = w["embed"].to(dtype)[tokens] * config["embedding"]["scale"]
    after, shared = [], {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](x, w, p + ".mix", layer["mixer"], eps, shared)
        x = x + rms(y, eps) * w[p + ".norm1"].to(dtype)
        if layer.get("mlp"):
            y = feed_forward(x, tokens, w, p + ".mlp", layer["mlp"])
            x = x + rms(y, eps) * w[p + ".norm2"].to(dtype)
        after.append(x)
    logits = (rms(x, eps) * w["final.norm"].to(dtype)) @ w["head"].to(dtype).T
    return torch.stack(after), soft_cap(logits, config.get("logit_softcap"))


def forward(config, w, tokens, dtype=torch.float64):
    return layers(config, w, tokens, dtype)[1]
