"""A plain, slow Vobusun: whole sequences through straightforward torch code, one function per mechanism, written
from the design's equations and sharing nothing with the package.  ``weights``: tensor name -> tensor as stored."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def angles(n, rot, dtype):
    """(cos, sin) of every position's angles, ``[n, dims / 2]``."""
    i = torch.arange(rot["dims"] // 2, dtype=torch.float64)
    f = float(rot["base"]) ** (-2.0 * i / max(rot["dims"], 1))
    a = torch.arange(n, dtype=torch.float64)[:, None] * f[None, :]
    return torch.cos(a).to(dtype), torch.sin(a).to(dtype)


def turn_halves(x, cos, sin, dims):
    """``x [T, heads, d]``: the first ``dims`` of every head turned, pairs ``(i, i + dims / 2)``."""
    out = x.clone()
    n = dims // 2
    a, b = x[..., :n], x[..., n:dims]
    c, s = cos[:, None, :], sin[:, None, :]
    out[..., :n] = a * c - b * s
    out[..., n:dims] = b * c + a * s
    return out


def turn_neighbours(x, cos, sin, dims):
    """The same with pairs ``(2i, 2i + 1)``."""
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    c, s = cos[:, None, :], sin[:, None, :]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def embedding(tokens, w, config, dtype):
    """Scaled token rows plus the row of the pair (token before, token), normed."""
    x = w["embed"].to(dtype)[tokens] * config["embedding"]["scale"]
    b = config["embedding"].get("bigram")
    if b:
        rows = []
        for t, tok in enumerate(tokens.tolist()):
            rows.append(b["buckets"] if t == 0 else (tokens[t - 1].item() * b["mul_prev"] + tok * b["mul_cur"]) % b["buckets"])
        x = x + w["bigram"].to(dtype)[torch.tensor(rows)]
    return rms(x, config["norm"]["eps"]) * w["embed.norm"].to(dtype)


def retention(h, w, name, m, eps):
    """Token by token: ``S <- decay S + k v^T``, ``o = S^T q``."""
    T, dt = h.shape[0], h.dtype
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[f"{name}.{n}"].to(dt).T).view(T, H, -1) for n in "qkv")
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    cos, sin = angles(T, rot, dt)
    q = turn_halves(q, cos, sin, rot["dims"])
    k = turn_halves(k, cos, sin, rot["dims"]) * d ** -0.5
    decay = torch.tensor(m["decay"], dtype=dt)[:, None, None]
    S = torch.zeros(H, d, e, dtype=dt)
    o = torch.zeros(T, H, e, dtype=dt)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(dim=1)
    gate = h @ w[name + ".g"].to(dt).T
    return (rms(o, eps).reshape(T, H * e) * gate * torch.sigmoid(gate)) @ w[name + ".o"].to(dt).T


def latent_attention(h, w, name, m, eps):
    T, dt = h.shape[0], h.dtype
    H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ w[name + ".dq"].to(dt).T, eps) * w[name + ".dq.norm"].to(dt)
    q = (cq @ w[name + ".uq"].to(dt).T).view(T, H, d + r)
    down = h @ w[name + ".dkv"].to(dt).T
    c = rms(down[:, :R], eps) * w[name + ".dkv.norm"].to(dt)
    cos, sin = angles(T, m["rot"], dt)
    k_turned = turn_neighbours(down[:, None, R:], cos, sin, r)[:, 0]
    q_turned = turn_neighbours(q[:, :, d:], cos, sin, r)
    keys = (c @ w[name + ".uk"].to(dt).T).view(T, H, d)
    values = (c @ w[name + ".uv"].to(dt).T).view(T, H, e)
    gate = torch.sigmoid(h @ w[name + ".g"].to(dt).T)
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    seen = (back >= 0) & (back < m["mask"]["size"])
    heads = []
    for a in range(H):
        s = (q[:, a, :d] @ keys[:, a].T + q_turned[:, a] @ k_turned.T) * m["scale"]
        heads.append(torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ values[:, a] * gate[:, a:a + 1])
    return torch.cat(heads, dim=-1) @ w[name + ".o"].to(dt).T


def short_convolution(u, taps_weight, bias):
    """``y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j)``, zeros before the start."""
    T, C = u.shape
    taps = taps_weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u])
    y = bias.to(u.dtype)[None, :].repeat(T, 1)
    for j in range(taps):
        y = y + padded[j:j + T] * taps_weight[:, j].to(u.dtype)[None, :]
    return y


def gates_by_block(u, weight, bias):
    """``sigmoid(weight[b] u_b + bias[b])`` for every equal part ``u_b`` of ``u``."""
    n, size = weight.shape[0], weight.shape[1]
    parts = [u[:, b * size:(b + 1) * size] @ weight[b].to(u.dtype).T + bias[b].to(u.dtype) for b in range(n)]
    return torch.sigmoid(torch.cat(parts, dim=-1))


def rglru(h, w, name, m, eps):
    T, dt = h.shape[0], h.dtype
    f = lambda s: w[f"{name}.{s}"].to(dt)
    y = gelu_tanh(h @ f("y").T + f("y.b"))
    u = short_convolution(h @ f("x").T + f("x.b"), f("conv"), f("conv.b"))
    r = gates_by_block(u, f("ra"), f("ra.b"))
    i = gates_by_block(u, f("ri"), f("ri.b"))
    log_a = -8.0 * r * torch.nn.functional.softplus(f("lam"))
    a = torch.exp(log_a)
    x = torch.sqrt(1.0 - a * a) * i * u
    S = torch.zeros(m["width"], dtype=dt)
    out = torch.zeros(T, m["width"], dtype=dt)
    for t in range(T):
        S = a[t] * S + x[t]
        out[t] = S
    return (out * y) @ f("o").T


def bounded_unit(h, w, name, limit):
    dt = h.dtype
    g = (h @ w[name + ".gate"].to(dt).T).clamp(max=limit)
    u = (h @ w[name + ".up"].to(dt).T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[name + ".down"].to(dt).T


MIXERS = {"retention": retention, "latent_attention": latent_attention, "rglru": rglru}


def read_streams(x, weights):
    """``x [streams, T, D]`` -> one row per token, a weighted sum over the streams."""
    return (x * weights.to(x.dtype)[:, None, None]).sum(dim=0)


def mix_streams(x, mix, out, y, m):
    """Every new stream ``t`` from all old ones: ``sum_s mix[s, t] x_s + m out[t] y``."""
    new = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for s in range(x.shape[0]):
            new[t] += mix[s, t].to(x.dtype) * x[s]
        new[t] += m * out[t].to(x.dtype) * y
    return new


def layers(config, w, tokens, dtype=torch.float64):
    """The sum of the streams after every layer, [layers, T, width], and the logits [T, vocab]."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, m = config["norm"]["eps"], config["residual_mult"]
    e = embedding(tokens, w, config, dtype)
    several = config.get("streams") is not None
    x = torch.stack([e] * (config["streams"] if several else 1))
    one = torch.ones(1)
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{layer.get('weights_of', i)}"
        sub = [lambda z: MIXERS[layer["type"]](z, w, p + ".mix", layer["mixer"], eps)]
        if layer.get("mlp") is not None:
            sub.append(lambda z: bounded_unit(z, w, p + ".mlp", layer["mlp"]["limit"]))
        for n, f in enumerate(sub, start=1):
            hc = f"{p}.hc{n}"
            u = read_streams(x, w[hc + ".in"] if several else one)
            y = f(rms(u, eps) * w[f"{p}.norm{n}"].to(dtype))
            x = mix_streams(x, w[hc + ".mix"], w[hc + ".out"], y, m) if several else x + m * y
        after.append(x.sum(dim=0))
    x = x.sum(dim=0)
    logits = (rms(x, eps) * w["final.norm"].to(dtype)) @ w["head"].to(dtype).T
    return torch.stack(after), logits


def forward(config, w, tokens, dtype=torch.float64):
    return layers(config, w, tokens, dtype)[1]
