"""The kernels Vobusun brought or widened, each alone against the plain implementation's functions in float64: the embedding
of token pairs with its state; the read and the update of a residual of several streams; retention token by token and in
tiles on tensor cores (with the heads' norm and gate, with states of large values, runs beside single rows); the real-gated
linear recurrent unit; the RMS norm of rows in the run's dtype and without a weight; the latent row beside queries in a
buffer of their own."""
import math

import pytest
import torch

import plain_vobusun as plain
from test_nufetar_kernels_gpu import DEV, i32

pytestmark = pytest.mark.gpu

ACT = [torch.float32, torch.bfloat16]


def stream():
    from mlx_lm_b200 import ops
    return ops.current_stream()


def layout(runs, gap=3):
    """Rows of a step for runs of the given lengths, ``gap`` filler rows behind each: token_req, first rows (one more than
    there are runs), total."""
    req, first = [], []
    for r, n in enumerate(runs):
        first.append(len(req))
        req += [r] * n + [-1] * gap
    return req, first + [len(req)], len(req)


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("D,S,muls", [(64, 3, (211, 17, 5)), (50, 1, (7, 3, 2)), (136, 5, (1000003, 900001, 2000003)), (8, 2, (1, 5, 7))])
def test_embedding_of_token_pairs(act, D, S, muls):
    """Three steps of two requests in slots of their own: the pair's row at the start, inside a run, and across steps."""
    from mlx_lm_b200 import ops
    torch.manual_seed(D)
    V, (buckets, mp, mc), scale, eps = 301, muls, 2.5, 1e-5
    buckets = min(buckets, 5000)
    table, pairs = torch.randn(V, D).to(act), (2 * torch.randn(buckets + 1, D)).to(act)
    weight = torch.randn(D)
    last = torch.full((4, 1), 77.0, device=DEV)
    seqs = [torch.randint(0, V, (40,)).tolist(), torch.randint(0, V, (40,)).tolist()]
    cfg = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}, "norm": {"eps": eps}}
    w = {"embed": table, "bigram": pairs, "embed.norm": weight}
    want = [plain.embedding(torch.tensor(s), w, cfg, torch.float64) for s in seqs]
    at, status = [0, 0], torch.zeros(1, dtype=torch.int32, device=DEV)
    for runs in ((5, 1), (1, 30), (34, 9)):
        req, first, T = layout(runs)
        toks, pos = [0] * T, [0] * T
        for r, n in enumerate(runs):
            toks[first[r]:first[r] + n] = seqs[r][at[r]:at[r] + n]
            pos[first[r]:first[r] + n] = range(at[r], at[r] + n)
        out = torch.full((T, S * D), 9.0, device=DEV)
        ops.embed_pairs(i32(toks), i32(pos), i32(req), i32(first), i32([3, 1]), table.to(DEV), pairs.to(DEV), last, weight.to(DEV),
                        out, S, status, stream(), scale=scale, buckets=buckets, mul_prev=mp, mul_cur=mc, eps=eps)
        got = out.cpu().double().view(T, S, D)
        for r, n in enumerate(runs):
            ref = want[r][at[r]:at[r] + n][:, None, :].expand(n, S, D)
            assert float((got[first[r]:first[r] + n] - ref).abs().max()) < 1e-5
            at[r] += n
            assert float(last[(3, 1)[r], 0]) == seqs[r][at[r] - 1]
        assert float(last[0, 0]) == 77.0 and float(last[2, 0]) == 77.0
    assert int(status) == 0
    # a token outside the vocabulary is reported and gives zeros
    ops.embed_pairs(i32([V, 1]), i32([0, 1]), i32([0, 0]), i32([0, 2]), i32([0]), table.to(DEV), pairs.to(DEV), last, weight.to(DEV),
                    out[:2], S, status, stream(), scale=scale, buckets=buckets, mul_prev=mp, mul_cur=mc, eps=eps)
    assert int(status) == ops.ST_TOKEN_RANGE and float(out[0].abs().max()) == 0.0


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("D", [64, 50, 1032, 2048, 7])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 8, 16])
def test_streams_are_read_and_updated(act, D, S):
    from mlx_lm_b200 import ops
    torch.manual_seed(D + S)
    T, eps = 9, 1e-5
    x0, y = torch.randn(T, S * D), torch.randn(T, D)
    mix, w_out, w_in, weight = torch.randn(S, S), torch.randn(S), torch.randn(S), torch.randn(D)
    req = [0] * T
    req[4] = -1
    xs = x0.double().view(T, S, D).transpose(0, 1)
    read = lambda xx: plain.rms(plain.read_streams(xx, w_in), eps) * weight.double()
    x, h = x0.clone().to(DEV), torch.zeros(T, D, dtype=act, device=DEV)
    d = lambda t: t.to(DEV)
    ops.streams_read(x, S, d(w_in), d(weight), h, eps, stream())
    tol = 2e-6 if act == torch.float32 else 5e-3
    assert float((h.cpu().double() - read(xs)).abs().max()) < tol * max(1.0, float(read(xs).abs().max()))
    rows = [7, 0, 0, 8]
    g = torch.zeros(4, D, dtype=act, device=DEV)
    ops.streams_read(x, S, d(w_in), d(weight), g, eps, stream(), rows=i32(rows))
    assert torch.equal(g.cpu(), h.cpu()[rows])
    new = plain.mix_streams(xs, mix, w_out, y.double(), 1.0)
    h.fill_(5.0)
    ops.streams_update(x, d(y), S, d(mix), d(w_out), stream(), token_req=i32(req), nxt=(d(w_in), d(weight)), next_out=h, eps=eps)
    live = [t for t in range(T) if t != 4]
    got = x.cpu().double().view(T, S, D).transpose(0, 1)
    assert float((got - new)[:, live].abs().max()) < 1e-5
    assert torch.equal(x.cpu()[4], x0[4]) and float(h.cpu()[4].float().min()) == 5.0
    assert float((h.cpu().double() - read(new))[live].abs().max()) < tol * max(1.0, float(read(new).abs().max()))
    x2 = x0.clone().to(DEV)                            # without a reader: the same streams
    ops.streams_update(x2, d(y), S, d(mix), d(w_out), stream(), token_req=i32(req))
    assert torch.equal(x2.cpu(), x.cpu())


def retention_inputs(act, runs, H, K, V, seed):
    g = torch.Generator().manual_seed(seed)
    req, first, T = layout(runs)
    n = (2 * H * K + 2 * H * V + 7) // 8 * 8
    proj = torch.randn(T, n, generator=g).to(act)
    state = torch.randn(len(runs) + 2, H, V, K, generator=g) * 3.0
    slots = list(range(len(runs), 0, -1))              # slot 0 and the last one belong to nobody
    start = [7 * r * r for r in range(len(runs))]
    pos = [0] * T
    for r, m in enumerate(runs):
        pos[first[r]:first[r] + m] = range(start[r], start[r] + m)
    return req, first, T, proj, state, slots, start, pos


def retention_reference(proj, first, runs, start, state, slots, H, K, V, half, base, decay):
    o, new = torch.zeros(proj.shape[0], H * V, dtype=torch.float64), state.double().clone()
    for r, m in enumerate(runs):
        rows = proj[first[r]:first[r] + m].double()
        q, k, v = rows[:, :H * K].view(m, H, K), rows[:, H * K:2 * H * K].view(m, H, K), rows[:, 2 * H * K:2 * H * K + H * V].view(m, H, V)
        if half:
            cos, sin = plain.angles(start[r] + m, {"dims": 2 * half, "base": base}, torch.float64)
            q, k = (plain.turn_halves(t, cos[start[r]:], sin[start[r]:], 2 * half) for t in (q, k))
        k = k * K ** -0.5
        S = new[slots[r]].transpose(1, 2).clone()
        for t in range(m):
            S = decay.double()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[first[r] + t] = (S * q[t][:, :, None]).sum(1).reshape(-1)
        new[slots[r]] = S.transpose(1, 2)
    return o, new


RETENTION = [(3, 16, 24, 4, [0.75, 0.9375, 0.99]), (1, 64, 128, 32, [0.998]), (2, 32, 32, 16, [0.0, 1.0]), (2, 40, 16, 20, [0.5, 0.9]),
             (1, 128, 64, 64, [0.97]), (1, 192, 80, 32, [0.995]), (2, 10, 7, 3, [0.8, 0.99]), (1, 24, 200, 0, [0.9995]), (1, 256, 72, 128, [0.9])]


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("H,K,V,half,decay", RETENTION)
def test_retention_token_by_token(act, H, K, V, half, decay):
    from mlx_lm_b200 import ops
    runs = (1, 2, 40, 1, 17)
    req, first, T, proj, state, slots, start, pos = retention_inputs(act, runs, H, K, V, K + V)
    decay = torch.tensor(decay, dtype=torch.float32)
    base = 1000.0
    freq = torch.tensor([base ** (-2.0 * i / (2 * half)) for i in range(half)], dtype=torch.float32).to(DEV) if half else None
    o = torch.full((T, H * V), 4.0, device=DEV)
    st = state.clone().to(DEV)
    go = lambda max_run: ops.retention_scan(proj.to(DEV), 0, H * K, 2 * H * K, freq, K ** -0.5, decay.to(DEV), st, i32(slots), i32(pos),
                                            i32(req), i32(first), o, H, stream(), max_run=max_run)
    go(0)
    want, new = retention_reference(proj, first, runs, start, state, slots, H, K, V, half, base, decay)
    live = [t for t in range(T) if req[t] >= 0]
    scale = float(want.abs().max())
    assert float((o.cpu().double() - want)[live].abs().max()) < 3e-6 * scale
    assert float((st.cpu().double() - new).abs().max()) < 3e-6 * float(new.abs().max())
    assert torch.equal(st.cpu()[0], state[0]) and torch.equal(st.cpu()[-1], state[-1])
    # only single rows: the others' rows and states stay as they are
    st.copy_(state)
    o.fill_(4.0)
    go(1)
    single = [first[0], first[3]]
    assert float((o.cpu().double() - want)[single].abs().max()) < 3e-6 * scale
    others = [t for t in range(T) if t not in single]
    assert float((o.cpu()[others] - 4.0).abs().max()) == 0.0
    assert all(torch.equal(st.cpu()[slots[r]], state[slots[r]]) for r in (1, 2, 4))


@pytest.mark.parametrize("tile_rows", [128, 64])
@pytest.mark.parametrize("H,K,V,half,decay", RETENTION)
def test_retention_in_tiles(H, K, V, half, decay, tile_rows):
    """Runs of two rows, of one tile, of a tile and a row, of several tiles; single rows are left alone.  The state's values
    and one loud key are far larger than the rest: what enters the products as two bfloat16 halves keeps float32's
    accuracy but for a few units in the sixteenth bit, a bfloat16 rounding would show a hundred times larger."""
    from mlx_lm_b200 import ops
    runs = (2, 1, 128, 129, 300, 64, 65, 15)
    req, first, T, proj, state, slots, start, pos = retention_inputs(torch.bfloat16, runs, H, K, V, K + V + 1)
    proj[first[4] + 3, H * K:2 * H * K] *= 16.0
    decay = torch.tensor(decay, dtype=torch.float32)
    base = 300.0
    freq = torch.tensor([base ** (-2.0 * i / (2 * half)) for i in range(half)], dtype=torch.float32).to(DEV) if half else None
    powers = (decay.double()[:, None] ** torch.arange(ops.RETENTION_TILE + 1, dtype=torch.float64)[None, :]).float().to(DEV)
    tiles = []
    for r, n in enumerate(runs):
        if n > 1:
            tiles += [(first[r] + a, min(tile_rows, n - a), r, start[r] + a) for a in range(0, n, tile_rows)]
    tiles.sort(key=lambda t: -(t[3] + t[1]))
    tiles.append((0, 0, 0, 0))
    scratch = torch.full((ops.retention_chunks_scratch(T, len(runs), H, K, V, tile_rows),), math.nan, device=DEV)
    args = lambda: (proj.to(DEV), 0, H * K, 2 * H * K, freq, K ** -0.5, powers, st, i32(slots), i32(req), i32(first), i32(start),
                    i32([x for t in tiles for x in t]), len(tiles), scratch, H, stream())
    want, new = retention_reference(proj, first, runs, start, state, slots, H, K, V, half, base, decay)
    live = [t for t in range(T) if req[t] >= 0 and t != first[1]]
    st = state.clone().to(DEV)
    o = torch.full((T, H * V), 4.0, device=DEV)
    ops.retention_chunks(*args(), out=o, tile_rows=tile_rows)
    scale = float(want.abs().max())
    assert float((o.cpu().double() - want)[live].abs().max()) < 4e-5 * scale
    idle = [t for t in range(T) if t not in live]
    assert float((o.cpu()[idle] - 4.0).abs().max()) == 0.0
    for r, n in enumerate(runs):
        if n > 1:
            assert float((st.cpu()[slots[r]].double() - new[slots[r]]).abs().max()) < 4e-5 * float(new[slots[r]].abs().max())
        else:
            assert torch.equal(st.cpu()[slots[r]], state[slots[r]])
    assert torch.equal(st.cpu()[0], state[0]) and torch.equal(st.cpu()[-1], state[-1])
    if not ops.retention_chunks_gated(K, V):
        return
    # the heads' norm and the gate in the same kernel
    eps = 1e-5
    st.copy_(state)
    gated = torch.full((T, (H * V + 7) // 8 * 8), 6.0, dtype=torch.bfloat16, device=DEV)[:, :H * V]
    gate = proj[:, 2 * H * K + H * V:2 * H * K + 2 * H * V]
    ops.retention_chunks(*args(), gate=gate.to(DEV), gated=gated, eps=eps, tile_rows=tile_rows)
    gd = gate.double()
    ref = plain.rms(want.view(T, H, V), eps).reshape(T, H * V) * gd * torch.sigmoid(gd)
    assert float((gated.cpu().double() - ref)[live].abs().max()) < 5e-3 * float(ref.abs().max())
    assert float((gated.cpu().float()[idle] - 6.0).abs().max()) == 0.0


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("W,blocks", [(48, 3), (128, 1), (33, 3), (16, 4), (200, 2)])
def test_real_gated_linear_recurrent_unit(act, W, blocks):
    """Runs of one row, of less and more than a block walks at a time (256 rows), channels that hardly forget and channels
    that forget at once; the state carries on from what it was."""
    from mlx_lm_b200 import ops
    torch.manual_seed(W)
    runs = (1, 2, 600, 1, 256, 257, 9)
    req, first, T = layout(runs)
    n = W // blocks
    gates = torch.randn(T, 2 * W)
    u, y = torch.randn(T, W).to(act), torch.randn(T, W).to(act)
    br, bi, lam = torch.randn(W), torch.randn(W), torch.linspace(-12.0, 3.0, W)
    state = torch.randn(len(runs) + 2, W) * 2.0
    slots = list(range(len(runs), 0, -1))
    decay = (-8.0 * torch.nn.functional.softplus(lam.double())).float()
    pr = gates.double().view(T, blocks, 2, n)[:, :, 0].reshape(T, W) + br.double()
    pi = gates.double().view(T, blocks, 2, n)[:, :, 1].reshape(T, W) + bi.double()
    a = torch.exp(torch.sigmoid(pr) * decay.double())
    x = torch.sqrt(1 - a * a) * torch.sigmoid(pi) * u.double()
    want, new = torch.zeros(T, W, dtype=torch.float64), state.double().clone()
    for r, m in enumerate(runs):
        S = new[slots[r]]
        for t in range(first[r], first[r] + m):
            S = a[t] * S + x[t]
            want[t] = S * plain.gelu_tanh(y[t].double())
        new[slots[r]] = S
    st = state.clone().to(DEV)
    out = torch.full((T, W), 4.0, dtype=act, device=DEV)
    ops.rglru_scan(gates.to(DEV), br.to(DEV), bi.to(DEV), decay.to(DEV), u.to(DEV), y.to(DEV), st, i32(slots), i32(req), i32(first),
                   out, n, stream())
    live = [t for t in range(T) if req[t] >= 0]
    tol = 1e-5 if act == torch.float32 else 5e-3
    assert float((out.cpu().double() - want)[live].abs().max()) < tol * max(1.0, float(want.abs().max()))
    assert float((st.cpu().double() - new).abs().max()) < 1e-5 * float(new.abs().max())
    idle = [t for t in range(T) if req[t] < 0]
    assert float((out.cpu().float()[idle] - 4.0).abs().max()) == 0.0
    assert torch.equal(st.cpu()[0], state[0]) and torch.equal(st.cpu()[-1], state[-1])


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("D,groups,gate", [(96, 1, False), (40, 1, False), (700, 1, False), (192, 6, True), (50, 5, True), (1024, 8, True), (19, 1, False)])
def test_rms_norm_of_rows_in_the_runs_dtype_and_without_a_weight(act, D, groups, gate):
    from mlx_lm_b200 import ops
    torch.manual_seed(D)
    T, eps, pad = 23, 1e-5, (D + 7) // 8 * 8
    x, w, g = torch.randn(T, D), torch.randn(D), torch.randn(T, pad).to(act)[:, :D]
    for weight in (w, None):
        for xin in (x, x.to(act)):
            out = torch.zeros(T, pad, dtype=act, device=DEV)[:, :D]
            buf = torch.zeros(T, pad, dtype=xin.dtype, device=DEV)
            buf[:, :D] = xin.to(DEV)
            gd = torch.zeros(T, pad, dtype=act, device=DEV)
            gd[:, :D] = g.to(DEV)
            ops.rmsnorm(buf[:, :D], None if weight is None else weight.to(DEV), out, eps, stream(), groups=groups,
                        gate=gd[:, :D] if gate else None, gate_mode=ops.GATE_AFTER if gate else ops.GATE_NONE)
            ref = plain.rms(xin.double().view(T, groups, -1), eps).reshape(T, D)
            if weight is not None:
                ref = ref * weight.double()
            if gate:
                ref = ref * g.double() * torch.sigmoid(g.double())
            tol = 2e-6 if act == torch.float32 else 5e-3
            assert float((out.cpu().double() - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("act", ACT)
def test_latent_row_beside_queries_of_their_own(act):
    """Queries in another buffer than the down projection give the bits they give as columns of the same one."""
    from mlx_lm_b200 import ops
    torch.manual_seed(3)
    T, H, d, dr, R, page = 21, 3, 12, 8, 40, 16
    row = 48
    q, down = torch.randn(T, H * (d + dr)).to(act).to(DEV), torch.randn(T, R + dr).to(act).to(DEV)
    both = torch.cat([q, down], dim=1).contiguous()
    weight, status = torch.randn(R, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    freq = torch.tensor([100.0 ** (-2.0 * i / dr) for i in range(dr // 2)], dtype=torch.float32, device=DEV)
    res = []
    for proj, c_off, kw in ((both, H * (d + dr), {}), (down, 0, {"queries": q})):
        pool = torch.zeros(4, 1, page, row, dtype=act, device=DEV)
        q_lat = torch.zeros(T, H * (R + dr), device=DEV)
        ops.latent_prepare(proj, 0, c_off, H, d, dr, R, weight, 1e-5, freq, True, i32(range(5, 5 + T)), i32([0] * T), i32([2, 0, -1]).view(1, 3),
                           pool, True, q_lat, R + dr, status, stream(), **kw)
        res.append((pool.cpu(), q_lat.cpu()))
    assert torch.equal(res[0][0], res[1][0]) and torch.equal(res[0][1], res[1][1]) and int(status) == 0
    assert float(res[0][1].abs().max()) > 0 and float(res[0][0].float().abs().max()) > 0
