"""The kernels Fisesun brought or widened, each alone against the plain implementation's functions in float64: the matrix
memory's gates along runs of rows and for single rows, the recurrence token by token and in tiles on tensor cores (states and
keys of large values, runs beside single rows), the division with the heads' norm and gate; the stream's update through a norm
of a sum; the plan of experts named by a table; the cap on logits; queries, keys and values with mixed values."""
import math

import pytest
import torch

import plain_fisesun as plain
from test_nufetar_kernels_gpu import DEV, i32
from test_vobusun_kernels_gpu import layout, stream

pytestmark = pytest.mark.gpu

ACT = [torch.float32, torch.bfloat16]


# heads, key columns, value columns, cap, offset of the forget gates (large: hardly forgets; very negative: forgets at once)
MEMORY = [(3, 16, 24, 10.0, 3.0), (1, 64, 128, 12.0, 6.0), (2, 32, 32, 15.0, -9.0), (2, 40, 16, 4.0, 1.0), (1, 128, 64, 6.0, 5.0),
          (1, 192, 80, 8.0, 4.0), (2, 10, 7, 9.0, 2.0), (1, 24, 200, 12.0, 8.0), (1, 256, 72, 3.0, 2.0)]


def memory_inputs(act, runs, H, K, V, shift, seed):
    g = torch.Generator().manual_seed(seed)
    req, first, T = layout(runs)
    n = (2 * H * K + 2 * H * V + 7) // 8 * 8
    proj = torch.randn(T, n, generator=g).to(act)
    raw = torch.randn(T, 2 * H + 3, generator=g) * 3.0
    raw[:, H:2 * H] += shift
    R = len(runs)
    state = torch.randn(R + 2, H, V + 1, K, generator=g) * 3.0
    m0 = torch.randn(R + 2, H, generator=g) * 2.0
    slots = list(range(R, 0, -1))                      # slot 0 and the last one belong to nobody
    start = [7 * r * r for r in range(R)]
    return req, first, T, proj, raw, state, m0, slots, start


def memory_reference(proj, raw, first, runs, state, m0, slots, H, K, V, cap):
    """o (divided), the state and the maxima after the step, from the equations token by token."""
    o = torch.zeros(proj.shape[0], H, V, dtype=torch.float64)
    new, mx = state.double().clone(), m0.double().clone()
    i = plain.soft_cap(raw[:, :H].double(), cap)
    f = torch.nn.functional.logsigmoid(plain.soft_cap(raw[:, H:2 * H].double(), cap))
    for r, n in enumerate(runs):
        rows = proj[first[r]:first[r] + n].double()
        q, k = rows[:, :H * K].view(n, H, K) * K ** -0.5, rows[:, H * K:2 * H * K].view(n, H, K)
        v = rows[:, 2 * H * K:2 * H * K + H * V].view(n, H, V)
        S, nn, m = new[slots[r]][:, :V].transpose(1, 2).clone(), new[slots[r]][:, V].clone(), mx[slots[r]].clone()
        for t in range(n):
            a = first[r] + t
            nm = torch.maximum(f[a] + m, i[a])
            keep, take = torch.exp(f[a] + m - nm), torch.exp(i[a] - nm)
            m = nm
            S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
            nn = keep[:, None] * nn + take[:, None] * k[t]
            d = torch.maximum((nn * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            o[a] = (S * q[t][:, :, None]).sum(1) / d[:, None]
        new[slots[r]] = torch.cat([S.transpose(1, 2), nn[:, None]], dim=1)
        mx[slots[r]] = m
    return o.reshape(proj.shape[0], H * V), new, mx


def divided(o, den, coef, H):
    T = o.shape[0]
    em = coef.view(-1)[:4 * T * H].view(T, H, 4)[:, :, 3].cpu().double()
    d = torch.maximum(den.view(-1)[:T * H].view(T, H).cpu().double().abs(), em) + 1e-6
    return (o.cpu().double().view(T, H, -1) / d[:, :, None]).reshape(T, -1)


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("H,K,V,cap,shift", MEMORY + [(1, 300, 24, 7.0, 3.0)])
def test_memory_token_by_token(act, H, K, V, cap, shift):
    from mlx_lm_b200 import ops
    runs = (1, 2, 40, 1, 17, 300)
    req, first, T, proj, raw, state, m0, slots, start = memory_inputs(act, runs, H, K, V, shift, K + V)
    want, new, mx = memory_reference(proj, raw, first, runs, state, m0, slots, H, K, V, cap)
    m, st = m0.clone().to(DEV), state.clone().to(DEV)
    coef = torch.full((4 * T * H,), math.nan, device=DEV)
    where = (i32(slots), i32(req), i32(first))
    ops.mlstm_gates(raw.to(DEV), H, cap, m, *where, coef, H, stream())
    assert float((m.cpu().double() - mx).abs().max()) < 1e-4 and torch.equal(m.cpu()[0], m0[0]) and torch.equal(m.cpu()[-1], m0[-1])
    o, den = torch.full((T, H * V), 4.0, device=DEV), torch.full((T * H,), 5.0, device=DEV)
    go = lambda max_run: ops.mlstm_scan(proj.to(DEV), 0, H * K, 2 * H * K, K ** -0.5, coef, st, *where, o, den, H, stream(), max_run=max_run)
    go(0)
    live = [t for t in range(T) if req[t] >= 0]
    err = (divided(o, den, coef, H) - want)[live].abs().amax(1) / want[live].abs().amax(1).clamp(min=1.0)
    assert float(err.max()) < 3e-4, float(err.max())
    # the state is kept divided by exp(m): compare with the reference's, brought to the same maximum
    shift_m = torch.exp(mx - m.cpu().double())[:, :, None, None]
    assert float((st.cpu().double() - new * shift_m).abs().max()) < 1e-4 * float(new.abs().max())
    assert torch.equal(st.cpu()[0], state[0]) and torch.equal(st.cpu()[-1], state[-1])
    # only single rows: the others' rows and states stay as they are
    st.copy_(state)
    o.fill_(4.0)
    go(1)
    single = [first[0], first[3]]
    others = [t for t in range(T) if t not in single]
    assert float((o.cpu()[others] - 4.0).abs().max()) == 0.0 and float((o.cpu()[single] - 4.0).abs().min()) > 0.0
    assert all(torch.equal(st.cpu()[slots[r]], state[slots[r]]) for r in (1, 2, 4, 5))


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("H,D", [(3, 64), (1, 50), (8, 1032), (5, 7), (2, 2048)])
def test_gates_of_single_rows_with_their_products(act, H, D):
    """One launch for products, caps and the maximum's step gives what a product and ``mlstm_gates`` give; padding requests (no
    row, or a row that is nobody's) keep their maxima."""
    from mlx_lm_b200 import ops
    torch.manual_seed(H + D)
    T, cap = 7, 9.0
    req = [0, 1, 2, -1, 4, -1, -1]
    first = [0, 1, 2, 3, 4, 5, 6, T, T]                # request 7 has no row at all
    slots = [3, 5, 1, 0, 2, 0, 0, 0]
    x, w, b = torch.randn(T, D).to(act), (torch.randn(2 * H, D) * 2 * D ** -0.5).to(act), torch.randn(2 * H)
    m0 = torch.randn(6, H) * 2
    z = x.double() @ w.double().T + b.double()
    i, f = plain.soft_cap(z[:, :H], cap), torch.nn.functional.logsigmoid(plain.soft_cap(z[:, H:], cap))
    m, coef = m0.clone().to(DEV), torch.full((4 * T * H,), 7.0, device=DEV)
    ops.mlstm_gates_single(x.to(DEV), w.to(DEV), b.to(DEV), cap, m, i32(slots), i32(req), i32(first), coef, H, stream())
    got = coef.cpu().double().view(T, H, 4)
    for t in range(T):
        if req[t] < 0:
            assert float((got[t] - 7.0).abs().max()) == 0.0
            continue
        s = slots[req[t]]
        new = torch.maximum(f[t] + m0[s].double(), i[t])
        assert float((m.cpu()[s].double() - new).abs().max()) < 1e-5
        want = torch.stack([torch.exp(f[t] + m0[s].double() - new), torch.exp(i[t] - new), torch.exp(-new)], dim=-1)
        assert float(((got[t][:, [0, 1, 3]] - want) / want.clamp(min=1e-3)).abs().max()) < 1e-4
    assert torch.equal(m.cpu()[[0, 4]], m0[[0, 4]])


@pytest.mark.parametrize("tile_rows", [128, 64])
@pytest.mark.parametrize("H,K,V,cap,shift", MEMORY)
def test_memory_in_tiles(H, K, V, cap, shift, tile_rows):
    """Runs of two rows, of one tile, of a tile and a row, of many tiles (more than the gates' kernel walks at a time); single
    rows are left alone.  The state's values and one loud key are far larger than the rest: what enters the products as two
    bfloat16 halves keeps float32's accuracy but for a few units in the sixteenth bit."""
    from mlx_lm_b200 import ops
    runs = (2, 1, 128, 129, 1100, 64, 65, 15)
    req, first, T, proj, raw, state, m0, slots, start = memory_inputs(torch.bfloat16, runs, H, K, V, shift, K + V + 1)
    proj[first[4] + 3, H * K:2 * H * K] *= 16.0
    want, new, mx = memory_reference(proj, raw, first, runs, state, m0, slots, H, K, V, cap)
    tiles = []
    for r, n in enumerate(runs):
        if n > 1:
            tiles += [(first[r] + a, min(tile_rows, n - a), r, start[r] + a) for a in range(0, n, tile_rows)]
    tiles.sort(key=lambda t: -(t[3] + t[1]))
    tiles.append((0, 0, 0, 0))
    m, st = m0.clone().to(DEV), state.clone().to(DEV)
    coef = torch.full((4 * T * H,), math.nan, device=DEV)
    where = (i32(slots), i32(req), i32(first))
    ops.mlstm_gates(raw.to(DEV), H, cap, m, *where, coef, H, stream(), tiled=True, tile_rows=tile_rows)
    scratch = torch.full((ops.mlstm_chunks_scratch(T, len(runs), H, K, V, tile_rows),), math.nan, device=DEV)
    args = lambda: (proj.to(DEV), 0, H * K, 2 * H * K, K ** -0.5, coef, st, *where, i32(start), i32([x for t in tiles for x in t]),
                    len(tiles), scratch, H, stream())
    o, den = torch.full((T, H * V), 4.0, device=DEV), torch.full((T * H,), 5.0, device=DEV)
    ops.mlstm_chunks(*args(), out=o, den=den, tile_rows=tile_rows)
    live = [t for t in range(T) if req[t] >= 0 and t != first[1]]
    # measured against the size of what is summed: where n . q or o comes close to zero the quotient blows rounding up
    err = (divided(o, den, coef, H) - want)[live].abs().amax(1) / want[live].abs().amax(1).clamp(min=1.0)
    print(f"tiles {H} {K} {V}: {float(err.max()):.3g} (median {float(err.median()):.3g})")
    assert float(err.median()) < 2e-5 and float(err.max()) < 2e-3
    idle = [t for t in range(T) if t not in live]
    assert float((o.cpu()[idle] - 4.0).abs().max()) == 0.0
    scale = torch.exp(mx - m.cpu().double())[:, :, None, None]
    for r, n in enumerate(runs):
        s = slots[r]
        if n > 1:
            assert float((st.cpu()[s].double() - new[s] * scale[s]).abs().max()) < 1e-4 * float(new[s].abs().max())
        else:
            assert torch.equal(st.cpu()[s], state[s])
    assert torch.equal(st.cpu()[0], state[0]) and torch.equal(st.cpu()[-1], state[-1])
    # the division, the heads' norm and the gate: as a kernel of their own, and inside the tiles' kernel
    eps, weight = 1e-5, torch.randn(H * V)
    gate = proj[:, 2 * H * K + H * V:2 * H * K + 2 * H * V]
    ref = plain.rms(want.view(T, H, V), eps).reshape(T, H * V) * weight.double() * torch.sigmoid(gate.double())
    pad = (H * V + 7) // 8 * 8
    y = torch.full((T, pad), 6.0, dtype=torch.bfloat16, device=DEV)[:, :H * V]
    ops.mlstm_finish(o, den, coef, weight.to(DEV), gate.to(DEV), y, H, eps, where[1], stream())
    quiet = lambda got: float(((got.cpu().double() - ref)[live].abs() / ref[live].abs().clamp(min=1.0)).max())
    assert quiet(y) < 2e-2
    if not ops.mlstm_chunks_gated(K, V):
        return
    st.copy_(state)
    gated = torch.full((T, pad), 6.0, dtype=torch.bfloat16, device=DEV)[:, :H * V]
    ops.mlstm_chunks(*args(), gate=gate.to(DEV), weight=weight.to(DEV), gated=gated, eps=eps, tile_rows=tile_rows)
    assert quiet(gated) < 2e-2
    assert float((gated.cpu().float()[idle] - 6.0).abs().max()) == 0.0


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("H,V", [(3, 24), (1, 300), (2, 7), (4, 256)])
def test_memory_rows_are_divided_normed_and_gated(act, H, V):
    """Both sides of the divisor: |n . q| above and below exp(-m), exp(-m) far from 1, and a tiny n . q."""
    from mlx_lm_b200 import ops
    torch.manual_seed(H + V)
    T, eps = 9, 1e-3
    o, gate, weight = torch.randn(T, H * V), torch.randn(T, H * V).to(act), torch.randn(H * V)
    den = torch.randn(T, H) * torch.tensor([0.01, 1.0, 100.0]).repeat(3)[:, None]
    em = torch.exp(torch.randn(T, H) * 4)
    coef = torch.randn(T, H, 4)
    coef[:, :, 3] = em
    req = [0] * T
    req[5] = -1
    y = torch.full((T, H * V), 6.0, dtype=act, device=DEV)
    d = lambda t: t.contiguous().to(DEV)
    ops.mlstm_finish(d(o), d(den), d(coef), d(weight), d(gate), y, H, eps, i32(req), stream())
    div = torch.maximum(den.double().abs(), em.double()) + 1e-6
    want = plain.rms(o.double().view(T, H, V) / div[:, :, None], eps).reshape(T, H * V) * weight.double() * torch.sigmoid(gate.double())
    live = [t for t in range(T) if t != 5]
    tol = 2e-6 if act == torch.float32 else 5e-3
    assert float((y.cpu().double() - want)[live].abs().max()) < tol * float(want.abs().max())
    assert float((y.cpu().float()[5] - 6.0).abs().max()) == 0.0


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("D", [64, 50, 7, 1032, 2048, 8192, 12000])
@pytest.mark.parametrize("terms,extra", [(1, False), (2, True), (3, False), (1, True)])
def test_stream_update_through_a_norm_of_a_sum(act, D, terms, extra):
    from mlx_lm_b200 import ops
    torch.manual_seed(D + terms)
    T, eps, scale = 6, 1e-5, 1.0 / terms
    x0, y1, y2, w = torch.randn(T, D), torch.randn(T * terms, D), torch.randn(T, D), torch.randn(D)
    req = [0] * T
    req[4] = -1
    y = y1.double().view(T, terms, D).sum(1) * scale + (y2.double() if extra else 0.0)
    want = x0.double() + plain.rms(y, eps) * w.double()
    x, cast = x0.clone().to(DEV), torch.full((T, D), 5.0, dtype=act, device=DEV)
    ops.norm_update(x, y1.to(DEV), w.to(DEV), eps, stream(), terms=terms, scale=scale, y2=y2.to(DEV) if extra else None,
                    token_req=i32(req), cast_out=cast)
    live = [0, 1, 2, 3, 5]
    assert float((x.cpu().double() - want)[live].abs().max()) < 1e-5 and torch.equal(x.cpu()[4], x0[4])
    assert torch.equal(cast.cpu()[live], x.cpu()[live].to(act)) and float((cast.cpu().float()[4] - 5.0).abs().max()) == 0.0
    again = x0.clone().to(DEV)                         # without a copy: the same rows
    ops.norm_update(again, y1.to(DEV), w.to(DEV), eps, stream(), terms=terms, scale=scale, y2=y2.to(DEV) if extra else None, token_req=i32(req))
    assert torch.equal(again.cpu(), x.cpu())


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("D", [64, 100, 1032, 2048, 8192])
def test_rms_norm_of_rows_kept_in_registers(act, D):
    from mlx_lm_b200 import ops
    torch.manual_seed(D)
    x, w, rows = torch.randn(9, D) * 3, torch.randn(D), [7, 0, 0, 8, -1]
    for offset in (0.0, 1.0):
        want = plain.rms(x.double(), 1e-5) * (offset + w.double())
        tol = (2e-6 if act == torch.float32 else 5e-3) * float(want.abs().max())
        out, picked = torch.zeros(9, D, dtype=act, device=DEV), torch.full((5, D), 4.0, dtype=act, device=DEV)
        assert ops.rmsnorm_rows_supported(x.to(DEV), w.to(DEV), out)
        ops.rmsnorm_rows(x.to(DEV), w.to(DEV), out, 1e-5, stream(), offset=offset)
        assert float((out.cpu().double() - want).abs().max()) < tol
        ops.rmsnorm_rows(x.to(DEV), w.to(DEV), picked, 1e-5, stream(), offset=offset, rows=i32(rows))
        assert torch.equal(picked.cpu()[:4], out.cpu()[rows[:4]]) and float(picked[4].float().abs().max()) == 0.0


@pytest.mark.parametrize("T,E,top,rows", [(5, 3, 1, 4), (700, 16, 2, 128), (64, 9, 4, 16), (1, 1, 1, 64), (2000, 40, 3, 64)])
def test_plan_of_experts_named_by_a_table(T, E, top, rows):
    from mlx_lm_b200 import ops
    torch.manual_seed(T + E)
    V = 101
    table = torch.rand(V, E).argsort(1)[:, :top].to(torch.int32).contiguous()
    toks = torch.randint(0, V, (T,)).tolist()
    req = [0 if t % 7 else -1 for t in range(T)] if T > 1 else [0]
    S, mt = T * top, ops.moe_max_tiles(T * top, E, rows)
    order, tiles = torch.full((S,), -7, dtype=torch.int32, device=DEV), torch.zeros(3 * mt + 1, dtype=torch.int32, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.moe_plan_table(i32(toks), i32(req), table.to(DEV), T, E, rows, order, tiles, tiles[3 * mt:], status, stream())
    assert int(status) == 0
    seen, n = {}, int(tiles[3 * mt])
    for e, first, count in tiles[:3 * n].view(n, 3).tolist():
        assert 0 < count <= rows
        for slot in order[first:first + count].tolist():
            assert slot not in seen
            seen[slot] = e
    want = {t * top + c: int(table[toks[t], c]) for t in range(T) if req[t] >= 0 for c in range(top)}
    assert seen == want
    # a token outside the table is reported and takes no part
    ops.moe_plan_table(i32([V, 3] if T > 1 else [V]), i32([0] * min(T, 2)), table.to(DEV), min(T, 2), E, rows, order, tiles, tiles[3 * mt:],
                       status, stream())
    assert int(status) == ops.ST_TOKEN_RANGE


@pytest.mark.parametrize("rows", ["simt", "tc", "few"])
@pytest.mark.parametrize("act", ACT)
def test_experts_product_without_weights(act, rows):
    """The gated product without routing weights gives what it gives with weights of one."""
    from mlx_lm_b200 import ops
    if act == torch.float32 and rows != "simt":
        return
    torch.manual_seed(1)
    T, D, F, E = 20, 64, 48, 3
    x, w = torch.randn(T, D).to(act).to(DEV), (torch.randn(E, 2 * F, D) * D ** -0.5).to(act).to(DEV)
    n = {"simt": ops.moe_tile_rows(False), "tc": ops.moe_tile_rows(True), "few": ops.moe_few_rows()}[rows]
    mt = ops.moe_max_tiles(T, E, n)
    order, tiles = torch.zeros(T, dtype=torch.int32, device=DEV), torch.zeros(3 * mt + 1, dtype=torch.int32, device=DEV)
    sel = i32([t % E for t in range(T)])
    ops.moe_plan(sel, T, E, n, order, tiles, tiles[3 * mt:], stream())
    res = []
    for sw in (None, torch.ones(T, device=DEV)):
        out = torch.zeros(T, F, dtype=act, device=DEV)
        ops.moe_gemm(x, 1, w, F, order, tiles, tiles[3 * mt:], mt, n, out, stream(), sel_weight=sw, gated=True)
        res.append(out.cpu())
    assert torch.equal(res[0], res[1]) and float(res[0].float().abs().max()) > 0.1


@pytest.mark.parametrize("shape", [(1, 7), (3, 77), (5, 640), (2, 32001)])
def test_soft_cap(shape):
    from mlx_lm_b200 import ops
    x = torch.randn(*shape) * 60
    y = x.clone().to(DEV)
    ops.soft_cap(y, 20.0, stream())
    assert float((y.cpu().double() - plain.soft_cap(x.double(), 20.0)).abs().max()) < 1e-5
    assert float(y.abs().max()) <= 20.0


@pytest.mark.parametrize("act", ACT)
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 16, 24, 16), (6, 6, 10, 7, 6), (2, 1, 64, 64, 0)])
def test_prepared_heads_with_normed_projections_and_mixed_values(act, H, G, dk, dv, rot):
    """Whole projections normed, heads turned by stretched frequencies; the first layer's values kept as they are, another
    layer's mixed with them; the rounded copy of the queries."""
    from mlx_lm_b200 import ops
    from mlx_lm_b200.parts import rotation_frequencies
    torch.manual_seed(dk + dv)
    T, page, eps, lam, start = 21, 16, 1e-5, 0.3, 40
    kr, vr = (dk + 7) // 8 * 8, (dv + 7) // 8 * 8
    scaling = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60}
    r = {"dims": rot, "base": 100.0, "scaling": scaling}
    freq = torch.tensor(rotation_frequencies(rot, 100.0, scaling)[0], dtype=torch.float64).float().to(DEV) if rot else None
    wq, wk = torch.randn(H * dk), torch.randn(G * dk)
    status, block = torch.zeros(1, dtype=torch.int32, device=DEV), i32([5, 4, 2, 0, -1]).view(1, 5)
    keep = torch.full((T, G * dv), 9.0, dtype=act, device=DEV)
    pad_row = 3                                        # a row that is nobody's
    req = [0] * T
    req[pad_row] = -1
    pos = [start + t - (1 if t > pad_row else 0) for t in range(T)]
    firsts = None
    for layer in (0, 1):
        proj = torch.randn(T, H * dk + G * (dk + dv)).to(act)
        kp, vp = torch.zeros(6, G, page, kr, dtype=act, device=DEV), torch.zeros(6, G, page, vr, dtype=act, device=DEV)
        q = torch.full((T, H * kr), 8.0, device=DEV)
        q16 = torch.full((T, H * kr), 8.0, dtype=torch.bfloat16, device=DEV) if act == torch.bfloat16 else None
        mix = dict(v_keep=keep) if layer == 0 else dict(v_first=keep, v_lambda=lam)
        ops.qkv_prepare(proj.to(DEV), 0, H * dk, (H + G) * dk, H, G, dk, dv, wq.to(DEV), wk.to(DEV), eps, freq, i32(pos), i32(req), block,
                        kp, vp, q, True, status, stream(), q_rounded=q16, **mix)
        assert int(status) == 0
        rows = [t for t in range(T) if t != pad_row]
        p64 = proj.double()[rows]
        turned = lambda x, n: plain.turn(torch.cat([torch.zeros(start, n, dk, dtype=torch.float64), x.view(len(rows), n, dk)]), r)[start:] if rot \
            else x.view(len(rows), n, dk)
        wantq = turned(plain.rms(p64[:, :H * dk], eps) * wq.double(), H)
        wantk = turned(plain.rms(p64[:, H * dk:(H + G) * dk], eps) * wk.double(), G)
        v = p64[:, (H + G) * dk:]
        if layer == 0:
            firsts = v
            assert torch.equal(keep.cpu()[rows], proj[rows][:, (H + G) * dk:]) and float((keep.cpu().float()[pad_row] - 9.0).abs().max()) == 0.0
        else:
            v = plain.mix_values(v, firsts, lam)
        tol = 1e-5 if act == torch.float32 else 2e-2
        got = q.cpu().double().view(T, H, kr)[rows]
        assert float((got[:, :, :dk] - wantq).abs().max()) < 2e-5 * max(1.0, float(wantq.abs().max())) and float(got[:, :, dk:].abs().sum()) == 0.0
        if q16 is not None:
            assert torch.equal(q16.cpu()[rows], q.cpu()[rows].to(torch.bfloat16)) and float((q16.cpu().float()[pad_row] - 8.0).abs().max()) == 0.0
        for n, t in enumerate(rows):
            pg, at = int(block[0, pos[t] // page]), pos[t] % page
            assert float((kp[pg, :, at, :dk].cpu().double() - wantk[n]).abs().max()) < tol * max(1.0, float(wantk.abs().max()))
            assert float((vp[pg, :, at, :dv].cpu().double() - v[n].view(G, dv)).abs().max()) < tol * max(1.0, float(v.abs().max()))
