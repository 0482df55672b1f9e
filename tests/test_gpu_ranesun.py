"""Ranesun on the GPU against the plain float64 oracle (tests/ranesun_oracle.py): every mechanism alone through the C ABI,
then whole models of several shapes through the engine, its caches, its recurrent state and the scheduler."""
import json
import math
import os

import pytest
import torch

import ranesun_oracle as O
from test_gpu_ninisun import Paged, _close, _i32, _rows_close, _tokens

pytestmark = pytest.mark.gpu
F64 = torch.float64
PAGE = 64
TOL = {torch.float32: 3e-5, torch.bfloat16: 5e-2}
STRAY = {torch.float32: 0.0, torch.bfloat16: 0.02}
CT = {torch.float32: 0, torch.bfloat16: 1}
DTYPES = [torch.float32, torch.bfloat16]


def _lib():
    from pg_b200 import _cabi as cabi
    return cabi, cabi.lib(), cabi.stream()


def _engine(cfg, seed=0, dtype=torch.float32, pool_tokens=1024, **kw):
    from pg_b200.ranesun import RanesunEngine
    ck = O.make_checkpoint(cfg, seed)
    return RanesunEngine(cfg, ck, device="cuda:0", dtype=dtype, kv_pool_tokens=pool_tokens, **kw), ck


def _segs(lens, slots):
    segs, row = [], 0
    for n, s in zip(lens, slots):
        segs += [s, row, n]
        row += n
    return segs


def _p(t):
    return None if t is None else t.data_ptr()


# ------------------------------------------------------------------ mechanisms alone (C ABI)
@pytest.mark.parametrize("D", [48, 50, 1000, 1500, 2100, 5000])
@pytest.mark.parametrize("rows", [3, 400])
@pytest.mark.parametrize("dtype", DTYPES)
def test_row_kernel_between_sublayers(D, rows, dtype):
    """Dense and expert outputs, the embedding row set and added, a pass's vector, both layouts of the result, picked rows,
    an id outside the vocabulary: widths and row counts that take every variant of the kernel."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(D + rows)
    V, top, eps = 19, 2, 1e-3
    rnd = lambda *s: torch.randn(*s, generator=g)
    x0, y, table = rnd(rows, D) * 3 + 1.0, rnd(rows, D + 8).to(dtype), rnd(V, D).to(dtype)
    ey = rnd(rows * top, D).to(dtype)
    places = torch.randperm(rows * top, generator=g).to(torch.int32)
    vec, w, b = rnd(D).to(dtype), (1 + 0.3 * rnd(D)).to(dtype), rnd(D).to(dtype)
    ids = torch.randint(0, V, (rows,), generator=g)
    dv = dict(y=y.cuda(), table=table.cuda(), ey=ey.cuda(), places=places.cuda(), vec=vec.cuda(), w=w.cuda(), b=b.cuda(), ids=ids.cuda())
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    f = lambda t: t.to(F64)

    def call(x, out, *, ldo=None, y=None, ldy=0, pos=None, yw=1.0, emb=0, vec=None, scale=1.0, idx=None, opos=None, n=rows, ids=dv["ids"]):
        cabi.check(L.pg_residual_layernorm(_p(out), D if ldo is None else ldo, x.data_ptr(), _p(y), ldy, _p(pos), top, yw, ids.data_ptr(),
                                           dv["table"].data_ptr(), V, emb, _p(vec), dv["w"].data_ptr(), dv["b"].data_ptr(), eps, scale,
                                           _p(idx), _p(opos), top, n, D, err.data_ptr(), CT[dtype], st))
    tol = 4e-3 if dtype == torch.bfloat16 else 2e-6
    new = lambda n, c=D: torch.zeros(n, c, dtype=dtype, device="cuda")
    # the first sublayer: the stream is the embedding row (x is not read)
    x, out = torch.full((rows, D), float("nan"), device="cuda"), new(rows)
    call(x, out, emb=1)
    want = f(table)[ids]
    assert torch.equal(x.cpu().to(F64), want)
    _close(out, O.layer_norm(want, w.float(), b.float(), eps), tol)
    # a dense output, the embedding once more, a vector; the result in rows with a gap, scaled
    x, out = x0.cuda(), new(rows, D + 4)
    call(x, out, ldo=D + 4, y=dv["y"], ldy=D + 8, emb=2, vec=dv["vec"], scale=0.37)
    want = f(x0) + f(y)[:, :D] + f(table)[ids] + f(vec)
    _close(x, want, 1e-6)
    _close(out[:, :D], 0.37 * O.layer_norm(want, w.float(), b.float(), eps), tol)
    assert float(out[:, D:].abs().max()) == 0
    # expert outputs through their places, the result at the places of the next experts; one token has none
    pos2 = places.clone()
    pos2[2 * top:3 * top] = -1
    nxt = torch.randperm(rows * top, generator=g).to(torch.int32)
    nxt[top - 1] = -1
    x, out = x0.cuda(), new(rows * top)
    call(x, out, y=dv["ey"], ldy=D, pos=pos2.cuda(), yw=1.0 / top, opos=nxt.cuda())
    want = f(x0).clone()
    for t in range(rows):
        for k in range(top):
            if int(pos2[t * top + k]) >= 0:
                want[t] += f(ey)[int(pos2[t * top + k])] / top
    _close(x, want, 1e-6)
    ln = O.layer_norm(want, w.float(), b.float(), eps)
    scattered = torch.zeros(rows * top, D, dtype=F64)
    for i, p in enumerate(nxt.tolist()):
        if p >= 0:
            scattered[p] = ln[i // top]
    _close(out, scattered, tol)
    # picked rows (one of them twice): the sum enters the result, the stream stays
    idx = [rows - 1, 0, rows - 1]
    x, out = x0.cuda(), new(3)
    call(x, out, y=dv["y"], ldy=D + 8, idx=_i32(idx), n=3)
    assert torch.equal(x.cpu(), x0)
    _close(out, O.layer_norm((f(x0) + f(y)[:, :D])[idx], w.float(), b.float(), eps), tol)
    # the sum alone, then an id outside the vocabulary
    x = x0.cuda()
    call(x, None, y=dv["y"], ldy=D + 8)
    _close(x, f(x0) + f(y)[:, :D], 1e-6)
    torch.cuda.synchronize()
    assert int(err) == 0
    ids2 = ids.clone()
    ids2[1] = V
    x = x0.cuda()
    call(x, None, emb=1, ids=ids2.cuda())
    torch.cuda.synchronize()
    assert int(err) == 1 and float(x[1].abs().max()) == 0 and torch.equal(x[0].cpu().to(F64), f(table)[ids[0]])


def test_layer_norm_of_rows_far_from_zero():
    """A mean of 300 with deviations of 0.01: the variance comes from the deviations, not from a difference of squares."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(1)
    for D in (64, 66, 3000):
        x0 = (300.0 + 0.01 * torch.randn(5, D, generator=g)).float()
        x, out, w, b = x0.cuda(), torch.zeros(5, D, device="cuda"), torch.ones(D, device="cuda"), torch.zeros(D, device="cuda")
        cabi.check(L.pg_residual_layernorm(out.data_ptr(), D, x.data_ptr(), None, 0, None, 1, 1.0, None, None, 0, 0, None, w.data_ptr(),
                                           b.data_ptr(), 1e-6, 1.0, None, None, 1, 5, D, None, 0, st))
        _close(out, O.layer_norm(x0.to(F64), w.cpu(), b.cpu(), 1e-6), 3e-3)      # 300 holds 0.01 to 3 digits in fp32


@pytest.mark.parametrize("cols,k0,ld", [(96, 16, 128), (10, 3, 17), (256, 0, 264)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_cache_append(cols, k0, ld, dtype):
    cabi, L, st = _lib()
    positions, slots = [63, 64, 65, 0, 199, 127], [1, 1, 1, 0, 2, 3]
    pg = Paged([10, 70, 200, 128], cols, 1, dtype)
    proj = torch.randn(6, ld, generator=torch.Generator().manual_seed(ld)).to(dtype)
    pd = proj.cuda()
    cabi.check(L.pg_cache_append(pg.k.data_ptr(), cols, pd.data_ptr(), ld, k0, cols, pg.table.data_ptr(), pg.max_pages, PAGE,
                                 _i32(slots).data_ptr(), _i32(positions).data_ptr(), 6, CT[dtype], st))
    rows = [pg.rows(s, [p])[0] for s, p in zip(slots, positions)]
    flat = pg.k.view(-1, cols).cpu()
    assert torch.equal(flat[rows], proj[:, k0:k0 + cols])
    rest = torch.ones(flat.shape[0], dtype=torch.bool)
    rest[rows] = False
    assert bool((flat[rest] == 7.0).all())


@pytest.mark.parametrize("T", [1, 7, 33, 500, 9001])
def test_table_routing_groups_the_pairs_of_every_layer(T):
    """Layers with other expert counts and other `top` in one launch (9001 tokens: several rounds); one id is bad."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(T)
    V, sizes = 50, [(8, 2), (3, 3), (70, 1), (1, 1), (40, 5)]
    tables = [torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]).to(torch.int32) for E, top in sizes]
    desc, ent, tops, offs = [], 0, 0, 0
    for (E, top), t in zip(sizes, tables):
        desc += [ent, E, top, tops, offs]
        ent, tops, offs = ent + t.numel(), tops + top, offs + E + 1
    ids = torch.randint(0, V, (T,), generator=g)
    if T > 1:
        ids[T // 2] = V + 3
    offsets = torch.full((offs,), -7, dtype=torch.int32, device="cuda")
    pos = torch.full((T * tops,), -7, dtype=torch.int32, device="cuda")
    flat, idd = torch.cat([t.reshape(-1) for t in tables]).cuda(), ids.cuda()
    cabi.check(L.pg_moe_table_sort(offsets.data_ptr(), pos.data_ptr(), flat.data_ptr(), _i32(desc).data_ptr(), len(sizes), idd.data_ptr(),
                                   T, V, 70, st))
    offsets, pos = offsets.cpu(), pos.cpu()
    tops = offs = 0
    good = (ids < V)
    for (E, top), table in zip(sizes, tables):
        o, p = offsets[offs:offs + E + 1].tolist(), pos[T * tops:T * (tops + top)].view(T, top)
        tops, offs = tops + top, offs + E + 1
        want = table[ids.clamp(max=V - 1)][good].reshape(-1)
        assert o == [0] + torch.bincount(want, minlength=E).cumsum(0).tolist()
        assert bool((p[~good] == -1).all())
        placed = p[good].reshape(-1)
        assert sorted(placed.tolist()) == list(range(o[-1]))                     # every place once
        owner = torch.bucketize(placed, torch.tensor(o[1:]), right=True)         # ... inside the pair's own expert
        assert torch.equal(owner, want.to(owner.dtype))


@pytest.mark.parametrize("dtype,N,K,impl", [(torch.float32, 20, 30, 1), (torch.bfloat16, 36, 52, 1), (torch.bfloat16, 64, 72, 2),
                                            (torch.bfloat16, 200, 128, 2), (torch.float32, 128, 64, 0)])
def test_grouped_experts_with_squared_relu(dtype, N, K, impl):
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(N)
    counts = [0, 5, 130, 1, 0, 64]
    off = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
    P, E = int(off[-1]), len(counts)
    a, W = torch.randn(P, K, generator=g).to(dtype), (torch.randn(E, N, K, generator=g) / math.sqrt(K)).to(dtype)
    out, err = torch.zeros(P, N, dtype=dtype, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    ad, Wd, od = a.cuda(), W.cuda(), off.cuda()
    cabi.check(L.pg_moe_gemm_act(out.data_ptr(), N, ad.data_ptr(), K, None, Wd.data_ptr(), od.data_ptr(), P, E, N, K, cabi.ACT_RELU2, 0.0,
                                 impl, err.data_ptr(), CT[dtype], st))
    want = torch.cat([torch.relu(a[off[e]:off[e + 1]].to(F64) @ W[e].to(F64).T) ** 2 for e in range(E)])
    _close(out, want, 4e-3 if dtype == torch.bfloat16 else 2e-6)
    torch.cuda.synchronize()
    assert int(err) == 0


def _retention_run(L, cabi, st, rows, ld, cols, freq, rot_dims, H, d, e, S, dec, segs, pos, eps, dtype, interleaved=0):
    T = rows.shape[0]
    rec = torch.empty(L.pg_lightning_record_floats(T, H, d, e), device="cuda")
    cabi.check(L.pg_retention_prep(rec.data_ptr(), rows.data_ptr(), ld, cols[0], cols[1], cols[2], _p(freq), rot_dims, interleaved,
                                   d ** -0.5, _i32(pos).data_ptr(), T, H, d, e, CT[dtype], st))
    o = torch.zeros(T, H * e, device="cuda")
    cabi.check(L.pg_lightning_attention(o.data_ptr(), S.data_ptr(), rec.data_ptr(), dec.data_ptr(), _i32(segs).data_ptr(),
                                        len(segs) // 3, H, d, e, st))
    out = torch.zeros(T, H * e, dtype=dtype, device="cuda")
    cabi.check(L.pg_headnorm_gate_ex(out.data_ptr(), H * e, o.data_ptr(), None, rows[:, cols[3]:].data_ptr(), ld, 1, T, H, e, eps, 1.0,
                                     CT[dtype], st))
    return out, o, rec


@pytest.mark.parametrize("H,d,e,rot", [(4, 8, 6, 8), (1, 12, 20, 4), (3, 64, 32, 64), (2, 7, 9, 6), (5, 128, 130, 64), (2, 6, 3, 0), (1, 200, 16, 200)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_retention_over_portions_and_slots(H, d, e, rot, dtype):
    """Rotation, decayed state, per-head norm and silu gate of two sequences fed in portions side by side (one of them into
    a slot that another sequence left) against the oracle over whole sequences."""
    cabi, L, st = _lib()
    from pg_b200.ragged_engine import RotaryCfg
    from pg_b200.ranesun import rotary_pairs
    g = torch.Generator().manual_seed(H * 1000 + d)
    al = lambda n: (n + 7) // 8 * 8
    cols = [0, al(H * d), 2 * al(H * d), 2 * al(H * d) + al(H * e)]
    ld, eps, lens = cols[3] + al(H * e), 1e-4, {"a": 75, "b": 12}
    dec = [1.0 - 2.0 ** (-1.0 - 3.0 * h) for h in range(H)]
    proj = {k: (torch.randn(n, ld, generator=g) * 1.5).to(dtype) for k, n in lens.items()}
    want, raw = {}, {}
    for k, n in lens.items():
        u = proj[k].to(F64)
        q, kk, v = u[:, :H * d].view(n, H, d), u[:, cols[1]:cols[1] + H * d].view(n, H, d), u[:, cols[2]:cols[2] + H * e].view(n, H, e)
        if rot:
            f = O.frequencies(rot, 300.0)
            q, kk = O.rotate(q, list(range(n)), f), O.rotate(kk, list(range(n)), f)
        raw[k] = O.retention_scan(q, kk / math.sqrt(d), v, dec)
        want[k] = O.unit_rms(raw[k], eps).reshape(n, H * e) * O.silu(u[:, cols[3]:cols[3] + H * e])
    freq = rotary_pairs(RotaryCfg(rot, 300.0)).cuda() if rot else None
    decd = torch.tensor(dec, dtype=torch.float32, device="cuda")
    S = torch.zeros(2, H, d, e, device="cuda")
    slot = {"a": 1, "b": 0}
    S[0].normal_()                                        # what an earlier sequence left
    plan = [[("a", 2)], [("a", 1)], [("b", 1), ("a", 3)], [("a", 60), ("b", 2)], [("b", 8), ("a", 1)], [("a", 8), ("b", 1)]]
    fed, got, got_o = {k: 0 for k in lens}, {k: [] for k in lens}, {k: [] for k in lens}
    for step in plan:
        for k, _ in step:
            if fed[k] == 0:
                S[slot[k]].zero_()
        rows = torch.cat([proj[k][fed[k]:fed[k] + n] for k, n in step]).cuda()
        pos = [fed[k] + i for k, n in step for i in range(n)]
        segs = _segs([n for _, n in step], [slot[k] for k, _ in step]) + [0, 0, 0]
        out, o, _ = _retention_run(L, cabi, st, rows, ld, cols, freq, rot, H, d, e, S, decd, segs, pos, eps, dtype)
        at = 0
        for k, n in step:
            got[k].append(out[at:at + n].float().cpu())
            got_o[k].append(o[at:at + n].cpu())
            at += n
            fed[k] += n
    for k, n in lens.items():
        assert fed[k] == n
        _rows_close(torch.cat(got_o[k]), raw[k].reshape(n, H * e), 2e-5)
        _rows_close(torch.cat(got[k]), want[k], 5e-3 if dtype == torch.bfloat16 else 2e-3, 0.05)   # a head near zero: its norm magnifies
        _close(torch.cat(got[k]), want[k], 5e-3 if dtype == torch.bfloat16 else 3e-4)


def test_retention_angles_stay_exact_at_far_positions():
    """Position 60000 with unit frequency: one fp32 product alone would be some 2e-3 rad off; both pair layouts."""
    cabi, L, st = _lib()
    from pg_b200.ragged_engine import RotaryCfg
    from pg_b200.ranesun import rotary_pairs
    g = torch.Generator().manual_seed(4)
    d, pos = 16, [60001, 33333, 1, 0]
    proj = torch.randn(4, 3 * d, generator=g)
    f = O.frequencies(d, 7.0)
    freq = rotary_pairs(RotaryCfg(d, 7.0)).cuda()
    pd = proj.cuda()
    for interleaved in (0, 1):
        rec = torch.empty(L.pg_lightning_record_floats(4, 1, d, d), device="cuda")
        cabi.check(L.pg_retention_prep(rec.data_ptr(), pd.data_ptr(), 3 * d, 0, d, 2 * d, freq.data_ptr(), d, interleaved, 0.25,
                                       _i32(pos).data_ptr(), 4, 1, d, d, 0, st))
        order = torch.arange(d).view(d // 2, 2).T.reshape(-1) if interleaved else torch.arange(d)
        back = torch.argsort(order)
        q = O.rotate(proj[:, :d].to(F64)[:, order], pos, f)[:, back]
        k = O.rotate(proj[:, d:2 * d].to(F64)[:, order], pos, f)[:, back] * 0.25
        _rows_close(rec.view(4, 3 * d), torch.cat([q, k, proj[:, 2 * d:].to(F64)], -1), 1e-6)


def test_retention_state_carries_a_first_token_far():
    """A decay of almost 1 beside one of 1/2: what the first token wrote is read 700 tokens later by the one head and gone in
    the other, whole or cut into portions."""
    cabi, L, st = _lib()
    H, d, e, T, eps = 2, 8, 8, 701, 1e-12
    cols, ld = [0, 16, 32, 48], 64
    proj = torch.zeros(T, ld)
    proj[0, 16:48] = 3.0                                  # k and v of the first token
    proj[T - 1, :16] = 2.0                                # the last token asks
    dec = [1.0 - 2.0 ** -14, 0.5]
    k, v, q = proj[:, 16:32].view(T, H, d).to(F64), proj[:, 32:48].view(T, H, e).to(F64), proj[:, :16].view(T, H, d).to(F64)
    want = O.retention_scan(q, k / math.sqrt(d), v, dec)
    assert float(want[-1, 0].min()) > 10 and float(want[-1, 1].abs().max()) < 1e-30
    decd = torch.tensor(dec, dtype=torch.float32, device="cuda")
    rows = proj.cuda()
    for cuts in ([T], [1, 2, 61, 64, 200, 2, 1, 369, 1]):
        assert sum(cuts) == T
        S, at, outs = torch.zeros(1, H, d, e, device="cuda"), 0, []
        for n in cuts:
            _, o, _ = _retention_run(L, cabi, st, rows[at:at + n], ld, cols, None, 0, H, d, e, S, decd, [0, 0, n], list(range(at, at + n)),
                                     eps, torch.float32)
            outs.append(o)
            at += n
        _close(torch.cat(outs)[:, :e], want[:, 0], 2e-5)
        assert float(torch.cat(outs)[-1, e:].abs().max()) < 1e-30


def _tied_case(H, G, d, softcap, temp, lens, new, sinks, dtype=torch.float32, tower=None, seed=0, tc=False, scale=0.5, q_gain=1.0):
    """Sequences of lens[s] cached keys (which are the values) of which the last new[s] are this step's queries.  tower
    (function of the last position): the place of one key whose score stands far out for the last query."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(seed)
    pg = Paged(lens, G * d, 1, dtype)
    ldq = H * d + 8
    qs, want, slots, positions = [], [], [], []
    sink = torch.tensor(sinks, dtype=torch.float32) if sinks is not None else None
    o_temp = temp if temp[1] else (0.0, 1)                # every = 0: the kernels' way to say that there is no temperature
    for s, (n, m) in enumerate(zip(lens, new)):
        q, k = q_gain * torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g)
        if tower is not None:
            j = tower(n - 1)
            k[j] = 0.0
            k[j, :, 0] = 9.0
            q[n - 1, :, :] = 0.0
            q[n - 1, :, 0] = 30.0
            k[torch.arange(n) != j, :, 0] = 0.0
        q, k = q.to(dtype).float(), k.to(dtype).float()
        pg.fill(s, k, torch.zeros(n, 1))
        for_h = [O.tied_attention(q[n - m:, h].to(F64), k[:, h // (H // G)].to(F64), scale, softcap, o_temp,
                                  float("-inf") if sink is None else sink[h], first=n - m) for h in range(H)]
        qs.append(torch.cat([q[n - m:].reshape(m, H * d), torch.zeros(m, 8)], -1))
        want.append(torch.stack(for_h, 1).reshape(m, H * d))
        slots += [s] * m
        positions += list(range(n - m, n))
    q_all = torch.cat(qs).to(dtype).cuda()
    T = q_all.shape[0]
    out = torch.full((T, H * d + 8), 5.0, dtype=dtype, device="cuda")
    sd = None if sink is None else sink.cuda()
    coef, every = temp
    if tc:
        tiles, t0 = [], 0
        while t0 < T:
            t1 = t0 + 1
            while t1 < T and t1 - t0 < 128 and slots[t1] == slots[t0]:
                t1 += 1
            tiles += [t0, t1 - t0, slots[t0], positions[t0]]
            t0 = t1
        err = torch.zeros(1, dtype=torch.int32, device="cuda")
        cabi.check(L.pg_attention_ragged_tc_capped(
            out.data_ptr(), H * d + 8, q_all.data_ptr(), ldq, None, 0, 0, pg.k.data_ptr(), 0, pg.k.data_ptr(), 0, pg.k.shape[0] * PAGE,
            pg.table.data_ptr(), pg.max_pages, PAGE, _i32(tiles).data_ptr(), len(tiles) // 4, T, H, G, d, d, scale, 0, 0, 0, None, 0,
            None, _p(sd), softcap or 0.0, coef, every, None, 0, 1.0, err.data_ptr(), CT[dtype], st))
        torch.cuda.synchronize()
        assert int(err) == 0
    else:
        ws = torch.empty(1 << 20, device="cuda")
        cabi.check(L.pg_attention_ragged_capped(
            out.data_ptr(), H * d + 8, q_all.data_ptr(), ldq, None, 0, 0, pg.k.data_ptr(), 0, pg.k.data_ptr(), 0, pg.table.data_ptr(),
            pg.max_pages, PAGE, _i32(slots).data_ptr(), _i32(positions).data_ptr(), T, H, G, d, d, scale, 0, 0, 0, None, 0, None, _p(sd),
            softcap or 0.0, coef, every, None, 0, 1.0, ws.data_ptr(), ws.numel(), CT[dtype], st))
        torch.cuda.synchronize()
    assert bool((out[:, H * d:] == 5.0).all())
    return out[:, :H * d].float(), torch.cat(want)


MIXED = dict(lens=[150, 76, 1, 65, 129], new=[150, 1, 1, 3, 2])          # a prompt, decoded tokens, page borders
DECODE = dict(lens=[300, 64, 65, 1, 777], new=[1, 1, 1, 1, 1])           # single tokens: keys cut over CTAs and merged


@pytest.mark.parametrize("H,G,d", [(4, 2, 8), (6, 1, 12), (2, 2, 48), (8, 1, 32), (3, 1, 96), (1, 1, 17), (16, 2, 128), (2, 1, 200)])
@pytest.mark.parametrize("softcap,temp", [(6.0, (0.4, 7)), (50.0, (0.3, 64)), (20.0, (0.0, 0)), (None, (0.5, 16)), (2.0, (1.5, 1))])
@pytest.mark.parametrize("what", ["mixed", "decode"])
def test_capped_attention_over_tied_keys(H, G, d, softcap, temp, what):
    sinks = [0.5 - 1.0 * h for h in range(H)]
    sinks[0] = 4.0
    got, want = _tied_case(H, G, d, softcap, temp, sinks=sinks, seed=d, **(MIXED if what == "mixed" else DECODE))
    _rows_close(got, want, 3e-5)


@pytest.mark.parametrize("H,G,d", [(4, 2, 64), (3, 1, 128), (2, 2, 96), (4, 1, 40), (2, 1, 8), (1, 1, 136), (2, 1, 200), (1, 1, 256)])
@pytest.mark.parametrize("softcap,temp", [(15.0, (0.4, 40)), (60.0, (0.3, 64)), (None, (0.0, 0)), (40.0, (1.0, 1))])
def test_tensor_core_capped_attention_over_tied_keys(H, G, d, softcap, temp):
    """Head sizes that fill, half fill and hardly fill the 64-column tiles; caps that allow one pass and caps that do not."""
    got, want = _tied_case(H, G, d, softcap, temp, lens=[300, 190, 77, 64], new=[300, 131, 50, 64], sinks=[3.0 - 2.0 * h for h in range(H)],
                           dtype=torch.bfloat16, tc=True, seed=d, scale=1.5 / math.sqrt(d))
    _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("mode", ["prompt", "decode", "tc"])
@pytest.mark.parametrize("where", ["first", "page_end", "page_start", "previous", "self"])
def test_one_far_key_among_hundreds(mode, where):
    """A key whose capped score is far above the others', at position 0, on both sides of a page border, right before the
    query and at the query."""
    n = 331
    j = {"first": 0, "page_end": 191, "page_start": 192, "previous": n - 2, "self": n - 1}[where]
    dtype = torch.bfloat16 if mode == "tc" else torch.float32
    got, want = _tied_case(2, 1, 64, 18.0, (0.2, 100), lens=[n], new=[1 if mode == "decode" else n], sinks=[1.0, 2.0], dtype=dtype,
                           tower=lambda _: j, tc=mode == "tc", scale=0.4)
    assert float(want[-1, 0]) > 8.0                       # the far key takes the weight
    _rows_close(got, want, 2e-2 if mode == "tc" else 3e-5)


@pytest.mark.parametrize("mode", ["prompt", "decode", "tc"])
def test_a_sink_that_takes_almost_everything_and_one_that_takes_nothing(mode):
    """Sinks of +12, +100, -50 beside scores that the cap keeps within 5: left out, scaled, capped or counted twice, the
    result would be another."""
    n = 200
    dtype = torch.bfloat16 if mode == "tc" else torch.float32
    got, want = _tied_case(3, 1, 64, 5.0, (0.3, 50), lens=[n], new=[1 if mode == "decode" else n], sinks=[12.0, 100.0, -50.0], dtype=dtype,
                           tc=mode == "tc", scale=0.2)
    one = lambda t, h: t[:, 64 * h:64 * (h + 1)]
    assert float(one(want, 0).abs().max()) < 0.2 * float(one(want, 2).abs().max())
    _rows_close(one(got, 0), one(want, 0), 2e-2 if mode == "tc" else 3e-5)
    _rows_close(one(got, 2), one(want, 2), 2e-2 if mode == "tc" else 3e-5)
    assert float(one(got, 1).abs().max()) < 1e-30


@pytest.mark.parametrize("every", [1, 3, 64, 100])
@pytest.mark.parametrize("mode", ["prompt", "decode", "tc"])
def test_query_temperature_steps_at_their_positions(every, mode):
    """Strong temperature: positions every - 2, every - 1 (the step), every, and the next step, in a prompt and decoded."""
    dtype = torch.bfloat16 if mode == "tc" else torch.float32
    if mode == "decode":
        lens = sorted({max(n, 1) for n in (every - 1, every, every + 1, 2 * every - 1, 2 * every, 2 * every + 1)})
        new = [1] * len(lens)
    else:
        lens, new = [2 * every + 70], [2 * every + 70]
    got, want = _tied_case(2, 1, 32, 10.0, (2.0, every), lens=lens, new=new, sinks=[0.0, 1.0], dtype=dtype, tc=mode == "tc", scale=0.3)
    _rows_close(got, want, 3e-2 if mode == "tc" else 3e-5)
    off, _ = _tied_case(2, 1, 32, 10.0, (2.0, every), lens=lens, new=new, sinks=[0.0, 1.0], dtype=dtype, tc=mode == "tc", scale=0.3)
    assert torch.equal(off, got)                          # the same launch twice: the same bits


# ------------------------------------------------------------------ whole models
CONFIGS = {
    # every branch: both mixers, both feed-forwards and none, a looped block in the middle, grouped key heads, part of the
    # head rotated, other expert counts per layer
    "small": O.make_config(width=48, vocab=61, loop=(1, 3, 2), logit_scale=1.5, layers=[
        O.layer(O.attention(heads=4, kv_heads=2, dim=12, softcap=8.0, coef=0.5, every=16), O.dense(40)),
        O.layer(O.retention(heads=3, dim=8, vdim=6), O.moe(5, 2, 16)),
        O.layer(O.attention(heads=2, kv_heads=2, dim=8, softcap=30.0, coef=0.2, every=64), O.moe(4, 1, 12)),
        O.layer(O.retention(heads=2, dim=6, vdim=10, rot_dims=4))]),
    # values the other configurations make equal or 1: one head, values wider than keys, every expert chosen, a loop that
    # holds the first layer and all others, three passes, a temperature step at every position, sizes off every multiple
    "odd": O.make_config(width=50, vocab=67, loop=(0, 3, 3), eps=1e-3, logit_scale=0.5, layers=[
        O.layer(O.retention(heads=1, dim=10, vdim=13, decay=[0.97], rot_dims=6, base=50.0), O.moe(3, 3, 9)),
        O.layer(O.attention(heads=5, kv_heads=1, dim=6, softcap=45.0, coef=0.8, every=1)),
        O.layer(O.attention(heads=1, kv_heads=1, dim=20, softcap=3.0, coef=0.3, every=33, scale=0.5), O.dense(30))]),
    # no looped block; attention alone first and last, one expert in all
    "flat": O.make_config(width=64, vocab=90, layers=[
        O.layer(O.attention(heads=4, kv_heads=4, dim=16, every=5), O.moe(1, 1, 24)),
        O.layer(O.retention(heads=4, dim=16, vdim=16), O.dense(64)),
        O.layer(O.attention(heads=3, kv_heads=1, dim=24), O.moe(6, 4, 16))]),
    # head sizes of real models: the 16-bit run crosses the tensor-core attention (whole, filled-up and two-pass tiles) and
    # the tensor-core GEMMs; one pass only, with its step vector
    "wide": O.make_config(width=256, vocab=300, loop=(1, 4, 2), layers=[
        O.layer(O.attention(heads=4, kv_heads=2, dim=64, softcap=20.0, coef=0.3, every=48), O.dense(256)),
        O.layer(O.attention(heads=2, kv_heads=1, dim=104, softcap=50.0, coef=0.2, every=100), O.moe(6, 2, 128)),
        O.layer(O.retention(heads=4, dim=64, vdim=64), O.moe(8, 2, 64)),
        O.layer(O.attention(heads=3, kv_heads=3, dim=40, softcap=12.0), O.moe(3, 1, 128)),
        O.layer(O.retention(heads=2, dim=128, vdim=64, rot_dims=64), O.dense(128))]),
    "once": O.make_config(width=32, vocab=40, loop=(1, 2, 1), layers=[
        O.layer(O.retention(heads=2, dim=8, vdim=8), O.dense(16)),
        O.layer(O.attention(heads=2, kv_heads=1, dim=8), O.moe(4, 2, 16))]),
}
_ORACLE_CACHE = {}


def _stray(name, dtype):
    """16-bit runs: rows that may differ.  A retention head's output is normed by its own length: at the first positions
    it is v (q . k) over its rms, so with q . k near zero the sign of a head is a matter of rounding the projections."""
    return 0.06 if (name != "wide" and dtype == torch.bfloat16) else STRAY[dtype]


def _oracle(name, n, seed=0):
    key = (name, n, seed)
    if key not in _ORACLE_CACHE:
        cfg = CONFIGS[name]
        ck = O.make_checkpoint(cfg, 0)
        toks = _tokens(n, cfg["vocab"], 100 + seed)
        sink = []
        _ORACLE_CACHE[key] = (toks, O.forward(cfg, ck, toks, sink), sink)
    return _ORACLE_CACHE[key]


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt_logits_and_every_layer(name, dtype):
    n = 150
    toks, want, layers = _oracle(name, n)
    eng, _ = _engine(CONFIGS[name], dtype=dtype)
    assert [r.layer for r in eng.runs] == [i for i, _ in O.run_order(CONFIGS[name])]
    if name == "wide" and dtype == torch.bfloat16:
        assert [bool(w["attn_tc"]) for w in eng.layers] == [True, True, False, True, False]
    b = eng.new_batcher(slots=2)
    b.admit("a")
    sink = []
    got = b.run_entries([("a", toks, list(range(n)))], layer_sink=sink)
    eng.check_errors(sync=True)
    assert len(sink) == len(layers) == len(O.run_order(CONFIGS[name]))
    for x, ref in zip(sink, layers):
        _rows_close(x, ref, TOL[dtype], _stray(name, dtype))
    _rows_close(got, want, TOL[dtype] * 2, _stray(name, dtype))
    b.finish("a")
    b.admit("again")                                       # without the per-layer reads: sums stay pending between sublayers
    _rows_close(b.run_entries([("again", toks, [149, 0, 77, 149])]), want[[149, 0, 77, 149]], TOL[dtype] * 2, 0.26 if _stray(name, dtype) else 0.0)
    b.close()


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_then_token_by_token_and_portions(name, dtype):
    n = 150
    toks, want, _ = _oracle(name, n)
    eng, _ = _engine(CONFIGS[name], dtype=dtype, pool_tokens=448)
    b = eng.new_batcher(slots=2)
    b.admit("a")
    rows = [b.run_entries([("a", toks[:100], [99])])]
    rows += [b.run_entries([("a", [t], [0])]) for t in toks[100:]]
    _rows_close(torch.cat(rows), want[99:], TOL[dtype] * 2, _stray(name, dtype))
    b.finish("a")
    b.admit("b")          # the slot, the state and the pages of "a" again; portions down to two tokens and single ones
    at, got = 0, []
    for size in [2, 37, 2, 1, 31, 13, 1, 1, 2, 50, 3, 7]:
        got.append(b.run_entries([("b", toks[at:at + size], list(range(size)))]))
        at += size
    assert at == n
    _rows_close(torch.cat(got), want, TOL[dtype] * 2, _stray(name, dtype))
    eng.check_errors(sync=True)
    b.close()


@pytest.mark.parametrize("name,dtype", [("small", torch.float32), ("odd", torch.float32), ("flat", torch.float32),
                                        ("wide", torch.float32), ("wide", torch.bfloat16)])
def test_unequal_requests_in_one_batch_with_slots_and_pages_used_again(name, dtype):
    cfg = CONFIGS[name]
    lens = {"a": 131, "b": 23, "c": 97, "d": 150, "e": 70}
    ref = {k: _oracle(name, n, seed=i) for i, (k, n) in enumerate(lens.items())}
    eng, _ = _engine(cfg, dtype=dtype, pool_tokens=6 * PAGE)          # a pool that forces pages to be handed on
    b = eng.new_batcher(slots=3)
    fed = {k: 0 for k in lens}
    got = {k: [] for k in lens}
    plan = [
        [("a", 64), ("b", 21), ("c", 2)], [("a", 3), ("b", 1), ("c", 90)], [("a", 1), ("b", 1), ("c", 1)],
        [("a", 60), ("c", 1)], [("c", 1), ("a", 1)], [("c", 2)], [("a", 2), ("d", 65)], [("d", 2), ("e", 64)],
        [("d", 80), ("e", 1)], [("e", 5), ("d", 1)], [("d", 2)]]
    for step in plan:
        entries = []
        for k, n in step:
            if k not in b.slot_of:
                b.admit(k)
            entries.append((k, ref[k][0][fed[k]:fed[k] + n], list(range(n))))
            fed[k] += n
        out = b.run_entries(entries)
        at = 0
        for k, n in step:
            got[k].append(out[at:at + n])
            at += n
        for k, _ in step:
            if fed[k] == lens[k] and k in b.slot_of:
                b.finish(k)
    eng.check_errors(sync=True)
    for k in lens:
        assert fed[k] == lens[k]
        _rows_close(torch.cat(got[k]), ref[k][1], TOL[dtype] * 2, STRAY[dtype])
    b.close()
    assert eng.pages_in_use() == 0


def test_long_decoding_through_pages_and_temperature_steps():
    name, n = "small", 330
    toks, want, _ = _oracle(name, n)
    for dtype in DTYPES:
        eng, _ = _engine(CONFIGS[name], dtype=dtype)
        b = eng.new_batcher(slots=1)
        b.admit("a")
        rows = [b.run_entries([("a", toks[:5], list(range(5)))])]
        rows += [b.run_entries([("a", [t], [0])]) for t in toks[5:]]
        _rows_close(torch.cat(rows), want, TOL[dtype] * 2, STRAY[dtype])
        b.close()


def test_every_pass_of_the_loop_has_its_own_cache_and_state():
    cfg = CONFIGS["small"]
    eng, _ = _engine(cfg)
    assert sorted(eng.k_pools) == [0, 2, 4]                # attention runs: layer 0, layer 2 in both passes
    b = eng.new_batcher(slots=2)
    s = b.kv.state.layers
    assert sorted(s) == [1, 3, 5] and s[1].shape == (2, 3, 8, 6) and s[5].shape == (2, 2, 6, 10)
    b.admit("a")
    b.run_entries([("a", _tokens(70, 61, 1), [])])
    assert all(float(t[0].abs().max()) > 0 and float(t[1].abs().max()) == 0 for t in s.values())
    assert not torch.equal(s[1], s[3]) and not torch.equal(eng.k_pools[2], eng.k_pools[4])
    b.finish("a")
    b.admit("again")                                      # the slot is handed on with a zero state
    assert all(float(t[0].abs().max()) == 0 for t in s.values())
    b.close()


def test_decoding_with_a_second_slot_table_uses_its_own_state():
    """Small steps replay captured graphs.  A second scheduler whose page table happens to get the address of a released one
    must not run on the released one's state: the same request through many schedulers, each with other allocations alive."""
    toks, want, _ = _oracle("small", 150)
    eng, _ = _engine(CONFIGS["small"])
    alive = []
    for i in range(4):
        b = eng.new_batcher(slots=2)
        b.admit("a")
        got = [b.run_entries([("a", toks[:3], [2])])] + [b.run_entries([("a", [t], [0])]) for t in toks[3:30]]
        _rows_close(torch.cat(got), want[2:30], 6e-5)
        b.close()
        del b
        alive.append(torch.full((1 + 40 * i,), float("nan"), device="cuda"))       # takes up released blocks


def test_a_token_outside_the_vocabulary_is_reported():
    eng, _ = _engine(CONFIGS["small"])
    b = eng.new_batcher(slots=1)
    b.admit("a")
    b.run_entries([("a", [3, 61, 5], [2])])
    with pytest.raises(RuntimeError, match="vocabulary"):
        eng.check_errors(sync=True)
    b.close()


def _random_config(rng):
    """Sizes, layer order, loop and constants drawn at random from what real checkpoints use."""
    div = lambda n: [d for d in range(1, n + 1) if n % d == 0]
    n = rng.randint(2, 5)
    layers = []
    for _ in range(n):
        if rng.random() < 0.5:
            H = rng.choice([2, 4, 6, 8, 12])
            L = O.attention(heads=H, kv_heads=rng.choice(div(H)), dim=rng.choice([16, 32, 48, 64, 80, 96, 128]),
                            softcap=rng.choice([5.0, 20.0, 30.0, 50.0]), coef=rng.choice([0.1, 0.5]), every=rng.choice([7, 64, 100, 1000]))
        else:
            H, dim = rng.choice([1, 2, 3, 4, 8]), rng.choice([16, 24, 32, 64, 128])
            L = O.retention(heads=H, dim=dim, vdim=rng.choice([16, 32, 40, 64, 128]), rot_dims=rng.choice([dim, dim // 2]),
                            base=rng.choice([1e4, 2e5, 1e6]))
        E = rng.choice([2, 4, 8, 16])
        layers.append(O.layer(L, rng.choice([None, O.dense(rng.choice([128, 256, 320])), O.moe(E, rng.choice([1, 2]), rng.choice([32, 64, 160]))])))
    a = rng.randrange(n)
    return O.make_config(width=rng.choice([128, 192, 256, 320]), vocab=rng.choice([300, 512]), layers=layers,
                         loop=rng.choice([None, (a, rng.randint(a + 1, n), rng.choice([2, 3]))]), eps=rng.choice([1e-5, 1e-6]),
                         logit_scale=rng.choice([1.0, 2.0, 0.7]))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_models_drawn_at_random_whole_and_cut(seed):
    """Layer order, loops, head layouts, experts and constants at random: a whole prompt and the same tokens in portions and
    single tokens, in fp32 (every row) and in bf16 (typical error of a few percent)."""
    import random
    rng = random.Random(seed)
    cfg = _random_config(rng)
    ck = O.make_checkpoint(cfg, seed)
    n = 160
    toks = _tokens(n, cfg["vocab"], seed)
    want = O.forward(cfg, ck, toks)
    for dtype in DTYPES:
        eng, _ = _engine(cfg, seed=seed, dtype=dtype)
        b = eng.new_batcher(slots=2)
        b.admit("w")
        whole = b.run_entries([("w", toks, list(range(n)))])
        b.finish("w")
        b.admit("c")
        at, got = 0, []
        for size in [3, 61, 2, 50, 17]:
            got.append(b.run_entries([("c", toks[at:at + size], list(range(size)))]))
            at += size
        got += [b.run_entries([("c", [t], [0])]) for t in toks[at:]]
        eng.check_errors(sync=True)
        b.close()
        for out in (whole, torch.cat(got)):
            if dtype == torch.float32:
                _rows_close(out, want, 1e-4)
            else:
                _rows_close(out, want, 8e-2, 0.05)


def test_greedy_generation_through_the_scheduler():
    cfg = CONFIGS["small"]
    ck = O.make_checkpoint(cfg, 0)
    eng, _ = _engine(cfg)
    prompts = [_tokens(n, cfg["vocab"], 40 + n) for n in (3, 70, 18)]
    b = eng.new_batcher(slots=2, token_budget=32)
    rids = [b.submit(p, max_new_tokens=6) for p in prompts]
    done = b.run()
    for rid, p in zip(rids, prompts):
        seq = list(p)
        for _ in range(6):                                     # the oracle's own greedy loop
            seq.append(int(O.forward(cfg, ck, seq)[-1].argmax()))
        assert done[rid].tokens == seq[len(p):]
    b.close()
    assert eng.pages_in_use() == 0
    runs = []
    for _ in range(2):
        b = eng.new_batcher(slots=2, token_budget=32, do_sample=True, temperature=0.9, top_p=0.8, seed=5)
        rids = [b.submit(p, max_new_tokens=5) for p in prompts[:2]]
        done = b.run()
        runs.append([done[r].tokens for r in rids])
        b.close()
    assert runs[0] == runs[1] and all(0 <= t < cfg["vocab"] for seq in runs[0] for t in seq)


def test_model_folder_through_the_registry_and_command_line(tmp_path):
    import subprocess
    import sys
    import numpy as np
    from pg_b200.checkpoint import write_safetensors
    from pg_b200.registry import load_engine
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CONFIGS["odd"]
    ck = O.make_checkpoint(cfg, 3)
    model = tmp_path / "model"
    model.mkdir()
    with open(model / "config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors(str(model / "model.safetensors"), {k: v if v.dtype == torch.int32 else v.to(torch.bfloat16) for k, v in ck.items()})
    eng = load_engine(str(model), device="cuda:0", dtype=torch.float32, kv_pool_tokens=256)
    assert type(eng).__name__ == "RanesunEngine"
    toks = _tokens(40, cfg["vocab"], 9)
    b = eng.new_batcher(slots=1)
    b.admit(0)
    _rows_close(b.run_entries([(0, toks, [39, 0])]), O.forward(cfg, ck, toks)[[39, 0]], 1e-4)
    b.close()
    make = lambda w, **kw: type(eng)(cfg, w, device="cuda:0", dtype=torch.float32, kv_pool_tokens=64, **kw)
    more = dict(ck)
    more["l0.mix.extra"] = torch.zeros(3)
    with pytest.warns(UserWarning):
        make(more)
    with pytest.raises(ValueError):
        make(more, strict=True)
    with pytest.raises(KeyError):
        make({k: v for k, v in ck.items() if k != "l1.mix.sink"})
    with pytest.raises(ValueError):
        make(dict(ck, **{"l0.mlp.table": ck["l0.mlp.table"] + 1}))          # an expert that does not exist
    seq = {k: _tokens(n, cfg["vocab"], 60 + n) for k, n in (("a", 22), ("b", 5), ("c", 70))}
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": seq["a"][:20], "want": [19]}, {"id": "b", "tokens": seq["b"], "want": [0, 4]}],
         "end": ["b"]},
        {"step": 1, "entries": [{"id": "a", "tokens": seq["a"][20:21], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "c", "tokens": seq["c"], "want": [69]}, {"id": "a", "tokens": seq["a"][21:], "want": [0]}],
         "end": ["a", "c"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = {k: O.forward(cfg, ck, v) for k, v in seq.items()}
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, cfg["vocab"]))
    _rows_close(got0, torch.stack([ref["a"][19], ref["b"][0], ref["b"][4]]), 1e-4)
    got2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    _rows_close(got2, torch.stack([ref["c"][69], ref["a"][21]]), 1e-4)
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "generate"), "--model", str(model), "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, seq["b"])), "--max-new-tokens", "4", "--max-tokens", "256",
                        "--slots", "2"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    s = list(seq["b"])
    for _ in range(4):
        s.append(int(O.forward(cfg, ck, s)[-1].argmax()))
    assert lines[0] == {"request": 0, "tokens": s[len(seq["b"]):]}
