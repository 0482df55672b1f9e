"""Mutirax on the GPU against the plain float64 oracle (tests/mutirax_oracle.py): every mechanism alone through the C ABI,
then whole models of several shapes through the engine, its caches, its per-sequence state and the scheduler."""
import json
import math
import os

import pytest
import torch

import mutirax_oracle as O
from test_gpu_ninisun import Paged, _close, _i32, _rows_close, _tokens

pytestmark = pytest.mark.gpu
F64 = torch.float64
PAGE = 64
TOL = {torch.float32: 3e-5, torch.bfloat16: 5e-2}
CT = {torch.float32: 0, torch.bfloat16: 1}
DTYPES = [torch.float32, torch.bfloat16]


def _lib():
    from pg_b200 import _cabi as cabi
    return cabi, cabi.lib(), cabi.stream()


def _engine(cfg, seed=0, dtype=torch.float32, pool_tokens=1024, **kw):
    from pg_b200.mutirax import MutiraxEngine
    ck = O.make_checkpoint(cfg, seed)
    return MutiraxEngine(cfg, ck, device="cuda:0", dtype=dtype, kv_pool_tokens=pool_tokens, **kw), ck


def _segs(lens, slots):
    segs, row = [], 0
    for n, s in zip(lens, slots):
        segs += [s, row, n]
        row += n
    return segs


def _p(t):
    return None if t is None else t.data_ptr()


def _al(n):
    return (n + 7) // 8 * 8


# ------------------------------------------------------------------ mechanisms alone (C ABI)
@pytest.mark.parametrize("S,D", [(1, 48), (2, 1000), (3, 50), (4, 256), (4, 2100), (5, 64), (6, 36), (7, 520), (8, 128), (11, 40)])
@pytest.mark.parametrize("rows", [3, 400])
@pytest.mark.parametrize("dtype", DTYPES)
def test_row_kernel_between_sublayers(S, D, rows, dtype):
    """Streams from the embedding, dense / expert / paired outputs, the operand and its norm, picked rows, an id outside the
    vocabulary; stream counts and widths that take every variant of the kernel."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(100 * S + D + rows)
    V, top, eps, m = 17, 3, 1e-3, 0.6
    rnd = lambda *s: torch.randn(*s, generator=g)
    x0, y, y2 = rnd(rows, S, D), rnd(rows, D + 8).to(dtype), (3 * rnd(rows, D)).to(dtype)
    table, ey = rnd(V, D).to(dtype), rnd(rows * top, D).to(dtype)
    places, ew = torch.randperm(rows * top, generator=g).to(torch.int32), torch.rand(rows * top, generator=g)
    places[2 * top] = -1
    mix, wo, wi = rnd(S, S), rnd(S), rnd(S)
    alpha, w, b, n1, n2 = torch.tensor([0.4]), (1 + 0.3 * rnd(D)).to(dtype), rnd(D).to(dtype), (1 + 0.3 * rnd(D)).to(dtype), rnd(D).to(dtype)
    ids = torch.randint(0, V, (rows,), generator=g)
    dv = {k: v.cuda() for k, v in dict(y=y, y2=y2, table=table, ey=ey, places=places, ew=ew, mix=mix, wo=wo * m, w_in=torch.cat([wi, alpha]),
                                       w=w, b=b, n1=n1, n2=n2, ids=ids).items()}
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    f = lambda t: t.to(F64)
    tol = 4e-3 if dtype == torch.bfloat16 else 3e-6

    def call(x, out, *, y=None, ldy=0, pos=None, pair=False, ids=None, idx=None, n=rows, ldo=None):
        cabi.check(L.pg_hyper_connect(_p(out), D if ldo is None else ldo, x.data_ptr(), S, _p(y), ldy, _p(pos), _p(dv["ew"]) if pos is not None else None,
                                      top, _p(dv["y2"]) if pair else None, D, _p(dv["n1"]), _p(dv["n2"]), eps, 0.5, _p(ids), dv["table"].data_ptr(), V,
                                      dv["mix"].data_ptr(), dv["wo"].data_ptr(), dv["w_in"].data_ptr(), dv["w"].data_ptr(), dv["b"].data_ptr(), _p(idx),
                                      n, D, err.data_ptr(), CT[dtype], st))
    new = lambda n, c=D: torch.zeros(n, c, dtype=dtype, device="cuda")
    W = {"n": w.float(), "n.b": b.float(), "n.alpha": alpha[0]}
    operand = lambda streams: O.dyt(O.hyper_read(streams, wi), W, "n")
    str_ = lambda x: f(x).transpose(0, 1)                         # [rows, S, D] -> [S, rows, D]
    emb = f(table)[ids][None].repeat(S, 1, 1)
    # the first operand: every stream is the embedding row; the streams are neither read nor written
    x, out = torch.full((rows, S, D), float("nan"), device="cuda"), new(rows)
    call(x, out, ids=dv["ids"])
    _close(out, operand(emb), tol)
    assert bool(torch.isnan(x).all())
    # the first sum: from the embedding rows into the streams
    call(x, out, y=dv["y"], ldy=D + 8, ids=dv["ids"])
    want = O.hyper_write(emb, mix, wo, f(y)[:, :D], m)
    _close(str_(x.cpu()), want, 1e-6)
    _close(out, operand(want), tol)
    # a dense output; the operand in rows with a gap
    x, out = x0.cuda(), new(rows, D + 4)
    call(x, out, y=dv["y"], ldy=D + 8, ldo=D + 4)
    want = O.hyper_write(str_(x0), mix, wo, f(y)[:, :D], m)
    _close(str_(x.cpu()), want, 1e-6)
    _close(out[:, :D], operand(want), tol)
    assert float(out[:, D:].abs().max()) == 0
    # expert rows through their places and weights, one place missing
    moe = torch.zeros(rows, D, dtype=F64)
    for i, p in enumerate(places.tolist()):
        if p >= 0:
            moe[i // top] += float(ew[i]) * f(ey)[p]
    x, out = x0.cuda(), new(rows)
    call(x, out, y=dv["ey"], ldy=D, pos=dv["places"])
    want = O.hyper_write(str_(x0), mix, wo, moe, m)
    _close(str_(x.cpu()), want, 1e-6)
    _close(out, operand(want), tol)
    # two branches, each normed over the row
    x, out = x0.cuda(), new(rows)
    call(x, out, y=dv["y"], ldy=D + 8, pair=True)
    both = 0.5 * (O.rms(f(y)[:, :D], n1.float(), eps) + O.rms(f(y2), n2.float(), eps))
    want = O.hyper_write(str_(x0), mix, wo, both, m)
    _close(str_(x.cpu()), want, 1e-6)
    _close(out, operand(want), tol)
    # picked rows (one of them twice): the sum enters the result, the streams stay
    idx = [rows - 1, 0, rows - 1]
    x, out = x0.cuda(), new(3)
    call(x, out, y=dv["y"], ldy=D + 8, pair=True, idx=_i32(idx), n=3)
    assert torch.equal(x.cpu(), x0)
    _close(out, operand(want)[idx], tol)
    # the sum alone; the operand alone
    x = x0.cuda()
    call(x, None, y=dv["ey"], ldy=D, pos=dv["places"])
    _close(str_(x.cpu()), O.hyper_write(str_(x0), mix, wo, moe, m), 1e-6)
    x, out = x0.cuda(), new(rows)
    call(x, out)
    _close(out, operand(str_(x0)), tol)
    torch.cuda.synchronize()
    assert int(err) == 0
    ids2 = ids.clone()
    ids2[1] = V
    x = x0.cuda()
    call(x, None, y=dv["y"], ldy=D + 8, ids=ids2.cuda())
    torch.cuda.synchronize()
    assert int(err) == 1
    _close(x[1].cpu().to(F64), (m * wo.to(F64)[:, None] * f(y)[1, :D]), 1e-6)     # a zero row


def _gla_run(cabi, L, st, rows, cols, rank, a2, b2, tau, H, d, e, S, segs, dtype):
    T, ld = rows.shape
    rec = torch.empty(L.pg_gla_record_floats(T, H, d, e), device="cuda")
    cabi.check(L.pg_gla_prep(rec.data_ptr(), rows.data_ptr(), ld, cols[0], cols[1], cols[2], cols[3], rank, a2.data_ptr(), b2.data_ptr(),
                             d ** -0.5, 1.0 / tau, T, H, d, e, CT[dtype], st))
    o = torch.zeros(T, H * e, device="cuda")
    cabi.check(L.pg_gla_attention(o.data_ptr(), S.data_ptr(), rec.data_ptr(), _i32(segs).data_ptr(), len(segs) // 3, H, d, e, st))
    return o


@pytest.mark.parametrize("H,d,e,rank,tau", [(4, 8, 6, 8, 16.0), (1, 12, 20, 5, 1.0), (3, 64, 32, 16, 4.0), (2, 7, 9, 3, 8.0), (5, 128, 130, 24, 2.0),
                                            (2, 6, 3, 1, 0.5), (1, 200, 16, 40, 16.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_linear_attention_over_portions_and_slots(H, d, e, rank, tau, dtype):
    """Decays per key channel, the scan and its state: two sequences in portions side by side, one of them in a slot that
    another sequence left, against whole sequences."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(H * 1000 + d)
    cols = [0, _al(H * d), 2 * _al(H * d), 2 * _al(H * d) + _al(H * e)]
    ld, lens = cols[3] + _al(rank), {"a": 75, "b": 12}
    proj = {k: (torch.randn(n, ld, generator=g) * 1.5).to(dtype) for k, n in lens.items()}
    a2, b2 = (torch.randn(H * d, rank, generator=g) * 2 / math.sqrt(rank)).to(dtype), (2.0 * torch.randn(H * d, generator=g)).to(dtype)
    want = {}
    for k, n in lens.items():
        u = proj[k].to(F64)
        z = u[:, cols[3]:cols[3] + rank] @ a2.to(F64).T + b2.to(F64)
        want[k] = O.gla_scan(u[:, :H * d].view(n, H, d) / math.sqrt(d), u[:, cols[1]:cols[1] + H * d].view(n, H, d),
                             (O.sigmoid(z) ** (1.0 / tau)).view(n, H, d), u[:, cols[2]:cols[2] + H * e].view(n, H, e)).reshape(n, H * e)
    a2d, b2d = a2.cuda(), b2.cuda()
    S = torch.zeros(2, H, d, e, device="cuda")
    slot = {"a": 1, "b": 0}
    S[0].normal_()                                        # what an earlier sequence left
    plan = [[("a", 2)], [("a", 1)], [("b", 1), ("a", 3)], [("a", 60), ("b", 2)], [("b", 8), ("a", 1)], [("a", 8), ("b", 1)]]
    fed, got = {k: 0 for k in lens}, {k: [] for k in lens}
    for step in plan:
        for k, _ in step:
            if fed[k] == 0:
                S[slot[k]].zero_()
        rows = torch.cat([proj[k][fed[k]:fed[k] + n] for k, n in step]).cuda()
        o = _gla_run(cabi, L, st, rows, cols, rank, a2d, b2d, tau, H, d, e, S, _segs([n for _, n in step], [slot[k] for k, _ in step]) + [0, 0, 0],
                     dtype)
        at = 0
        for k, n in step:
            got[k].append(o[at:at + n].cpu())
            at += n
            fed[k] += n
    for k, n in lens.items():
        assert fed[k] == n
        _rows_close(torch.cat(got[k]), want[k], 2e-5)


def test_gated_linear_attention_keeps_one_channel_and_drops_the_other():
    """Channel 0 decays by almost nothing, channel 1 by half a token: what the first token wrote is read 700 tokens later in the
    one and gone in the other, whole or cut into portions."""
    cabi, L, st = _lib()
    H, d, e, T, rank = 1, 2, 8, 701, 1
    cols, ld = [0, 8, 16, 24], 32
    proj = torch.zeros(T, ld)
    proj[0, 8:10], proj[0, 16:24] = 3.0, 2.0              # k and v of the first token
    for ask in (0, 1):
        rows = proj.clone()
        rows[T - 1, ask] = 1.0                            # the last token asks one channel
        a2, b2 = torch.zeros(2, 1).cuda(), torch.tensor([12.0, 0.0]).cuda()
        a = O.sigmoid(torch.tensor([12.0, 0.0], dtype=F64)) ** 0.5
        want = 3.0 * 2.0 * float(a[ask]) ** (T - 1) / math.sqrt(2.0)
        for cuts in ([T], [1, 2, 61, 64, 200, 2, 1, 369, 1]):
            assert sum(cuts) == T
            S, at = torch.zeros(1, H, d, e, device="cuda"), 0
            for n in cuts:
                o = _gla_run(cabi, L, st, rows[at:at + n].cuda(), cols, rank, a2, b2, 2.0, H, d, e, S, [0, 0, n], torch.float32)
                at += n
            assert (want > 4.0) == (ask == 0)
            if ask == 0:
                _close(o[-1], torch.full((e,), want, dtype=F64), 2e-4)     # 700 steps with a decay rounded to 24 bits
            else:
                assert float(o[-1].abs().max()) < 1e-30



@pytest.mark.parametrize("H,G,d,rot,taps", [(4, 2, 16, 16, 4), (6, 3, 8, 8, 3), (3, 1, 48, 32, 2), (2, 2, 10, 6, 4), (5, 1, 6, 0, 5), (2, 1, 64, 64, 1),
                                            (4, 4, 24, 8, 8), (3, 1, 16, 16, 11), (1, 1, 17, 2, 3), (20, 5, 128, 128, 4), (30, 10, 128, 64, 4)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_convolved_norms_rotation_and_append(H, G, d, rot, taps, dtype):
    """Convolution, values, norm over the whole projection, rotation and paged rows of sequences in portions side by side (a
    long step, steps of two and one tokens, a slot used again), with more rows of state than this convolution needs."""
    cabi, L, st = _lib()
    from pg_b200.ragged_engine import RotaryCfg, rotary_pairs
    g = torch.Generator().manual_seed(H * 100 + d + taps)
    nq, nk, eps = H * d, G * d, 1e-3
    q0, k0 = 8, 8 + _al(nq)
    ld, cols = k0 + _al(nk) + 8, k0 - 8 + nk
    K, Ks = taps - 1, taps + 1                            # the state holds two rows more than K
    scols = cols + 5
    lens = {"a": 210, "b": 150, "c": 40}
    proj = {k: torch.randn(n, ld, generator=g).to(dtype) for k, n in lens.items()}
    conv = (torch.randn(taps, cols, generator=g)).to(dtype)
    qw, kw = (1 + 0.3 * torch.randn(nq, generator=g)).to(dtype), (1 + 0.3 * torch.randn(nk, generator=g)).to(dtype)
    f = O.frequencies(rot, 700.0)[0] if rot else None
    want = {}
    for k, n in lens.items():
        u = proj[k].to(F64)
        q = O.causal_conv(u[:, q0:q0 + nq], conv[:, :nq].T)
        kk = O.causal_conv(u[:, k0:k0 + nk], conv[:, k0 - q0:].T)
        v = kk
        q, kk = O.rms(q, qw, eps).view(n, H, d), O.rms(kk, kw, eps).view(n, G, d)
        if rot:
            q, kk = O.rotate(q, range(n), f), O.rotate(kk, range(n), f)
        want[k] = (q.reshape(n, nq), kk.reshape(n, nk), v)
    slot = {"a": 0, "b": 2, "c": 2}                       # c takes the slot that b left
    pg = Paged([lens["a"], 1, lens["b"]], nk, nk, dtype)
    state = torch.zeros(3, Ks, scols, device="cuda")
    state.normal_()
    freq = rotary_pairs(RotaryCfg(rot, 700.0)).cuda() if rot else None
    cd, qwd, kwd = conv.cuda(), qw.cuda(), kw.cuda()
    plan = [[("a", 2)], [("b", 1), ("a", 1)], [("a", 198), ("b", 140)], [("b", 2), ("a", 1)], [("a", 2), ("b", 7)], [("c", 3), ("a", 6)], [("c", 37)]]
    fed, got, pooled = {k: 0 for k in lens}, {k: [] for k in lens}, {}
    for step in plan:
        for k, _ in step:
            if fed[k] == 0:
                state[slot[k]].zero_()
        rows = torch.cat([proj[k][fed[k]:fed[k] + n] for k, n in step]).cuda()
        T = rows.shape[0]
        slots, pos = [slot[k] for k, n in step for _ in range(n)], [fed[k] + i for k, n in step for i in range(n)]
        q_out = torch.zeros(T, nq, dtype=dtype, device="cuda")
        cabi.check(L.pg_conv_qk_append(q_out.data_ptr(), rows.data_ptr(), ld, q0, H, k0, G, d, cd.data_ptr(), taps, state.data_ptr(), Ks, scols,
                                       qwd.data_ptr(), kwd.data_ptr(), eps, _p(freq), rot, pg.k.data_ptr(), pg.v.data_ptr(), pg.table.data_ptr(),
                                       pg.max_pages, PAGE, _i32(slots).data_ptr(), _i32(pos).data_ptr(), T, CT[dtype], st))
        segs = _segs([n for _, n in step], [slot[k] for k, _ in step]) + [0, 0, 0]
        wide = torch.zeros(T, scols, dtype=dtype, device="cuda")
        wide[:, :cols] = rows[:, q0:q0 + cols]
        cabi.check(L.pg_time_conv_state(state.data_ptr(), wide.data_ptr(), scols, 0, 0, _i32(segs).data_ptr(), len(segs) // 3, scols, Ks + 1,
                                        CT[dtype], st))
        at = 0
        for k, n in step:
            got[k].append(q_out[at:at + n].float().cpu())
            at += n
            fed[k] += n
            if fed[k] == lens[k]:
                r = pg.rows(slot[k], list(range(lens[k])))
                pooled[k] = (pg.k.view(-1, nk)[r].float().cpu(), pg.v.view(-1, nk)[r].float().cpu())
    tol = 6e-3 if dtype == torch.bfloat16 else 3e-6
    for k, n in lens.items():
        assert fed[k] == n
        _rows_close(torch.cat(got[k]), want[k][0], tol)
        _rows_close(pooled[k][0], want[k][1], tol)
        _rows_close(pooled[k][1], want[k][2], tol)


@pytest.mark.parametrize("taps", [2, 4, 7])
def test_convolution_reaches_exactly_its_taps(taps):
    """One token far above the others: visible taps - 1 tokens later and not one token further, in a prompt and with the step
    cut at every place around it."""
    cabi, L, st = _lib()
    d, n, at = 8, 30, 9
    for cuts in ([n], [at, n - at], [at + 1, n - at - 1], [at + 2, 1, n - at - 3], [at + taps - 1, n - at - taps + 1], [1] * n, [2] * (n // 2)):
        pg = Paged([n], d, d, torch.float32)
        state = torch.zeros(1, taps - 1, 2 * d, device="cuda")
        proj = torch.full((n, 2 * d), 0.01)
        proj[at] = 100.0
        conv, ones = torch.ones(taps, 2 * d, device="cuda"), None
        pd, pos = proj.cuda(), 0
        for c in cuts:
            q = torch.zeros(c, d, device="cuda")
            rows = pd[pos:pos + c].contiguous()
            cabi.check(L.pg_conv_qk_append(q.data_ptr(), rows.data_ptr(), 2 * d, 0, 1, d, 1, d, conv.data_ptr(), taps, state.data_ptr(), taps - 1,
                                           2 * d, ones, ones, 1e-6, None, 0, pg.k.data_ptr(), pg.v.data_ptr(), pg.table.data_ptr(), pg.max_pages,
                                           PAGE, _i32([0] * c).data_ptr(), _i32(list(range(pos, pos + c))).data_ptr(), c, 0, st))
            cabi.check(L.pg_time_conv_state(state.data_ptr(), rows.data_ptr(), 2 * d, 0, 0, _i32([0, 0, c]).data_ptr(), 1, 2 * d, taps, 0, st))
            pos += c
        v = pg.v.view(-1, d)[pg.rows(0, list(range(n)))].cpu()[:, 0]
        assert [i for i in range(n) if float(v[i]) > 50] == list(range(at, at + taps))
        assert abs(float(v[0]) - 0.01) < 1e-6             # nothing before the sequence


def _attn_case(H, G, d, lens, new, sinks, dtype=torch.float32, tower=None, seed=0, tc=False, scale=0.3):
    """Attention with a sink over keys and values of their own; tower: the place of a key far above the others for the last query."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(seed)
    pg = Paged(lens, G * d, G * d, dtype)
    qs, want, slots, positions = [], [], [], []
    sink = torch.tensor(sinks, dtype=torch.float32)
    for s, (n, m) in enumerate(zip(lens, new)):
        q, k, v = torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, G, d, generator=g)
        if tower is not None:
            j = tower(n - 1)
            k[:, :, 0] = 0.0
            k[j, :, 0] = 12.0
            q[n - 1, :, :] = 0.0
            q[n - 1, :, 0] = 10.0
            v[j] += 5.0
        q, k, v = q.to(dtype).float(), k.to(dtype).float(), v.to(dtype).float()
        pg.fill(s, k, v)
        outs = [O.softmax_attention(q[n - m:, h].to(F64), k[:, h // (H // G)].to(F64), v[:, h // (H // G)].to(F64), scale, sink[h], first=n - m)
                for h in range(H)]
        qs.append(q[n - m:].reshape(m, H * d))
        want.append(torch.stack(outs, 1).reshape(m, H * d))
        slots += [s] * m
        positions += list(range(n - m, n))
    q_all = torch.cat(qs).to(dtype).cuda()
    T = q_all.shape[0]
    out = torch.zeros(T, H * d, dtype=dtype, device="cuda")
    sd = sink.cuda()
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
            out.data_ptr(), H * d, q_all.data_ptr(), H * d, None, 0, 0, pg.k.data_ptr(), 0, pg.v.data_ptr(), 0, pg.k.shape[0] * PAGE,
            pg.table.data_ptr(), pg.max_pages, PAGE, _i32(tiles).data_ptr(), len(tiles) // 4, T, H, G, d, d, scale, 0, 0, 0, None, 0, None,
            sd.data_ptr(), 0.0, 0.0, 0, None, 0, 1.0, err.data_ptr(), CT[dtype], st))
        torch.cuda.synchronize()
        assert int(err) == 0
    else:
        ws = torch.empty(1 << 20, device="cuda")
        cabi.check(L.pg_attention_ragged_capped(
            out.data_ptr(), H * d, q_all.data_ptr(), H * d, None, 0, 0, pg.k.data_ptr(), 0, pg.v.data_ptr(), 0, pg.table.data_ptr(), pg.max_pages,
            PAGE, _i32(slots).data_ptr(), _i32(positions).data_ptr(), T, H, G, d, d, scale, 0, 0, 0, None, 0, None, sd.data_ptr(), 0.0, 0.0, 0,
            None, 0, 1.0, ws.data_ptr(), ws.numel(), CT[dtype], st))
    return out.float(), torch.cat(want)


@pytest.mark.parametrize("H,G,d", [(6, 2, 24), (3, 1, 40), (4, 4, 64), (10, 2, 72), (9, 3, 96), (2, 1, 128)])
@pytest.mark.parametrize("mode", ["prompt", "decode", "tc"])
def test_attention_with_sinks(H, G, d, mode):
    dtype = torch.bfloat16 if mode == "tc" else torch.float32
    case = dict(lens=[300, 64, 65, 1, 777], new=[1] * 5) if mode == "decode" else dict(lens=[200, 77, 64, 129], new=[200, 50, 64, 2])
    got, want = _attn_case(H, G, d, sinks=[3.0 - 1.5 * h for h in range(H)], dtype=dtype, seed=d, tc=mode == "tc", **case)
    _rows_close(got, want, 2e-2 if mode == "tc" else 3e-5)


@pytest.mark.parametrize("mode", ["prompt", "decode", "tc"])
@pytest.mark.parametrize("where", ["first", "page_end", "page_start", "previous", "self"])
def test_one_far_key_among_hundreds(mode, where):
    n = 331
    j = {"first": 0, "page_end": 191, "page_start": 192, "previous": n - 2, "self": n - 1}[where]
    dtype = torch.bfloat16 if mode == "tc" else torch.float32
    got, want = _attn_case(3, 1, 48, lens=[n], new=[1 if mode == "decode" else n], sinks=[1.0, 20.0, 40.0], dtype=dtype, tower=lambda _: j,
                           tc=mode == "tc")
    assert float(want[-1, :48].mean()) > 3.5 and float(want[-1, 96:].abs().max()) < 0.2       # the key takes the weight; a sink above it
    _rows_close(got, want, 2e-2 if mode == "tc" else 3e-5)


@pytest.mark.parametrize("rot,halves", [(8, 1), (8, 0), (64, 1), (2, 1)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_rows_and_rotated_query_columns(rot, halves, dtype):
    """Both pair layouts, far positions in fp32, the magnitude, norms of both latents and the paged rows."""
    cabi, L, st = _lib()
    from pg_b200.ragged_engine import RotaryCfg, rotary_pairs
    g = torch.Generator().manual_seed(rot)
    qr, kr, H, dim, mag, eps = 20, 24, 3, 5, 1.3, 1e-4
    pos, slots = [60001 % 190, 63, 64, 0], [0, 1, 1, 2]
    pg = Paged([200, 70, 1], 8 * ((kr + rot + 7) // 8), 1, dtype)
    ldp = pg.k.shape[2]
    proj = torch.randn(4, 80 + kr + rot, generator=g).to(dtype)
    wq, wk = (1 + 0.2 * torch.randn(qr, generator=g)).to(dtype), (1 + 0.2 * torch.randn(kr, generator=g)).to(dtype)
    pairs = rotary_pairs(RotaryCfg(rot, 11.0)).cuda()
    hi, lo = pairs[:, 0].contiguous(), pairs[:, 1].contiguous()
    cq = torch.zeros(4, qr, dtype=dtype, device="cuda")
    pd, wqd, wkd = proj.cuda(), wq.cuda(), wk.cuda()
    cabi.check(L.pg_latent_prep_ex(cq.data_ptr(), pd.data_ptr(), pd.stride(0), 8, qr, wqd.data_ptr(), 40, kr, wkd.data_ptr(), rot, hi.data_ptr(),
                                   lo.data_ptr(), halves, mag, eps, pg.k.data_ptr(), ldp, pg.table.data_ptr(), pg.max_pages, PAGE,
                                   _i32(slots).data_ptr(), _i32(pos).data_ptr(), 4, CT[dtype], st))
    u, f = proj.to(F64), O.frequencies(rot, 11.0)[0]
    order = torch.arange(rot) if halves else torch.arange(rot).view(rot // 2, 2).T.reshape(-1)     # pairs -> halves
    back = torch.argsort(order)
    turn = lambda x: O.rotate(x[..., order], pos, f, mag)[..., back]
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    _rows_close(cq, O.rms(u[:, 8:8 + qr], wq, eps), tol)
    flat = pg.k.view(-1, ldp)[[pg.rows(s, [p])[0] for s, p in zip(slots, pos)]]
    _rows_close(flat[:, :kr], O.rms(u[:, 40:40 + kr], wk, eps), tol)
    _rows_close(flat[:, kr:kr + rot], turn(u[:, 40 + kr:]), tol)
    pos = [60001, 33333, 1, 0]                            # one fp32 product alone would be some 2e-3 rad off
    q = torch.randn(4, H * (dim + rot), generator=g).to(dtype)
    dst, qd = torch.zeros(4, H * (kr + rot), dtype=dtype, device="cuda"), q.cuda()
    cabi.check(L.pg_rotary_cols_ex(dst.data_ptr(), dst.stride(0), kr, kr + rot, qd.data_ptr(), qd.stride(0), dim, dim + rot, H, rot, hi.data_ptr(),
                                   lo.data_ptr(), halves, mag, _i32(pos).data_ptr(), 4, CT[dtype], st))
    want = O.rotate(q.to(F64).view(4, H, dim + rot)[..., dim:][..., order], pos, f, mag)[..., back]
    _rows_close(dst.view(4, H, kr + rot)[..., kr:].reshape(4, -1), want.reshape(4, -1), tol)


@pytest.mark.parametrize("width,taps", [(16, 4), (18, 3), (13, 2), (64, 1), (24, 8), (20, 11), (2052, 4)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrent_unit_convolution(width, taps, dtype):
    """Portions, slots used again, state with rows to spare; the input bias does not reach before the sequence."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(width + taps)
    x0, ld = 16, 16 + _al(width)
    K, Ks, scols = taps - 1, taps + 1, width + (4 if width % 4 == 0 else 3)
    lens = {"a": 360, "b": 40}
    proj = {k: torch.randn(n, ld, generator=g).to(dtype) for k, n in lens.items()}
    bx, cb, conv = torch.full((width,), 3.0).to(dtype), torch.randn(width, generator=g).to(dtype), torch.randn(taps, width, generator=g).to(dtype)
    want = {k: O.causal_conv(proj[k].to(F64)[:, x0:x0 + width] + bx.to(F64), conv.T, cb) for k in lens}
    state, slot = torch.zeros(2, Ks, scols, device="cuda"), {"a": 1, "b": 0}
    state[0].normal_()
    bxd, cbd, cd = bx.cuda(), cb.cuda(), conv.cuda()
    plan = [[("a", 1)], [("b", 2), ("a", 2)], [("a", 300), ("b", 25)], [("b", 1), ("a", 1)], [("a", 56), ("b", 12)]]
    fed, got = {k: 0 for k in lens}, {k: [] for k in lens}
    for step in plan:
        for k, _ in step:
            if fed[k] == 0:
                state[slot[k]].zero_()
        rows = torch.cat([proj[k][fed[k]:fed[k] + n] for k, n in step]).cuda()
        T = rows.shape[0]
        slots, pos = [slot[k] for k, n in step for _ in range(n)], [fed[k] + i for k, n in step for i in range(n)]
        u = torch.zeros(T, width, dtype=dtype, device="cuda")
        cabi.check(L.pg_lru_conv(u.data_ptr(), rows.data_ptr(), ld, x0, bxd.data_ptr(), cd.data_ptr(), cbd.data_ptr(), taps, state.data_ptr(), Ks,
                                 scols, _i32(slots).data_ptr(), _i32(pos).data_ptr(), T, width, CT[dtype], st))
        wide = torch.zeros(T, scols, dtype=dtype, device="cuda")
        wide[:, :width] = rows[:, x0:x0 + width]
        segs = _segs([n for _, n in step], [slot[k] for k, _ in step]) + [0, 0, 0]
        cabi.check(L.pg_time_conv_state(state.data_ptr(), wide.data_ptr(), scols, 0, 0, _i32(segs).data_ptr(), len(segs) // 3, scols, Ks + 1,
                                        CT[dtype], st))
        at = 0
        for k, n in step:
            got[k].append(u[at:at + n].float().cpu())
            at += n
            fed[k] += n
    for k, n in lens.items():
        assert fed[k] == n
        _rows_close(torch.cat(got[k]), want[k], 5e-3 if dtype == torch.bfloat16 else 2e-6)


def _lru_case(width, blocks, lens_slots, S, dtype, impl, seed=0, lam=None, zscale=1.0, cuts=None):
    """Runs the recurrence over sequences [(tokens, slot)]; cuts: portions per step for each sequence (None: whole)."""
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(seed)
    bs = width // blocks
    lam = torch.randn(width, generator=g) * 3 - 3 if lam is None else lam
    yb, rb, ib = (torch.randn(width, generator=g).to(dtype) for _ in range(3))
    seqs = []
    for n, slot in lens_slots:
        z, u, y = zscale * torch.randn(n, blocks, 2, bs, generator=g), torch.randn(n, width, generator=g).to(dtype), torch.randn(n, width + 8, generator=g).to(dtype)
        r = O.sigmoid(z[:, :, 0].reshape(n, width).to(F64) + rb.to(F64))
        i = O.sigmoid(z[:, :, 1].reshape(n, width).to(F64) + ib.to(F64))
        a = torch.exp(-8.0 * r * O.softplus(lam.to(F64)))
        want = O.lru_scan(a, i * u.to(F64)) * O.gelu_tanh(y[:, :width].to(F64) + yb.to(F64))
        seqs.append((slot, z, u, y, want))
    dv = {k: v.cuda() for k, v in dict(lam=lam.float(), yb=yb, rb=rb, ib=ib).items()}
    steps = [[n for n, _ in lens_slots]] if cuts is None else cuts
    fed, got = [0] * len(seqs), [[] for _ in seqs]
    for step in steps:
        take = [(s, n) for s, n in enumerate(step) if n]
        cat = lambda idx: torch.cat([seqs[s][idx][fed[s]:fed[s] + n] for s, n in take]).cuda()
        z, u, y = cat(1), cat(2), cat(3)
        T = z.shape[0]
        segs = _segs([n for _, n in take], [seqs[s][0] for s, _ in take]) + [0, 0, 0, 0, 0, 0]
        ns = len(segs) // 3
        out = torch.zeros(T, width, dtype=dtype, device="cuda")
        ws = torch.full((L.pg_lru_ws_floats(T, ns, width),), float("nan"), device="cuda")
        cabi.check(L.pg_lru_scan(out.data_ptr(), width, S.data_ptr(), z.data_ptr(), u.data_ptr(), y.data_ptr(), width + 8, dv["yb"].data_ptr(),
                                 dv["rb"].data_ptr(), dv["ib"].data_ptr(), dv["lam"].data_ptr(), 8.0, _i32(segs).data_ptr(), ns, T, width, blocks,
                                 ws.data_ptr(), impl, CT[dtype], st))
        at = 0
        for s, n in take:
            got[s].append(out[at:at + n].float().cpu())
            at += n
            fed[s] += n
    return [(torch.cat(x), q[4]) for x, q in zip(got, seqs)]


@pytest.mark.parametrize("width,blocks", [(16, 2), (24, 8), (13, 1), (30, 5), (256, 4), (2048, 8)])
@pytest.mark.parametrize("impl", [0, 1, 2])
@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrent_unit_token_by_token_and_chunked(width, blocks, impl, dtype):
    """Lengths around the chunk size, several segments, a slot with what another sequence left, portions that carry the state."""
    S = torch.zeros(6, width, device="cuda")
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-5
    for got, want in _lru_case(width, blocks, [(31, 3), (32, 0), (33, 5), (1, 2), (97, 1), (64, 4)], S, dtype, impl, seed=width):
        _rows_close(got, want, tol)
    S.normal_()
    S[1].zero_(), S[4].zero_()
    left = S[[0, 2, 3, 5]].clone()
    for got, want in _lru_case(width, blocks, [(150, 4), (75, 1)], S, dtype, impl, seed=width + 1,
                               cuts=[[2, 0], [1, 33], [95, 2], [32, 1], [0, 38], [20, 1]]):
        _rows_close(got, want, tol)
    assert torch.equal(S[[0, 2, 3, 5]], left)             # other slots stay


@pytest.mark.parametrize("impl", [1, 2])
def test_recurrent_unit_with_decays_close_to_one(impl):
    """softplus(lam) down to 1e-6: 1 - a^2 must not come from a difference of numbers near 1, and a token is still there 700
    tokens later; large lam forgets within a token."""
    lam = torch.linspace(-14.0, 4.0, 32)
    S = torch.zeros(2, 32, device="cuda")
    (got, want), = _lru_case(32, 4, [(701, 1)], S, torch.float32, impl, seed=5, lam=lam)
    _rows_close(got.T, want.T, 4e-5)
    S.zero_()
    (got, want), = _lru_case(32, 4, [(701, 1)], S, torch.float32, impl, seed=5, lam=lam, cuts=[[1], [2], [61], [64], [200], [2], [1], [369], [1]])
    _rows_close(got.T, want.T, 4e-5)


@pytest.mark.parametrize("T,heads,N,K,dtype,impl", [(3, 4, 20, 10, torch.float32, 0), (40, 3, 24, 12, torch.bfloat16, 0), (5, 2, 64, 32, torch.bfloat16, 0),
                                                    (200, 4, 64, 32, torch.bfloat16, 2), (130, 2, 200, 104, torch.bfloat16, 2),
                                                    (70, 1, 16, 264, torch.bfloat16, 2), (100, 3, 18, 9, torch.float32, 0)])
def test_per_head_products_unrounded(T, heads, N, K, dtype, impl):
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(N)
    a, w = torch.randn(T, heads * K + 8, generator=g).to(dtype), torch.randn(heads, N, K, generator=g).to(dtype)
    out, err = torch.full((T, heads * N + 8), 5.0, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    ad, wd = a.cuda(), w.cuda()
    cabi.check(L.pg_head_gemm_f32(out.data_ptr(), heads * N + 8, N, ad.data_ptr(), heads * K + 8, K, wd.data_ptr(), T, heads, N, K, impl,
                                  err.data_ptr(), CT[dtype], st))
    want = torch.einsum("thk,hnk->thn", a.to(F64)[:, :heads * K].view(T, heads, K), w.to(F64)).reshape(T, heads * N)
    _close(out[:, :heads * N], want, 2e-6)                # 16-bit operands too: nothing is rounded on the way out
    torch.cuda.synchronize()
    assert int(err) == 0 and bool((out[:, heads * N:] == 5.0).all())


@pytest.mark.parametrize("T,D,E,top", [(1, 64, 8, 2), (5, 50, 3, 3), (40, 33, 70, 5), (400, 128, 20, 1), (301, 72, 5, 4)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_router_softmax_over_the_chosen(T, D, E, top, dtype):
    cabi, L, st = _lib()
    g = torch.Generator().manual_seed(T + E)
    h, w, b = torch.randn(T, D + 8, generator=g).to(dtype), (2 * torch.randn(E, D, generator=g) / math.sqrt(D)).to(dtype), torch.randn(E, generator=g).to(dtype)
    ref_idx, ref_w = O.route(h[:, :D].to(F64), {"router": w, "router.b": b}, "", top)
    hd, wd, bd = h.cuda(), w.cuda(), b.cuda()
    given = (h[:, :D].double() @ w.double().T).float().cuda()
    for z in (None, given):
        idx, wts = torch.full((T, top), -1, dtype=torch.int32, device="cuda"), torch.zeros(T, top, device="cuda")
        cabi.check(L.pg_moe_route_topk(idx.data_ptr(), wts.data_ptr(), _p(z), hd.data_ptr(), D + 8, wd.data_ptr(), bd.data_ptr(), T, D, E, top,
                                       CT[dtype], st))
        assert torch.equal(idx.cpu().long(), ref_idx)
        _close(wts, ref_w, 3e-6)
    flat = torch.zeros(T, E, device="cuda")               # ties: the lowest index first, equal weights
    cabi.check(L.pg_moe_route_topk(idx.data_ptr(), wts.data_ptr(), flat.data_ptr(), None, 0, None, None, T, D, E, top, CT[dtype], st))
    assert torch.equal(idx.cpu(), torch.arange(top, dtype=torch.int32).repeat(T, 1))
    _close(wts, torch.full((T, top), 1.0 / top, dtype=F64), 1e-6)


@pytest.mark.parametrize("F", [64, 50, 1032])
@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_pairing(F, dtype):
    cabi, L, st = _lib()
    gu = (torch.randn(37, 2 * F, generator=torch.Generator().manual_seed(F)) * 4).to(dtype)
    out, gd = torch.zeros(37, F, dtype=dtype, device="cuda"), gu.cuda()
    cabi.check(L.pg_glu_clamped(out.data_ptr(), gd.data_ptr(), 37, F, 2.5, 1.702, CT[dtype], st))
    u = gu.to(F64)
    g, v = u[:, :F].clamp(max=2.5), u[:, F:].clamp(-2.5, 2.5)
    _close(out, g * O.sigmoid(1.702 * g) * (v + 1.0), 6e-3 if dtype == torch.bfloat16 else 1e-6)


# ------------------------------------------------------------------ whole models
CONFIGS = {
    # every branch: the three mixers, both feed-forwards and none, a looped block in the middle, grouped key heads, part of the
    # head rotated, branches with other numbers of taps
    "small": O.make_config(width=48, vocab=61, streams=3, m=0.8, loop=(1, 3, 2), layers=[
        O.layer(O.parallel(heads=4, kv_heads=2, dim=12, width=24, blocks=3, conv=4, rconv=3, rot_dims=8), O.dense(40)),
        O.layer(O.gla(heads=3, dim=8, vdim=6, tau=4.0), O.moe(5, 2, 16)),
        O.layer(O.latent(heads=2, dim=8, rot_dim=4, vdim=10, q_rank=12, kv_rank=14), O.moe(4, 1, 12)),
        O.layer(O.parallel(heads=2, kv_heads=1, dim=8, width=16, blocks=2, conv=2, rconv=5)),
        O.layer(O.gla(heads=2, dim=6, vdim=10, tau=1.0), O.dense(24, limit=0.5))]),
    # values the other configurations make equal or 1: one stream, one head, one block, one tap, every expert chosen, a loop that
    # holds the first layer and all others, three passes, no frequency scaling, sizes off every multiple
    "odd": O.make_config(width=50, vocab=67, streams=1, m=1.3, loop=(0, 3, 3), eps=1e-3, layers=[
        O.layer(O.latent(heads=1, dim=5, rot_dim=6, vdim=7, q_rank=9, kv_rank=11, scaling=None, scale=0.5), O.moe(3, 3, 9)),
        O.layer(O.parallel(heads=5, kv_heads=5, dim=6, width=15, blocks=1, conv=1, rconv=1, rot_dims=2, base=50.0)),
        O.layer(O.gla(heads=1, dim=10, vdim=13, tau=0.7), O.dense(30, limit=1.0))]),
    # no looped block, more streams than the row kernel's fast path; each mixer once without a feed-forward behind it
    "flat": O.make_config(width=64, vocab=90, streams=9, m=0.5, layers=[
        O.layer(O.gla(heads=4, dim=16, vdim=16)),
        O.layer(O.latent(heads=4, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scaling=(8.0, 32, 4.0, 1.0))),
        O.layer(O.parallel(heads=3, kv_heads=1, dim=24, width=40, blocks=5, conv=9, rconv=2), O.moe(6, 4, 16)),
        O.layer(O.gla(heads=2, dim=8, vdim=24), O.moe(1, 1, 20))]),
    # head sizes of real models: the 16-bit run crosses the tensor-core attention (whole and filled-up tiles), the tensor-core
    # GEMMs, per-head products and experts
    "wide": O.make_config(width=256, vocab=300, streams=4, m=0.9, loop=(1, 4, 2), layers=[
        O.layer(O.latent(heads=4, dim=64, rot_dim=32, vdim=64, q_rank=96, kv_rank=96), O.dense(256)),
        O.layer(O.parallel(heads=4, kv_heads=2, dim=64, width=256, blocks=4), O.moe(8, 2, 128)),
        O.layer(O.gla(heads=4, dim=64, vdim=64), O.moe(6, 3, 64)),
        O.layer(O.parallel(heads=3, kv_heads=1, dim=104, width=128, blocks=2, conv=3, rconv=4, rot_dims=64), O.dense(128)),
        O.layer(O.latent(heads=2, dim=32, rot_dim=64, vdim=128, q_rank=64, kv_rank=128), O.moe(3, 1, 128))]),
    # no attention without state and none with: linear attention alone, and latent attention alone
    "linear": O.make_config(width=32, vocab=40, streams=2, loop=(0, 1, 2), layers=[O.layer(O.gla(heads=2, dim=8, vdim=8), O.dense(16))]),
    "latent": O.make_config(width=32, vocab=40, streams=2, layers=[O.layer(O.latent(heads=2, dim=8, rot_dim=4, vdim=8, q_rank=8, kv_rank=16), O.moe(4, 2, 16)),
                                                                   O.layer(O.latent(heads=1, dim=4, rot_dim=8, vdim=8, q_rank=8, kv_rank=8))]),
}
_ORACLE_CACHE = {}


def _stray(name, dtype):
    """16-bit runs: rows that may differ.  A linear-attention head's output is normed by its own length: at the first positions
    it is v (q . k) over its rms, so with q . k near zero the sign of a head is a matter of rounding the projections; and two
    experts' logits may lie within that rounding.  "odd" has a single head, whose sign is all there is (the oracle with its
    projections rounded to bf16 strays in a fifth of its rows)."""
    if dtype == torch.float32:
        return 0.0
    return 0.2 if name == "odd" else 0.08


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
    assert [r.layer for r in eng.runs] == O.run_order(CONFIGS[name])
    if name == "wide" and dtype == torch.bfloat16:
        assert [bool(w["attn_tc"]) for w in eng.layers] == [True, True, False, True, True]
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
        _rows_close(torch.cat(got[k]), ref[k][1], TOL[dtype] * 2, _stray(name, dtype))
    b.close()
    assert eng.pages_in_use() == 0


def test_long_decoding_through_pages():
    name, n = "small", 330
    toks, want, _ = _oracle(name, n)
    for dtype in DTYPES:
        eng, _ = _engine(CONFIGS[name], dtype=dtype)
        b = eng.new_batcher(slots=1)
        b.admit("a")
        rows = [b.run_entries([("a", toks[:5], list(range(5)))])]
        rows += [b.run_entries([("a", [t], [0])]) for t in toks[5:]]
        _rows_close(torch.cat(rows), want, TOL[dtype] * 2, _stray(name, dtype))
        b.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_crosses_the_prompt_sized_kernels(dtype):
    """More than 296 tokens in one step (tiled rows, chunked recurrence, router logits as a GEMM of their own) beside a second
    prompt and a decoding sequence, then single tokens after it."""
    name, n = "wide", 340
    toks, want, _ = _oracle(name, n)
    t2, w2, _ = _oracle(name, 150, seed=1)
    eng, _ = _engine(CONFIGS[name], dtype=dtype)
    b = eng.new_batcher(slots=3)
    for k in "abc":
        b.admit(k)
    b.run_entries([("c", t2[:149], [])])
    out = b.run_entries([("a", toks[:330], list(range(330))), ("c", [t2[149]], [0]), ("b", t2[:70], list(range(70)))])
    rest = torch.cat([b.run_entries([("a", [t], [0])]) for t in toks[330:]])
    tol, stray = TOL[dtype] * 2, _stray(name, dtype)
    _rows_close(torch.cat([out[:330], rest]), want, tol, stray)
    _rows_close(out[331:], w2[:70], tol, stray)
    _rows_close(out[330:331], w2[149:150], tol * (1 if dtype == torch.float32 else 4))
    eng.check_errors(sync=True)
    b.close()


def test_every_pass_of_the_loop_has_its_own_cache_and_state():
    cfg = CONFIGS["small"]
    eng, _ = _engine(cfg)
    assert sorted(eng.c_pools) == [2, 4] and sorted(eng.k_pools) == sorted(eng.v_pools) == [0, 5]      # run order: 0, 1, 2, 1, 2, 3, 4
    b = eng.new_batcher(slots=2)
    s = b.kv.state.layers
    assert sorted(s) == sorted([("gla", 1), ("gla", 3), ("gla", 6), ("lru", 0), ("lru", 5), ("conv", 0), ("conv", 5)])
    assert s[("gla", 1)].shape == (2, 3, 8, 6) and s[("lru", 5)].shape == (2, 16) and s[("conv", 0)].shape == (2, 3, 48 + 24 + 24)
    assert s[("conv", 5)].shape[1] == 4                    # the longer of the two convolutions
    b.admit("a")
    b.run_entries([("a", _tokens(70, 61, 1), [])])
    assert all(float(t[0].abs().max()) > 0 and float(t[1].abs().max()) == 0 for t in s.values())
    assert not torch.equal(s[("gla", 1)], s[("gla", 3)]) and not torch.equal(eng.c_pools[2], eng.c_pools[4])
    b.finish("a")
    b.admit("again")                                      # the slot is handed on with a zero state
    assert all(float(t[0].abs().max()) == 0 for t in s.values())
    b.close()


def test_decoding_with_a_second_slot_table_uses_its_own_state():
    """Small steps replay captured graphs; every scheduler brings a slot table and a state of its own."""
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
        kind = rng.choice(["gla", "latent", "parallel"])
        if kind == "gla":
            L = O.gla(heads=rng.choice([1, 2, 3, 4, 8]), dim=rng.choice([16, 24, 32, 64, 128]), vdim=rng.choice([16, 32, 40, 64, 128]),
                      tau=rng.choice([1.0, 2.0, 8.0, 16.0]))
        elif kind == "latent":
            L = O.latent(heads=rng.choice([1, 2, 3, 4, 6]), dim=rng.choice([16, 32, 48, 64]), rot_dim=rng.choice([8, 16, 32, 64]),
                         vdim=rng.choice([16, 32, 64, 96]), q_rank=rng.choice([40, 64, 96]), kv_rank=rng.choice([32, 64, 80, 128, 192]),
                         base=rng.choice([1e4, 1e6]), scaling=rng.choice([(2.0, 64, 32.0, 1.0), (8.0, 512, 16.0, 2.0), (4.0, 100, 8.0, 0.5), None]))
        else:
            H, width = rng.choice([2, 4, 6, 8]), rng.choice([64, 96, 128, 192])
            L = O.parallel(heads=H, kv_heads=rng.choice(div(H)), dim=rng.choice([16, 32, 48, 64, 80, 96, 128]), width=width,
                           blocks=rng.choice([1, 2, 4, 8]), conv=rng.choice([2, 3, 4, 5]), rconv=rng.choice([2, 3, 4, 5]), base=rng.choice([1e4, 2e5]))
        E = rng.choice([2, 4, 8, 10, 16])
        layers.append(O.layer(L, rng.choice([None, O.dense(rng.choice([128, 256, 320]), rng.choice([1.0, 4.0])),
                                             O.moe(E, rng.randint(1, min(E, 4)), rng.choice([32, 64, 160]))])))
    a = rng.randrange(n)
    return O.make_config(width=rng.choice([128, 192, 256, 288]), vocab=rng.choice([300, 512]), layers=layers, streams=rng.choice([2, 3, 4, 5, 6]),
                         m=rng.choice([0.5, 1.0]), loop=rng.choice([None, (a, rng.randint(a + 1, n), rng.choice([2, 3]))]), eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
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
                _rows_close(out, want, 8e-2, 0.1)


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
    write_safetensors(str(model / "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in ck.items()})
    eng = load_engine(str(model), device="cuda:0", dtype=torch.float32, kv_pool_tokens=256)
    assert type(eng).__name__ == "MutiraxEngine"
    toks = _tokens(40, cfg["vocab"], 9)
    b = eng.new_batcher(slots=1)
    b.admit(0)
    _rows_close(b.run_entries([(0, toks, [39, 0])]), O.forward(cfg, ck, toks)[[39, 0]], 1e-3)
    b.close()
    make = lambda w, **kw: type(eng)(cfg, w, device="cuda:0", dtype=torch.float32, kv_pool_tokens=64, **kw)
    more = dict(ck)
    more["l0.mix.extra"] = torch.zeros(3)
    with pytest.warns(UserWarning):
        make(more)
    with pytest.raises(ValueError):
        make(more, strict=True)
    with pytest.raises(KeyError):
        make({k: v for k, v in ck.items() if k != "l1.mix.left.sink"})
    with pytest.raises(ValueError):
        make(dict(ck, **{"l0.hc1.mix": torch.zeros(2, 2)}))
    with pytest.raises(ValueError):
        make(dict(ck, **{"l2.mix.a1": torch.zeros(4, 49)}))
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
    _rows_close(got0, torch.stack([ref["a"][19], ref["b"][0], ref["b"][4]]), 1e-3)
    got2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    _rows_close(got2, torch.stack([ref["c"][69], ref["a"][21]]), 1e-3)
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "generate"), "--model", str(model), "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, seq["b"])), "--max-new-tokens", "4", "--max-tokens", "256",
                        "--slots", "2"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    s = list(seq["b"])
    for _ in range(4):
        s.append(int(O.forward(cfg, ck, s)[-1].argmax()))
    assert lines[0] == {"request": 0, "tokens": s[len(seq["b"]):]}
