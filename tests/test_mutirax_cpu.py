"""Host-side parts of the Mutirax path that need no GPU: config parsing, the registry, the frequency table, and the oracle's own
consistency (causality, what every mechanism contributes)."""
import math

import pytest
import torch

import mutirax_oracle as O
from pg_b200 import registry
from pg_b200.mutirax import MutiraxConfig
from pg_b200.ragged_engine import RotaryCfg, layer_runs, loop_cfg

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    cfg = O.make_config(width=40, vocab=77, eps=3e-4, streams=5, m=0.35, loop=(1, 3, 4), layers=[
        O.layer(O.parallel(heads=6, kv_heads=3, dim=10, width=21, blocks=7, conv=2, rconv=6, rot_dims=4, base=77.0, scale=0.2), O.dense(24, 1.5)),
        O.layer(O.gla(heads=3, dim=8, vdim=14, tau=2.5), O.moe(7, 3, 12)),
        O.layer(O.latent(heads=2, dim=4, rot_dim=6, vdim=5, q_rank=9, kv_rank=11, scale=0.7, base=30.0, scaling=(4.0, 99, 7.0, 0.5)))])
    c = MutiraxConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.eps, c.streams, c.residual_mult) == (77, 40, 3e-4, 5, 0.35)
    a, r = c.layers[0].mixer.left, c.layers[0].mixer.right
    assert (c.layers[0].kind, a.heads, a.kv_heads, a.dim, a.scale, a.taps, a.rot.dims, a.rot.base) == ("parallel", 6, 3, 10, 0.2, 2, 4, 77.0)
    assert (r.width, r.blocks, r.taps) == (21, 7, 6)
    g = c.layers[1].mixer
    assert (c.layers[1].kind, g.heads, g.dim, g.vdim, g.tau) == ("gla", 3, 8, 14, 2.5)
    m = c.layers[1].mlp
    assert (m.kind, m.experts, m.top, m.ff) == ("moe", 7, 3, 12)
    l = c.layers[2].mixer
    assert (c.layers[2].kind, l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.rot.base, l.window, l.halves) == \
        ("latent_attention", 2, 4, 6, 5, 9, 11, 0.7, 30.0, 0, True)
    assert l.rot.scaling == {"factor": 4.0, "original": 99, "fast": 7.0, "slow": 0.5}
    d = c.layers[0].mlp
    assert (d.kind, d.ff, d.limit, c.layers[2].mlp) == ("dense", 24, 1.5, None)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 4)
    assert registry.resolve(cfg).__name__ == "MutiraxEngine" and "Mutirax" in registry.architectures()


def test_config_rejects_what_the_design_does_not_have():
    def bad(layers, **kw):
        with pytest.raises(ValueError):
            MutiraxConfig.from_dict(O.make_config(width=16, vocab=20, layers=layers, **kw))
    par = lambda **kw: O.parallel(**dict(dict(heads=2, kv_heads=1, dim=4, width=8, blocks=2), **kw))
    ok = O.layer(par())
    bad([O.layer(par(heads=3, kv_heads=2))])
    bad([O.layer(par(rot_dims=6))])
    bad([O.layer(par(rot_dims=3))])
    bad([O.layer(par(conv=0))])
    bad([O.layer(par(rconv=0))])
    bad([O.layer(par(blocks=3))])
    apart = par()
    apart["mixer"]["left"]["vdim"] = 6                          # the values are the keys
    bad([O.layer(apart)])
    scaled = par()
    scaled["mixer"]["left"]["rot"]["scaling"] = {"factor": 2.0}   # frequencies are scaled in the latent mixer alone
    bad([O.layer(scaled)])
    turned = O.latent(heads=1, dim=4, rot_dim=4, vdim=4, q_rank=4, kv_rank=4)
    turned["mixer"]["rot"]["dims"] = 2                          # the rotated part is rotated whole
    bad([O.layer(turned)])
    bad([dict(ok, type="convolution")])
    bad([dict(ok, mlp={"kind": "router"})])
    bad([dict(ok, mlp=O.moe(2, 3, 4))])
    bad([ok], loop=(0, 2, 2))
    bad([ok], loop=(0, 1, 0))
    bad([ok], streams=0)


def test_run_order_and_frequencies_agree_with_the_oracle():
    for n, loop in ((5, (2, 3, 3)), (4, (0, 1, 1)), (3, (0, 3, 2)), (3, None)):
        cfg = {"layers": [0] * n}
        if loop:
            cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
        assert [r.layer for r in layer_runs(n, loop_cfg(cfg.get("loop"), n))] == O.run_order(cfg)
    for dims, base, sc in ((8, 1e4, None), (64, 1e6, dict(factor=2.0, original=1000, fast=32.0, slow=1.0)),
                           (16, 50.0, dict(factor=8.0, original=64, fast=4.0, slow=2.0))):
        f, mag = RotaryCfg(dims, base, sc).table()
        want, wmag = O.frequencies(dims, base, sc)
        assert torch.allclose(f, want, rtol=1e-14, atol=0) and abs(mag - wmag) < 1e-15


def test_oracle_hyper_connections_by_hand():
    """Two streams, one number each: the mix is indexed from, to, and all new streams come from the old ones."""
    x = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    mix = torch.tensor([[2.0, 3.0], [5.0, 7.0]])
    y = torch.tensor([[100.0]], dtype=F64)
    out = O.hyper_write(x, mix, torch.tensor([1.0, -1.0]), y, 0.5)
    assert out[:, 0, 0].tolist() == [2 * 1 + 5 * 10 + 50.0, 3 * 1 + 7 * 10 - 50.0]
    assert float(O.hyper_read(x, torch.tensor([4.0, 0.5]))) == 9.0


def test_oracle_gated_linear_attention_is_the_decayed_sum():
    g = torch.Generator().manual_seed(0)
    n, H, d, e = 9, 2, 4, 3
    q, k, v = (torch.randn(n, H, x, generator=g, dtype=F64) for x in (d, d, e))
    a = torch.rand(n, H, d, generator=g, dtype=F64)
    want = torch.zeros(n, H, e, dtype=F64)
    for i in range(n):
        for j in range(i + 1):
            decay = a[j + 1:i + 1].prod(0)
            want[i] += (q[i] * decay * k[j]).sum(-1)[:, None] * v[j]
    assert torch.allclose(O.gla_scan(q, k, a, v), want, atol=1e-12)


def test_oracle_recurrent_unit_by_hand():
    a, x = torch.tensor([[0.5], [0.8]], dtype=F64), torch.tensor([[2.0], [1.0]], dtype=F64)
    s0 = math.sqrt(0.75) * 2.0                              # also the first token is scaled
    assert torch.allclose(O.lru_scan(a, x)[:, 0], torch.tensor([s0, 0.8 * s0 + 0.6], dtype=F64), atol=1e-14)


def test_oracle_convolution_by_hand():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    w = torch.tensor([[2.0, 3.0]])
    assert O.causal_conv(u, w)[:, 0].tolist() == [3.0, 32.0, 320.0]
    assert O.causal_conv(u, w, torch.tensor([0.5]))[0, 0] == 3.5


def test_oracle_router_weights():
    h = torch.eye(3, dtype=F64)
    W = {"router": torch.tensor([[1.0, 0.0, 0.0], [2.0, 0.0, 5.0], [0.0, 1.0, 0.0]]), "router.b": torch.tensor([0.0, -3.0, 0.5])}
    idx, w = O.route(h, W, "", 2)
    assert idx.tolist() == [[0, 2], [2, 0], [1, 2]]         # the bias counts in the choice and in the weights
    assert abs(float(w[1, 0]) - 1 / (1 + math.exp(-1.5))) < 1e-12


def test_oracle_is_causal_and_every_mechanism_shows():
    """Later tokens change nothing earlier; leaving out one mechanism moves the logits (so that a test against the oracle would
    see it)."""
    cfg = O.make_config(width=24, vocab=30, streams=3, loop=(0, 2, 2), layers=[
        O.layer(O.parallel(heads=2, kv_heads=1, dim=8, width=12, blocks=3, conv=3, rconv=2, rot_dims=4), O.moe(4, 2, 8)),
        O.layer(O.latent(heads=2, dim=6, rot_dim=4, vdim=5, q_rank=8, kv_rank=10), O.dense(12, 1.0)),
        O.layer(O.gla(heads=2, dim=6, vdim=4))])
    ck = O.make_checkpoint(cfg, 2)
    toks = torch.randint(0, 30, (14,), generator=torch.Generator().manual_seed(3)).tolist()
    full = O.forward(cfg, ck, toks)
    assert torch.allclose(O.forward(cfg, ck, toks[:9]), full[:9], atol=1e-10)

    def moved(cfg2, **tensors):
        out = O.forward(cfg2, dict(ck, **{k.replace("__", "."): v for k, v in tensors.items()}), toks)
        return float((out - full)[5:].abs().amax(-1).min())

    def mixer(i, side=None, **kw):
        layers = [dict(L) for L in cfg["layers"]]
        m = dict(layers[i]["mixer"])
        m = dict(m, **{side: dict(m[side], **kw)}) if side else dict(m, **kw)
        layers[i]["mixer"] = m
        return dict(cfg, layers=layers)
    z = lambda k: {k.replace(".", "__"): torch.zeros_like(ck[k])}
    assert moved(cfg, **{"l0__mix__left__sink": torch.full((2,), -1e9)}) > 1e-3
    assert moved(mixer(0, "left", rot={"dims": 8, "base": 1e4})) > 1e-3
    assert moved(mixer(1, rot={"dims": 4, "base": 1e4})) > 1e-4
    assert moved(mixer(2, tau=1.0)) > 1e-3
    for k in ("l0.mix.right.x.b", "l0.mix.right.conv.b", "l0.mix.right.y.b", "l0.mix.right.ra.b", "l0.mix.right.ri.b", "l0.mix.left.out",
              "l0.mix.right.out", "l1.mix.g", "l2.mix.a2.b", "l0.mlp.router.b", "l0.norm1.b", "final.norm.b"):
        assert moved(cfg, **z(k)) > 1e-4, k
    assert moved(cfg, **{"l0__hc1__mix": ck["l0.hc1.mix"].T.contiguous()}) > 1e-3
    assert moved(cfg, **{"l0__mix__left__q__conv": ck["l0.mix.left.q.conv"].flip(1)}) > 1e-3
    assert moved(dict(cfg, residual_mult=1.0)) > 1e-3
    assert moved(dict(cfg, loop=dict(cfg["loop"], times=1))) > 1e-3
