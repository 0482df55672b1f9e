"""Host-side parts of the Ranesun path that need no GPU: config parsing, the registry, the run order of the looped block,
the rotary table, and the oracle's own consistency (causality, what a sink, a cap, a temperature and a table do)."""
import math

import pytest
import torch

import ranesun_oracle as O
from pg_b200 import registry
from pg_b200.ragged_engine import RotaryCfg, layer_runs, loop_cfg
from pg_b200.ranesun import RanesunConfig, rotary_pairs

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    cfg = O.make_config(width=40, vocab=77, eps=3e-4, logit_scale=2.5, loop=(1, 3, 4), layers=[
        O.layer(O.attention(heads=6, kv_heads=3, dim=10, softcap=7.5, coef=0.3, every=11, scale=0.2), O.dense(24)),
        O.layer(O.retention(heads=3, dim=8, vdim=14, decay=[0.5, 0.75, 0.9], rot_dims=6, base=77.0), O.moe(7, 3, 12)),
        O.layer(O.attention(heads=2, kv_heads=2, dim=4))])
    c = RanesunConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.eps, c.logit_scale) == (77, 40, 3e-4, 2.5)
    a = c.layers[0].mixer
    assert (c.layers[0].kind, a.heads, a.kv_heads, a.dim, a.scale, a.softcap, a.temp_coef, a.temp_every) == \
        ("attention", 6, 3, 10, 0.2, 7.5, 0.3, 11)
    r = c.layers[1].mixer
    assert (c.layers[1].kind, r.heads, r.dim, r.vdim, r.decay, r.rot.dims, r.rot.base) == \
        ("retention", 3, 8, 14, [0.5, 0.75, 0.9], 6, 77.0)
    m = c.layers[1].mlp
    assert (m.kind, m.experts, m.top, m.ff) == ("moe", 7, 3, 12)
    assert (c.layers[0].mlp.kind, c.layers[0].mlp.ff, c.layers[2].mlp) == ("dense", 24, None)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 4)
    assert registry.resolve(cfg).__name__ == "RanesunEngine" and "Ranesun" in registry.architectures()


def test_optional_entries():
    at = O.attention(heads=2, kv_heads=1, dim=4)
    del at["mixer"]["q_temp"], at["mixer"]["softcap"]
    re = O.retention(heads=1, dim=4, vdim=4)
    re["mixer"]["rot"] = None
    c = RanesunConfig.from_dict(dict(O.make_config(width=8, vocab=9, layers=[O.layer(at), O.layer(re)]), loop=None))
    assert (c.layers[0].mixer.softcap, c.layers[0].mixer.temp_every, c.layers[1].mixer.rot, c.loop) == (0.0, 0, None, None)


def test_config_rejects_what_the_design_does_not_have():
    def bad(layers, **kw):
        with pytest.raises(ValueError):
            RanesunConfig.from_dict(O.make_config(width=16, vocab=20, layers=layers, **kw))
    ok = O.layer(O.attention(heads=2, kv_heads=1, dim=4))
    bad([O.layer(O.attention(heads=3, kv_heads=2, dim=4))])
    bad([O.layer(O.retention(heads=3, dim=4, vdim=4, decay=[0.5]))])
    bad([O.layer(O.retention(heads=1, dim=4, vdim=4, rot_dims=6))])
    bad([O.layer(O.retention(heads=1, dim=4, vdim=4, rot_dims=3))])
    bad([dict(ok, type="convolution")])
    bad([dict(ok, mlp={"kind": "router"})])
    bad([dict(ok, mlp=O.moe(2, 3, 4))])
    bad([ok], loop=(0, 2, 2))
    bad([ok], loop=(0, 1, 0))
    apart = O.attention(heads=2, kv_heads=1, dim=4)
    apart["mixer"]["vdim"] = 6                                  # the values are the keys
    bad([O.layer(apart)])
    broken = O.attention(heads=2, kv_heads=1, dim=4)
    broken["mixer"]["q_temp"]["every"] = 2.5
    bad([O.layer(broken)])


def test_run_order_of_a_looped_block():
    def order(n, loop):
        return [(r.layer, r.loop_pass) for r in layer_runs(n, loop_cfg(loop, n))]
    assert order(3, None) == [(0, None), (1, None), (2, None)]
    assert order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert order(2, {"start": 0, "stop": 2, "times": 3}) == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None)]
    for n, loop in ((5, (2, 3, 3)), (4, (0, 1, 1)), (3, (2, 3, 2))):
        cfg = {"layers": [0] * n, "loop": dict(zip(("start", "stop", "times"), loop))}
        assert order(n, cfg["loop"]) == O.run_order(cfg)


def test_rotary_pairs_keep_what_one_float_loses():
    for dims, base in ((8, 10000.0), (64, 250000.0), (2, 5.0)):
        want = O.frequencies(dims, base)
        pairs = rotary_pairs(RotaryCfg(dims, base))
        assert pairs.shape == (dims // 2, 2) and pairs.dtype == torch.float32
        assert torch.allclose(pairs.to(F64).sum(-1), want, rtol=1e-13, atol=0)


def test_oracle_temperature_steps():
    assert O.query_temperature(0, 0.5, 4) == 1.0 and O.query_temperature(2, 0.5, 4) == 1.0
    assert O.query_temperature(3, 0.5, 4) == 1.0 + 0.5 * math.log(2.0)      # position 3 is the fourth token
    assert O.query_temperature(6, 0.5, 4) == 1.0 + 0.5 * math.log(2.0)
    assert O.query_temperature(7, 0.5, 4) == 1.0 + 0.5 * math.log(3.0)
    assert O.query_temperature(0, 0.7, 1) == 1.0 + 0.7 * math.log(2.0)


def test_oracle_tied_attention_by_hand():
    """Two keys, one query: the sink takes its share once, without the cap and the scale."""
    k = torch.tensor([[1.0, 2.0], [3.0, -1.0]], dtype=F64)
    q = torch.tensor([[0.5, 0.5]], dtype=F64)
    got = O.tied_attention(q, k, 2.0, 4.0, (0.3, 1), torch.tensor(0.7), first=1)[0]
    t = 1.0 + 0.3 * math.log(3.0)
    s = [4.0 * math.tanh(2.0 * t * z / 4.0) for z in (1.5, 1.0)]
    e = [math.exp(z) for z in s]
    den = sum(e) + math.exp(0.7)
    assert torch.allclose(got, (e[0] * k[0] + e[1] * k[1]) / den, atol=1e-14)


def test_oracle_retention_is_the_decayed_sum_over_all_earlier_tokens():
    g = torch.Generator().manual_seed(0)
    n, H, d, e = 9, 2, 4, 3
    q, k, v = (torch.randn(n, H, x, generator=g, dtype=F64) for x in (d, d, e))
    dec = [0.9, 0.5]
    want = torch.zeros(n, H, e, dtype=F64)
    for h in range(H):
        for i in range(n):
            for j in range(i + 1):
                want[i, h] += dec[h] ** (i - j) * float(q[i, h] @ k[j, h]) * v[j, h]
    assert torch.allclose(O.retention_scan(q, k, v, dec), want, atol=1e-12)
    # rotated q and k: their product depends on the distance alone
    f = O.frequencies(d, 50.0)
    a, b = q[:1, 0], k[:1, 0]
    one = float((O.rotate(a, [7], f) * O.rotate(b, [4], f)).sum())
    assert abs(one - float((O.rotate(a, [103], f) * O.rotate(b, [100], f)).sum())) < 1e-12


def test_oracle_is_causal_and_every_mechanism_shows():
    """Later tokens change nothing earlier; leaving out the sink, the cap, the temperature, a pass's embedding sum, its step
    vector, a bias, or taking the neighbour's expert moves the logits (so that a test against the oracle would see it)."""
    cfg = O.make_config(width=24, vocab=30, loop=(0, 2, 2), layers=[
        O.layer(O.attention(heads=2, kv_heads=1, dim=8, softcap=3.0, every=4), O.moe(4, 2, 8)),
        O.layer(O.retention(heads=2, dim=6, vdim=4, rot_dims=4), O.dense(12))])
    ck = O.make_checkpoint(cfg, 2)
    toks = torch.randint(0, 30, (14,), generator=torch.Generator().manual_seed(3)).tolist()
    full = O.forward(cfg, ck, toks)
    assert torch.allclose(O.forward(cfg, ck, toks[:9]), full[:9], atol=1e-10)

    def moved(cfg2, ck2):
        return float((O.forward(cfg2, ck2, toks) - full)[5:].abs().amax(-1).min())

    def mixer(**kw):
        first = dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], **kw))
        return dict(cfg, layers=[first, cfg["layers"][1]])
    assert moved(cfg, dict(ck, **{"l0.mix.sink": torch.full((2,), -1e9)})) > 1e-3
    assert moved(mixer(softcap=None), ck) > 1e-3
    assert moved(mixer(q_temp=None), ck) > 1e-3
    assert moved(cfg, dict(ck, **{"loop.step": ck["loop.step"] * torch.tensor([[1.0], [0.0]])})) > 1e-3
    assert moved(cfg, dict(ck, **{"l0.norm1.b": torch.zeros(24)})) > 1e-3
    assert moved(cfg, dict(ck, **{"l0.mlp.table": (ck["l0.mlp.table"] + 1) % 4})) > 1e-3
    assert moved(dict(cfg, loop=dict(cfg["loop"], times=1)), dict(ck, **{"loop.step": ck["loop.step"][:1]})) > 1e-3
