"""Relidra without a GPU: configuration, registry, cache bookkeeping, the oracle's own consistency."""
import copy
import math

import pytest
import torch

import relidra_cases as rc
from conftest import load
from oracle import relidra as orl


def test_config_is_read_from_the_file_alone():
    R = load("relidra")
    c = R.RelidraConfig.parse(rc.CONFIGS["odd"])
    assert (c.width, c.vocab, c.eps, c.streams) == (84, 101, 1e-5, 3)
    assert c.runs == (0, 1, 2, 1, 2, 3)
    assert c.layers[0] == (R.Delta(6, 2, 20, 12, 3), 150)
    assert c.layers[1] == (R.Attention(4, 2, 36, 20, 700.0, 2.5, 0.4, 23), None)
    assert c.layers[3][1] == 36
    assert R.RelidraConfig.parse(rc.CONFIGS["wide"]).runs == (0, 1)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="convolution"), "mixer type"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=35), "values are the keys"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=38), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="tree"), "feed-forward"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c.update(streams=0), "streams"),
])
def test_config_errors_are_named(change, message):
    cfg = copy.deepcopy(rc.CONFIGS["odd"])
    change(cfg)
    with pytest.raises(ValueError, match=message):
        load("relidra").RelidraConfig.parse(cfg)


def test_registry_knows_the_design():
    reg = load("registry")
    assert reg.design_of(rc.CONFIGS["odd"]).name == "Relidra"
    with pytest.raises(ValueError, match="adapters"):
        reg.build_model(rc.CONFIGS["odd"], {}, adapters=[{}], scales=[1.0])
    with pytest.raises(reg.UnsupportedPrecision):
        reg.build_model(rc.CONFIGS["odd"], {}, dtype=torch.float16)


def test_oracle_equations_on_hand_made_values():
    d = lambda *v: torch.tensor(v, dtype=torch.float64)
    x = d([1.0, 3.0])
    torch.testing.assert_close(orl.layer_norm(x, d(2.0, 5.0), 3.0), d([-1.0, 2.5]))        # mean 2, variance 1
    torch.testing.assert_close(orl.unit(d([3.0, 4.0])), d([0.6, 0.8]), atol=1e-6, rtol=0)
    torch.testing.assert_close(orl.short_conv(d([1.0], [2.0], [4.0]), d([10.0, 1.0])), d([1.0], [12.0], [24.0]))
    # two streams: stream 0 hands half of itself to stream 1; the sublayer sees 2 x_0 + x_1 and gives back its square
    got = orl.hyper_connect(d([[1.0]], [[10.0]]), d(2.0, 1.0), d([1.0, 0.5], [0.0, 3.0]), d(1.0, -1.0), lambda u: u * u)
    torch.testing.assert_close(got, d([[1.0 + 144.0]], [[0.5 + 30.0 - 144.0]]))
    # a delta rule of one row and column: M = 1 from the first token; the second halves it, then moves it by half the way
    # from k M = 1 to 7 along k = 2
    y, M = orl.delta_rule(d([1.0], [3.0]), d([1.0], [2.0]), d([1.0], [7.0]), d(1.0, 0.5), d(1.0, 0.5))
    assert M.item() == 0.5 + 2.0 * 0.5 * (7.0 - 1.0) and y.flatten().tolist() == [1.0, 3 * M.item()]
    torch.testing.assert_close(orl.delta_decay(d(0.3), d(math.log(2.0)), d(0.2)),
                               torch.exp(-2 * torch.log(1 + torch.exp(d(0.5)))))
    # rotation: column 0 with column 1, a quarter turn at position 1 (frequency pi / 2 by the divisor), column 2 untouched
    z = d([[[1.0, 0.0, 5.0]], [[1.0, 0.0, 5.0]]])
    torch.testing.assert_close(orl.rotate(z, torch.tensor([0, 1]), 2, 10.0, 2 / math.pi), d([[[1.0, 0.0, 5.0]], [[0.0, 1.0, 5.0]]]))
    assert orl.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    torch.testing.assert_close(orl.sink_softmax(d([[0.0, math.log(2.0)]]), d(math.log(5.0))), d([[1 / 8, 2 / 8]]))


def test_cases_make_small_mistakes_visible(monkeypatch):
    """The configurations the GPU tests use react to the smallest mistakes of a mask, a sink, a state or a connection by more
    than those tests allow."""
    def shown(name, attr, wrong):
        cfg = rc.CONFIGS[name]
        p, toks = rc.weights(cfg), rc.tokens(cfg, 60)
        want = orl.OracleRelidra(cfg, p).forward(toks)[0]
        with monkeypatch.context() as m:
            m.setattr(orl, attr, wrong(getattr(orl, attr)))
            return float(rc.error(orl.OracleRelidra(cfg, p).forward(toks)[0], want).max())

    for name in ("odd", "deep", "streams"):
        assert shown(name, "chunk_mask", lambda f: lambda n, size: f(n, size + 1)) > 0.2
        assert shown(name, "chunk_mask", lambda f: lambda n, size: f(n, size - 1)) > 0.2
        assert shown(name, "chunk_mask", lambda f: lambda n, size: f(n, None)) > 0.2
        assert shown(name, "sink_softmax", lambda f: lambda s, sink: f(s, sink - 100)) > 0.2
        assert shown(name, "rotate", lambda f: lambda x, pos, *a: f(x, pos * 1.3, *a)) > 0.06
        assert shown(name, "short_conv", lambda f: lambda x, w: torch.cat([f(x[:30], w), f(x[30:], w)])) > 0.2  # inputs lost
        assert shown(name, "hyper_connect", lambda f: lambda s, i, mix, o, sub: f(s, i, mix.T, o, sub)) > 0.06
        assert shown(name, "delta_rule", lambda f: lambda q, k, v, g, b: (torch.cat(
            [f(q[:30], k[:30], v[:30], g[:30], b[:30])[0], f(q[30:], k[30:], v[30:], g[30:], b[30:])[0]]), None)) > 0.2


def test_states_of_a_slot_can_be_put_back():
    """What a captured step's warm-up run changes: states by slot, not those of other sequences."""
    kv = load("kv_cache").HybridCache.__new__(load("kv_cache").HybridCache)
    kv.device, kv._slot_of = torch.device("cpu"), {7: 2, 9: 0}
    kv.states = {1: {"S": torch.arange(8.0).view(4, 2)}}
    undo = kv.snapshot([7])
    kv.states[1]["S"] += 100
    undo()
    assert kv.states[1]["S"].tolist() == [[100, 101], [102, 103], [4, 5], [106, 107]]
