"""Tevudra without a GPU: configuration, registry, the oracle's own consistency."""
import copy

import pytest
import torch

import tevudra_cases as tc
from conftest import load
from oracle import tevudra as ot


def test_config_is_read_from_the_file_alone():
    T = load("tevudra")
    c = T.TevudraConfig.parse(tc.CONFIGS["odd"])
    assert (c.width, c.vocab, c.eps, len(c.layers)) == (84, 101, 1e-5, 4)
    mixes = [m for m, _ in c.layers]
    assert [m.source for m in mixes] == [0, 1, 0, 1]
    assert mixes[1].scale == 0.4 and mixes[3].vdim == 40 and mixes[2].dim == 33
    ffs = [f for _, f in c.layers]
    assert ffs[0] == T.MoE(36, 7, 3, 52) and ffs[1] is None and ffs[2] == T.Dense(150) and ffs[3].shared_ff == 0


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="convolution"), "mixer type"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=45), "kv_rank"),
    (lambda c: c["layers"][2]["mlp"].update(kind="tree"), "feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"),
])
def test_config_errors_are_named(change, message):
    cfg = copy.deepcopy(tc.CONFIGS["odd"])
    change(cfg)
    with pytest.raises(ValueError, match=message):
        load("tevudra").TevudraConfig.parse(cfg)


def test_registry_names_designs_and_precisions():
    reg = load("registry")
    assert reg.design_of(tc.CONFIGS["odd"]).name == "Tevudra"
    assert reg.design_of({"architectures": ["LlamaForCausalLM"]}).name == "LlamaForCausalLM"
    assert reg.design_of({"hidden_size": 8}).name == "LlamaForCausalLM"
    with pytest.raises(ValueError, match="unknown model design"):
        reg.design_of({"architecture": "Nothing"})
    with pytest.raises(reg.UnsupportedPrecision):
        reg.build_model({"hidden_size": 8}, {}, dtype=torch.float32)
    with pytest.raises(ValueError, match="adapters"):
        reg.build_model(tc.CONFIGS["odd"], {}, adapters=[{}], scales=[1.0])


def test_oracle_equations_on_hand_made_values():
    x = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    torch.testing.assert_close(ot.dyt(x, 0.5, torch.tensor([2.0, 1.0]), torch.tensor([0.1, 0.0])),
                               torch.tensor([[2 * 0.46211715726 + 0.1, -0.76159415596]], dtype=torch.float64))
    torch.testing.assert_close(ot.rms(x, torch.tensor([1.0, 2.0]), 1.5), x / 2 * torch.tensor([1.0, 2.0]))
    torch.testing.assert_close(ot.relu2(x), torch.tensor([[1.0, 0.0]], dtype=torch.float64))
    idx, w = ot.route(x, torch.tensor([[1.0, 0], [0, 1.0], [0.5, 0]], dtype=torch.float64), torch.tensor([0.0, 5.0, 0.25]), 2)
    assert idx.tolist() == [[1, 0]]  # logits 1, 3, 0.75
    torch.testing.assert_close(w, torch.softmax(torch.tensor([[3.0, 1.0]], dtype=torch.float64), -1))


def test_cases_make_a_misplaced_key_visible():
    """The configurations the GPU tests use react to the smallest mistakes of an attention mask or a cache."""
    for name, cfg in tc.CONFIGS.items():
        p, toks = tc.weights(cfg), tc.tokens(cfg, 40)
        want = ot.OracleTevudra(cfg, p).forward(toks)[0]

        def planted(mistake):
            o = ot.OracleTevudra(cfg, p)
            true = ot.latent_attention
            try:
                ot.latent_attention = lambda h, c, *a: true(h, mistake(c), *a)
                return tc.error(o.forward(toks)[0], want)
            finally:
                ot.latent_attention = true

        shifted = planted(lambda c: torch.cat([c[:1], c[:-1]]))                       # every key one place late
        lost_first = planted(lambda c: torch.cat([torch.zeros_like(c[:1]), c[1:]]))   # the first key's row lost
        lost_mid = planted(lambda c: torch.cat([c[:16], torch.zeros_like(c[16:17]), c[17:]]))  # ... a page's first
        assert shifted[2:].median() > 0.1, name
        assert lost_first.max() > 0.1 and lost_mid[16:].max() > 0.1, name
