"""CPU checks of the Pazivik path: configuration, tensor shapes, registry, which layer's state a layer reads, and the oracle's own
consistency (portions against a whole prompt, its window mask, sink, bigram rows, position waves, router and weighed inputs)."""
import copy
import json
import math

import pytest
import torch

import lia_b200  # noqa: F401
from lia_b200 import registry
from lia_b200.modeling_pazivik import PazivikConfig
from lia_b200.seq_layers import LatentAttentionMixer, MoEFeedForward
from lia_b200.seq_state import SlotState

import pazivik_oracle as O
from pazivik_cases import CASES, config, dense, latent, moe

F32, F64 = torch.float32, torch.float64


def toks_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.mark.parametrize("name", sorted(CASES))
def test_configuration_and_shapes(name):
    cfg = CASES[name]
    c = PazivikConfig.from_dict(copy.deepcopy(cfg))
    assert {k: tuple(v) for k, v in c.tensor_shapes().items()} == O.tensor_shapes(cfg)
    back = PazivikConfig.from_dict(copy.deepcopy(c.to_dict()))
    assert back.tensor_shapes() == c.tensor_shapes() and back.layers == c.layers and back.bigram == c.bigram
    assert back.norm_eps == cfg["norm"]["eps"] and back.logit_softcap == cfg.get("logit_softcap", 0.0)
    names = set(c.tensor_shapes())
    assert ("bigram" in names) == ("embedding" in cfg) and "head" not in names
    for i, l in enumerate(cfg["layers"]):
        assert (f"l{i}.mix.dkv" in names) == ("kv_from" not in l["mixer"]) and (f"l{i}.norm2" in names) == (l["mlp"] is not None)


def test_configuration_refuses_what_it_does_not_know():
    def bad(change):
        c = copy.deepcopy(CASES["even"])
        change(c["layers"])
        with pytest.raises(ValueError):
            PazivikConfig.from_dict(c)
    bad(lambda ls: ls[0].update(type="convolution"))
    bad(lambda ls: ls[0]["mlp"].update(kind="sparse"))
    bad(lambda ls: ls[1]["mixer"].update(kv_from=1))               # itself
    bad(lambda ls: ls[1]["mixer"].update(kv_from=3))               # a later layer
    bad(lambda ls: ls[4]["mixer"].update(kv_from=1))               # a layer that has no latents of its own
    bad(lambda ls: ls[1]["mixer"].update(kv_rank=24))              # latents of another size


def test_registry_knows_the_design(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CASES["odd"]))
    assert registry.architecture_of(str(tmp_path)) == "pazivik"
    assert registry.model_class(str(tmp_path)).__name__ == "PazivikForCausalLM"


def _mixer_weights(H, d, v, r, W, own):
    w = {"q": torch.zeros(H * d, W), "uk": torch.zeros(H * d, r), "uv": torch.zeros(H * v, r), "sink": torch.zeros(H), "o": torch.zeros(W, H * v)}
    if own:
        w.update({"dkv": torch.zeros(r, W), "dkv.norm": torch.ones(r)})
    return w


def test_a_layer_without_latents_of_its_own_shares_the_source_layers_rows():
    slots = SlotState(2, 16, "cpu")
    own = LatentAttentionMixer(_mixer_weights(2, 4, 4, 8, 16, True), 2, 4, 0, 4, 8, 0, None, 0.5, 1e-5, F32, "cpu", gate=None, window=5, sink=True)
    reader = LatentAttentionMixer(_mixer_weights(3, 6, 2, 8, 16, False), 3, 6, 0, 2, 8, 0, None, 0.5, 1e-5, F32, "cpu", gate=None, window=9, sink=True,
                                  own_latent=False)
    state = own.new_state(slots)
    assert state[0].shape == (2, 16, 8) and reader.new_state(slots, state)[0] is state[0] and len(slots.rows) == 1
    with pytest.raises(ValueError):
        reader.new_state(slots)
    with pytest.raises(ValueError):
        reader.new_state(slots, (slots.add_rows(7, F32),))
    with pytest.raises(ValueError):
        LatentAttentionMixer(_mixer_weights(2, 4, 4, 8, 16, False), 2, 4, 2, 4, 8, 2, 100.0, 0.5, 1e-5, F32, "cpu", gate=None, own_latent=False)


def test_experts_refuse_options_they_do_not_know():
    ex = [{"gate": torch.zeros(4, 8), "up": torch.zeros(4, 8), "down": torch.zeros(8, 4)}]
    for kw in ({"score": "relu"}, {"weigh": "both"}, {"shared_gate": torch.zeros(1, 8)}):
        with pytest.raises(ValueError):
            MoEFeedForward(torch.zeros(1, 8), ex, 1, 4, 2, None, F32, "cpu", **kw)


@pytest.mark.parametrize("name", sorted(CASES))
def test_oracle_portions_equal_the_whole_prompt(name):
    cfg = CASES[name]
    w = O.random_weights(cfg, 3)
    toks = toks_for(cfg, 31, 1)
    whole = O.logits_of(cfg, w, toks)
    o = O.Oracle(cfg, w)
    with torch.no_grad():
        parts = torch.cat([o.forward(toks[a:b]) for a, b in ((0, 7), (7, 8), (8, 10), (10, 27), (27, 31))])
    assert float((parts - whole).abs().max()) < 1e-9
    if cfg.get("logit_softcap"):
        assert float(whole.abs().max()) <= cfg["logit_softcap"]


def test_oracle_window_sink_bigram_and_positions():
    assert O.window_mask(3, 2, 2).tolist() == [[False, False, True, True, False], [False, False, False, True, True]]
    assert O.window_mask(1, 2, 0).tolist() == [[True, True, False], [True, True, True]]
    assert O.window_mask(0, 3, 1).tolist() == torch.eye(3, dtype=torch.bool).tolist()
    s = torch.tensor([[0.3, -1.0, 2.0]], dtype=F64)
    wt = O.sink_softmax(s, torch.tensor([[True, False, True]]), 0.7)
    den = math.exp(0.3) + math.exp(2.0) + math.exp(0.7)
    assert torch.allclose(wt, torch.tensor([[math.exp(0.3) / den, 0.0, math.exp(2.0) / den]], dtype=F64))
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert O.bigram_rows([7, 2, 9], None, b) == [10, (21 + 8) % 10, (6 + 36) % 10] and O.bigram_rows([2], 7, b) == [(21 + 8) % 10]
    pe = O.sinusoid([0, 5], 5)
    assert pe[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0]
    f = [10000.0 ** (-2.0 * i / 5) for i in range(3)]
    assert torch.allclose(pe[1], torch.tensor([math.sin(5 * f[0]), math.cos(5 * f[0]), math.sin(5 * f[1]), math.cos(5 * f[1]), math.sin(5 * f[2])], dtype=F64))


def test_oracle_experts_are_weighed_on_the_way_in():
    g = torch.Generator().manual_seed(0)
    cfg, W = moe(4, 2, 6, shared=3), 8
    w = {k: torch.randn(s, generator=g, dtype=F64) for k, s in O.tensor_shapes(config([latent(1, 2, 2, 4, 3, mlp=cfg)], 10, W)).items()}
    p = "l0.mlp."
    h = torch.randn(5, W, generator=g, dtype=F64)
    idx, wt = O.route(h, w[p + "router"], 2)
    z = h @ w[p + "router"].T
    assert torch.equal(idx[:, 0], z.argmax(-1)) and torch.allclose(wt, torch.sigmoid(z.gather(1, idx)))          # not renormalised
    got = O.moe(h, w, p, cfg)
    shared = torch.sigmoid(h @ w[p + "shared.sg"].T) * O.gated(h, w, p + "shared.", O.silu)
    inp = torch.stack([sum(O.gated(wt[t, j] * h[t], w, p + f"e{int(idx[t, j])}.", O.silu) for j in range(2)) for t in range(5)])
    out = torch.stack([sum(wt[t, j] * O.gated(h[t], w, p + f"e{int(idx[t, j])}.", O.silu) for j in range(2)) for t in range(5)])
    assert torch.allclose(got, inp + shared) and float((inp - out).abs().max()) > 0.1            # the two places of the weight differ
