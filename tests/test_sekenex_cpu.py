"""CPU checks of the Sekenex path: configuration, tensor shapes, registry, what a slot holds, and the oracle's own consistency
(portions against a whole prompt; its convolution, rotation, recurrences, router, norms and streams against closed forms)."""
import copy
import json
import math

import pytest
import torch

import lia_b200  # noqa: F401
from lia_b200 import registry
from lia_b200.modeling_sekenex import SekenexConfig
from lia_b200.seq_layers import GatedRecurrentMixer, Linear, MoEFeedForward, ParallelMixer, SinkAttentionMixer, StateSpaceMixer
from lia_b200.seq_state import SlotState

import sekenex_oracle as O
from sekenex_cases import CASES, moe, parallel

F32, F64 = torch.float32, torch.float64


def gen(seed):
    return torch.Generator().manual_seed(seed)


def toks_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=gen(seed)).tolist()


@pytest.mark.parametrize("name", sorted(CASES))
def test_configuration_and_shapes(name):
    cfg = CASES[name]
    c = SekenexConfig.from_dict(copy.deepcopy(cfg))
    assert {k: tuple(v) for k, v in c.tensor_shapes().items()} == O.tensor_shapes(cfg)
    back = SekenexConfig.from_dict(copy.deepcopy(c.to_dict()))
    assert back.tensor_shapes() == c.tensor_shapes() and back.layers == c.layers and back.streams == cfg["streams"] and back.norm_eps == cfg["norm"]["eps"]
    for i, l in enumerate(cfg["layers"]):
        assert (f"l{i}.hc2.mix" in c.tensor_shapes()) == (f"l{i}.norm2" in c.tensor_shapes()) == (l["mlp"] is not None)


def test_configuration_fills_what_may_be_left_out():
    c = copy.deepcopy(CASES["even"])
    a = c["layers"][0]["mixer"]["left"]
    a.update(heads=4)
    del a["kv_heads"], a["vdim"], a["rot"], a["conv"]
    del c["layers"][0]["mlp"]["kind"], c["layers"][1]["mlp"]["kind"], c["layers"][2]["mixer"]["groups"], c["layers"][2]["mixer"]["norm_groups"]
    cfg = SekenexConfig.from_dict(c)
    s = cfg.tensor_shapes()
    assert s["l0.mix.left.k"] == (64, 64) and s["l0.mix.left.g"] == (64, 64) and "l0.mix.left.q.conv" not in s
    assert cfg.layers[0]["mlp"]["kind"] == "moe" and cfg.layers[1]["mlp"]["kind"] == "dense" and s["l2.mix.in"] == (2 * 72 + 2 * 16 + 3, 64)


def test_configuration_refuses_what_it_does_not_know():
    def bad(change):
        c = copy.deepcopy(CASES["even"])
        change(c)
        with pytest.raises(ValueError):
            SekenexConfig.from_dict(c)
    bad(lambda c: c["layers"][0].update(type="convolution"))
    bad(lambda c: c["layers"][1]["mlp"].update(kind="sparse"))
    bad(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    bad(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18))
    bad(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=5))
    bad(lambda c: c["layers"][0]["mixer"]["right"].update(blocks=5))
    bad(lambda c: c["layers"][1]["mixer"].update(groups=4))
    bad(lambda c: c["layers"][1]["mixer"].update(norm_groups=5))
    bad(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3))
    bad(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5))
    bad(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))            # more than two groups of two hold
    bad(lambda c: c.update(streams=0))


def test_registry_knows_the_design(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CASES["odd"]))
    assert registry.architecture_of(str(tmp_path)) == "sekenex"
    assert registry.model_class(str(tmp_path)).__name__ == "SekenexForCausalLM"


def test_what_a_slot_holds_and_the_projections_that_share_a_launch():
    w = {k[len("l0.mix."):]: v for k, v in O.random_weights(CASES["even"], 0).items() if k.startswith("l0.mix.")}
    wl, wr = ({k[len(s):]: v for k, v in w.items() if k.startswith(s)} for s in ("left.", "right."))
    left = SinkAttentionMixer(wl, 4, 2, 16, 24, 0.25, 1e-5, F32, "cpu", taps=3, rot={"base": 100.0, "dims": 8}, rot_halves=True, gate="channel", sink=False,
                              ride_along=GatedRecurrentMixer.ride_along(wr))
    right = GatedRecurrentMixer(wr, 48, 3, 4, F32, "cpu", projected=True)
    slots = SlotState(2, 16, "cpu")
    (kc, vc, conv_l), (S, conv_r) = ParallelMixer(left, right, wl["out"], wr["out"], "cpu").new_state(slots)
    assert kc.shape == (2, 16, 32) and vc.shape == (2, 16, 48) and conv_l.shape == (2, 2, 64 + 32 + 48) and S.shape == (2, 48) and conv_r.shape == (2, 3, 48)
    assert left.sink is None and left.proj.sizes == [64, 32, 48, 96, 48, 48] and right.proj is None
    assert torch.allclose(right.c.double(), -8.0 * torch.log1p(torch.exp(wr["lam"].double())), rtol=1e-6)
    m = {k[len("l2.mix."):]: v for k, v in O.random_weights(CASES["even"], 0).items() if k.startswith("l2.mix.")}
    ss = StateSpaceMixer(m, 3, 24, 16, 1, 1, 4, 1e-5, F32, "cpu")
    assert ss.proj.sizes == [72, 104, 3] and ss.proj.N == 184                          # the last columns are padding
    assert torch.equal(ss.proj.weight[ss.proj.offsets[2]:ss.proj.offsets[2] + 3], m["in"][-3:]) and not ss.proj.weight[179:].any()
    S, conv = ss.new_state(slots)
    assert S.shape == (2, 3, 24, 16) and conv.shape == (2, 3, 104)
    assert Linear([torch.zeros(5, 8)], F32, "cpu").N == 5


def test_mixers_and_experts_refuse_sizes_that_do_not_fit():
    ex = [{"up": torch.zeros(4, 8), "down": torch.zeros(8, 4)}] * 6
    for kw in ({"groups": (4, 1)}, {"groups": (3, 4)}, {"groups": (3, 0)}, {"groups": (6, 2)}):
        with pytest.raises(ValueError):
            MoEFeedForward(torch.zeros(6, 8), ex, 3, 4, 6, None, F32, "cpu", **kw)
    assert MoEFeedForward(torch.zeros(6, 8), ex, 3, 4, 6, None, F32, "cpu", groups=(2, 1)).keep == 1
    with pytest.raises(ValueError):
        StateSpaceMixer({}, 4, 8, 16, 3, 1, 4, 1e-5, F32, "cpu")
    with pytest.raises(ValueError):
        GatedRecurrentMixer({}, 10, 4, 4, F32, "cpu")


# ------------------------------------------------------------------------------------------------ the oracle itself
@pytest.mark.parametrize("name", sorted(CASES))
def test_oracle_portions_equal_the_whole_prompt(name):
    cfg = CASES[name]
    w = O.random_weights(cfg, 3)
    toks = toks_for(cfg, 21, 1)
    whole = O.logits_of(cfg, w, toks)
    o = O.Oracle(cfg, w)
    with torch.no_grad():
        parts = torch.cat([o.forward(toks[a:b]) for a, b in ((0, 1), (1, 3), (3, 10), (10, 11), (11, 21))])
    assert float((parts - whole).abs().max()) < 1e-9 * float(whole.abs().max())


def test_oracle_convolution_and_rotation():
    h = torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=F64)
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)                   # two back, one back, current
    assert O.causal_conv(h, 4, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0]
    assert O.causal_conv(h, 2, w, torch.tensor([0.5], dtype=F64))[:, 0].tolist() == [123.5, 234.5]
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    y = O.rotate_halves(x, torch.tensor([7]), 4, 100.0)[0, 0].tolist()
    for i, f in ((0, 1.0), (1, 0.1)):
        u, v = x[0, 0, i].item(), x[0, 0, i + 2].item()
        assert abs(y[i] - (u * math.cos(7 * f) - v * math.sin(7 * f))) < 1e-12 and abs(y[i + 2] - (v * math.cos(7 * f) + u * math.sin(7 * f))) < 1e-12
    assert y[4] == 5.0


def test_oracle_state_space_recurrence_is_a_masked_attention():
    """y_t = sum_(s <= t) (prod_(s < r <= t) exp(-A dt_r)) dt_s (C_t . B_s) x_s + D x_t, head by head."""
    g = gen(1)
    T, H, G, N, vd = 9, 4, 2, 5, 3
    x, B, C = torch.randn(T, H, vd, generator=g, dtype=F64), torch.randn(T, G, N, generator=g, dtype=F64), torch.randn(T, G, N, generator=g, dtype=F64)
    dt, A, D = torch.rand(T, H, generator=g, dtype=F64), torch.rand(H, generator=g, dtype=F64) + 0.1, torch.randn(H, generator=g, dtype=F64)
    y, last = O.ssd(x, B, C, dt, A, D, torch.zeros(H, N, vd, dtype=F64))
    for h in range(H):
        cum = torch.cumsum(-A[h] * dt[:, h], 0)
        L = torch.exp(cum[:, None] - cum[None, :]).tril()
        want = (L * (C[:, h // 2] @ B[:, h // 2].T) * dt[:, h][None, :]) @ x[:, h] + D[h] * x[:, h]
        assert torch.allclose(y[:, h], want)
    y2, last2 = O.ssd(x[5:], B[5:], C[5:], dt[5:], A, D, O.ssd(x[:5], B[:5], C[:5], dt[:5], A, D, torch.zeros(H, N, vd, dtype=F64))[1])
    assert torch.allclose(y2, y[5:]) and torch.allclose(last2, last)


def test_oracle_gated_recurrent_unit():
    w = {"ra": torch.tensor([[[2.0]], [[0.0]]], dtype=F64), "ra.b": torch.tensor([[0.5], [1.0]], dtype=F64), "ri": torch.tensor([[[0.0]], [[-1.0]]], dtype=F64),
         "ri.b": torch.tensor([[0.3], [0.0]], dtype=F64), "lam": torch.tensor([-2.0, -4.0], dtype=F64)}
    u = torch.tensor([[0.7, -0.4], [0.1, 2.0]], dtype=F64)
    out, last = O.rglru(u, w, "", 2, torch.zeros(2, dtype=F64))
    sig, s = lambda z: 1 / (1 + math.exp(-z)), [0.0, 0.0]  # noqa: E731
    for t in range(2):
        for c, (r, i) in enumerate(((sig(2.0 * u[t, 0].item() + 0.5), sig(0.3)), (sig(1.0), sig(-u[t, 1].item())))):
            a = math.exp(-8.0 * r * math.log1p(math.exp([-2.0, -4.0][c])))
            s[c] = a * s[c] + math.sqrt(1 - a * a) * i * u[t, c].item()
            assert abs(out[t, c].item() - s[c]) < 1e-12
    assert last.tolist() == out[1].tolist()


def test_oracle_router_norm_and_streams():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}
    z = torch.tensor([[1.0, 0.9, 3.0, -5.0, 2.0, 0.0], [0.0, 0.1, 0.2, 0.3, 0.4, 5.0]], dtype=F64)
    idx, wt = O.route(z, torch.eye(6, dtype=F64), r)
    assert idx.tolist() == [[2, 4], [5, 4]]
    assert torch.allclose(wt, torch.softmax(z, -1).gather(1, idx)) and float(wt.sum(-1).max()) < 1.0
    # groups of two with one kept: the second largest score (1.9) lies outside the best group
    idx, _ = O.route(torch.tensor([[2.0, -1.0, 1.9, 1.8]], dtype=F64), torch.eye(4, dtype=F64), {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert idx.tolist() == [[0, 1]]
    y, zg = torch.tensor([[1.0, 2.0, 30.0, 40.0]], dtype=F64), torch.ones(1, 4, dtype=F64)
    n = O.gated_group_norm(y, zg, torch.ones(4, dtype=F64), 2, 0.0)
    assert torch.allclose(n[0, :2], y[0, :2] / math.sqrt(2.5)) and torch.allclose(n[0, 2:], y[0, 2:] / math.sqrt(1250.0))
    a, b = torch.tensor([[1.0]], dtype=F64), torch.tensor([[10.0]], dtype=F64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)            # [from, to]
    new = O.hyper_write([a, b], torch.tensor([[100.0]], dtype=F64), mix, torch.tensor([1.0, -1.0], dtype=F64))
    assert new[0].item() == 1.0 + 30.0 + 100.0 and new[1].item() == 2.0 + 40.0 - 100.0
    assert O.hyper_read([a, b], torch.tensor([2.0, 0.5], dtype=F64)).item() == 7.0
    assert O.relu_squared(torch.tensor([-3.0, 2.0])).tolist() == [0.0, 4.0]


def test_the_cases_cover_every_branch():
    layers = [l for c in CASES.values() for l in c["layers"]]
    assert {l["type"] for l in layers} == {"parallel", "mamba2"} and any(l["mlp"] is None for l in layers)
    lefts = [l["mixer"]["left"] for l in layers if l["type"] == "parallel"]
    assert any("rot" not in a for a in lefts) and any("conv" not in a for a in lefts) and any(a["rot"]["dims"] == a["dim"] for a in lefts if "rot" in a)
    assert parallel(lefts[0], 4, 1)["mlp"] is None and "groups" not in moe(2, 1, 3)["router"]
    kinds = [l["mlp"] for l in layers if l["mlp"]]
    assert {m["kind"] for m in kinds} == {"dense", "moe"} and any("shared" not in m for m in kinds if m["kind"] == "moe")
