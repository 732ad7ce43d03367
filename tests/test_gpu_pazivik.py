"""GPU checks of the Pazivik path against the plain float64 oracle (tests/pazivik_oracle.py): every new kernel and the mixer alone,
then the model through the step engine -- whole prompts, token-by-token decoding, portions down to two tokens, unequal requests
in one step, slots that are freed and reused, a key far back among hundreds, keys just inside and just outside a window (in
prompts and in decoding), keys at the edges of the attention kernel's own tiles (32 cached positions per stage, 64 per key
range), the first tokens and their bigrams, long decoding, sizes that are equal or 1, greedy generation through generate(), the
trace runner and the command line."""
import copy
import json
import os

import pytest
import torch

import lia_b200  # noqa: F401
from lia_b200 import ops, registry
from lia_b200.checkpoint import write_safetensors
from lia_b200.engine import Engine
from lia_b200.modeling_pazivik import PazivikConfig, PazivikForCausalLM
from lia_b200.seq_layers import GatedMLP, LatentAttentionMixer, MoEFeedForward, StepBatch
from lia_b200.seq_state import SlotState

import pazivik_oracle as O
from pazivik_cases import CASES, config, dense, latent, moe

pytestmark = pytest.mark.gpu
BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
DEV = "cuda"


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(a, b):
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def bf(t):
    """bf16-representable fp32 numbers."""
    return t.to(BF16).float()


def make_batch(portions):
    """portions: (slot, first position, tokens) in row order."""
    segs, meta, row = [], [], 0
    for slot, p0, n in portions:
        segs.append((slot, p0, row, n))
        meta += [(slot, p0 + i) for i in range(n)]
        row += n
    return StepBatch(row, i32(segs), i32(meta), max(p0 + n for _, p0, n in portions), portions=segs)


CUTS = {"whole": [60], "token by token": [1] * 60, "twos": [2] * 30, "ragged": [31, 1, 1, 2, 22, 3], "stage edges": [32, 1, 27]}


# ------------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("W", [45, 256, 1000])
def test_embedding_with_bigram_and_waves(W):
    """Two sequences side by side: one from its first token, one that goes on at position 4000, so that its first bigram needs the
    id that an earlier step left; then the next token of the first one."""
    g = gen(0)
    table, big = bf(torch.randn(50, W, generator=g)), bf(torch.randn(24, W, generator=g))
    nw = 1.0 + 0.3 * torch.randn(W, generator=g)
    b = {"buckets": 23, "mul_prev": 1000003, "mul_cur": 17}
    freq = torch.tensor([10000.0 ** (-2.0 * i / W) for i in range((W + 1) // 2)], dtype=F64).to(DEV)
    first, second = [3, 49, 0, 3], [17, 20, 49]
    rows = O.bigram_rows(first[:3], None, b) + O.bigram_rows(second, 31, b) + O.bigram_rows(first[3:], first[2], b)
    pos = [0, 1, 2, 4000, 4001, 4002, 3]
    ids = first[:3] + second + first[3:]
    want = table[ids].double() + big[rows].double() + O.sinusoid(pos, W)
    for dt, tol in ((F32, 2e-6), (BF16, 5e-3)):
        tokens = torch.full((3, 4100, 1), 7, dtype=torch.int32, device=DEV)
        tokens[1, 3999] = 31
        outs = []
        for at, portions in ((0, [(2, 0, 3), (1, 4000, 3)]), (6, [(2, 3, 1)])):
            batch = make_batch(portions)
            x = torch.empty(batch.rows, W, device=DEV)
            h = torch.empty(batch.rows, W, dtype=dt, device=DEV)
            ops.embed_bigram_pos(torch.tensor(ids[at:at + batch.rows], device=DEV), table.to(DEV, dt), batch.meta, x, bigram=big.to(DEV, dt),
                                 hashing=(23, 1000003, 17), tokens=tokens, freq=freq, norm_w=nw.to(DEV), h=h, eps=1e-5)
            outs.append((x, h))
        x, h = (torch.cat([o[i] for o in outs]) for i in range(2))
        assert rel(x, want) < 1e-6                                    # the stream is fp32 whatever the tables are
        assert rel(h, O.rms_norm(want, nw.double(), 1e-5)) < tol
        assert tokens[2, :4, 0].tolist() == first and tokens[1, 3999:4003, 0].tolist() == [31] + second and bool((tokens[0] == 7).all())
    x2 = torch.empty(3, W, device=DEV)                                # without a bigram table, without waves, without a norm
    ops.embed_bigram_pos(torch.tensor(first[:3], device=DEV), table.to(DEV), make_batch([(0, 0, 3)]).meta, x2)
    assert torch.equal(x2.cpu(), table[first[:3]])


@pytest.mark.parametrize("rank,at", [(17, 5), (40, 5), (40, 8), (264, 8), (512, 16), (1024, 0), (1032, 8)])
def test_latent_store(rank, at):
    """Column slices that allow 128-bit accesses and slices that do not, rows that fit a warp's registers and longer ones."""
    g = gen(1)
    y, w = torch.randn(70, rank + 24, generator=g) * 3.0, 1.0 + 0.3 * torch.randn(rank, generator=g)
    for dt, tol in ((F32, 2e-6), (BF16, 5e-3)):
        yy = y.to(dt)
        cache = torch.zeros(3, 80, rank, dtype=dt, device=DEV)
        ops.latent_store(yy.to(DEV)[:, at:at + rank], w.to(DEV), make_batch([(2, 10, 69), (0, 79, 1)]).meta, cache, rank, 1e-6)
        want = O.rms_norm(yy.double()[:, at:at + rank], w.double(), 1e-6)
        assert rel(cache[2, 10:79], want[:69]) < tol and rel(cache[0, 79], want[69]) < tol
        assert not cache[1].any() and not cache[2, :10].any() and not cache[2, 79].any() and not cache[0, :79].any()


def _latent_reference(q, c, pos0, H, rank, scale, window, sink):
    T = q.shape[0]
    mask = O.window_mask(pos0, T, window)[:, :c.shape[0]]
    out = torch.zeros(T, H, rank, dtype=F64)
    for a in range(H):
        out[:, a] = O.sink_softmax(q.view(T, H, rank)[:, a].double() @ c.double().T * scale, mask, -1e9 if sink is None else sink[a]) @ c.double()
    return out.view(T, -1)


def _latent_rows(q, cache, slot, cuts, H, rank, scale, window, sink):
    out = torch.empty(q.shape[0], H * rank, device=DEV)
    at = 0
    for c in cuts:
        b = make_batch([(slot, at, c)])
        ops.latent_attn(q[at:at + c].to(DEV), cache, b.meta, None, out[at:at + c], H, rank, 0, scale, at + c, window=window,
                        sink=sink.to(DEV) if sink is not None else None)
        at += c
    return out


@pytest.mark.parametrize("H,rank,window", [(4, 32, 1), (3, 20, 5), (9, 264, 31), (2, 40, 32), (1, 64, 33), (5, 24, 65), (4, 32, 150), (4, 32, 1000), (2, 40, 0)])
def test_latent_attention_kernel_with_window_and_sink(H, rank, window):
    """Prompts, portions, and single rows (whose keys are split over several blocks once the window holds 128 of them)."""
    g = gen(2)
    n = 200
    c, q = bf(torch.randn(n, rank, generator=g)), torch.randn(n, H * rank, generator=g)
    for dt in (F32, BF16):                                            # bf16 caches hold the same numbers: the output is fp32 either way
        cache = torch.zeros(2, n, rank, dtype=dt, device=DEV)
        cache[1] = c.to(DEV, dt)
        for sink in (None, torch.randn(H, generator=gen(3)) * 2.0):
            want = _latent_reference(q, c, 0, H, rank, 0.3, window, sink)
            for cuts in ([n], [64, 2, 31, 103], [1] * n):
                assert rel(_latent_rows(q, cache, 1, cuts, H, rank, 0.3, window, sink), want) < 2e-5, (dt, cuts[:3], sink is None)


def test_a_key_just_inside_the_window_takes_all_the_weight_and_just_outside_none():
    """One key is made to score far above the others for every query: the last position whose window holds it returns its latent,
    the next position does not see it at all -- in a prompt, in portions and row by row.  A sink of the same size takes its part;
    a sink far above every score (beyond what exp can hold relative to them) leaves nothing and no NaN."""
    g = gen(4)
    H, rank, window, n, star = 3, 24, 70, 230, 95
    c, q = bf(torch.randn(n, rank, generator=g) * 0.1), torch.randn(n, H * rank, generator=g) * 0.1
    c[star, 0] = 8.0
    q.view(n, H, rank)[:, :, 0] = 8.0
    cache = c.to(DEV).unsqueeze(0).contiguous()
    for sink in (None, torch.tensor([64.0, 60.0, -300.0]), torch.tensor([400.0, 64.0, 0.0])):
        want = _latent_reference(q, c, 0, H, rank, 1.0, window, sink)
        for cuts in ([n], [1] * n, [94, 2, 68, 2, 64]):
            out = _latent_rows(q, cache, 0, cuts, H, rank, 1.0, window, sink)
            assert rel(out, want) < 2e-5 and bool(torch.isfinite(out).all())
            o = out.view(n, H, rank).cpu()
            a = 2 if sink is not None else 0
            for p in (95, 96, star + window - 1):
                assert rel(o[p, a], c[star]) < 1e-5                   # all the weight on the marked key
            assert rel(o[star + window, a], c[star]) > 0.1 and rel(o[94, a], c[star]) > 0.1
            if sink is not None and float(sink[0]) == 400.0:
                assert float(o[:, 0].abs().max()) < 1e-30


@pytest.mark.parametrize("E,top", [(6, 2), (1, 1), (8, 8), (70, 5)])
def test_router_with_sigmoid_scores(E, top):
    """Scores are not renormalised; the logits sit in the left columns of a wider buffer; large logits whose sigmoids round to 1 keep
    their order; a correction takes part in the choice only."""
    g = gen(5)
    M = 33
    z = torch.randn(M, E + 1, generator=g) * 3.0
    z[0, :E] = 20.0 + torch.randperm(E, generator=g).float()
    idx, wt = torch.empty(M, top, dtype=torch.int32, device=DEV), torch.empty(M, top, device=DEV)
    ops.router_topk(z.to(DEV)[:, :E], top, idx, wt, renorm=False, sigmoid=True)
    val, ref = torch.topk(z[:, :E], top, dim=-1)
    assert torch.equal(idx.cpu().long(), ref) and rel(wt, torch.sigmoid(val.double())) < 1e-6
    corr = torch.randn(E, generator=g)
    ops.router_topk(z.to(DEV)[:, :E], top, idx, wt, renorm=True, sigmoid=True, correction=corr.to(DEV))
    s = torch.sigmoid(z[:, :E].double())
    ref = torch.topk(s + corr.double(), top, dim=-1).indices
    v = s.gather(1, ref)
    assert torch.equal(idx.cpu().long()[1:], ref[1:]) and rel(wt[1:], (v / v.sum(-1, keepdim=True))[1:]) < 1e-5


@pytest.mark.parametrize("M,dtype,E,top,shared", [(5, F32, 6, 2, 16), (5, BF16, 6, 2, 40), (90, F32, 5, 3, 0), (90, BF16, 5, 3, 24), (300, BF16, 6, 2, 24),
                                                  (600, BF16, 3, 1, 0), (300, F32, 4, 4, 9), (7, F32, 1, 1, 8)])
def test_experts_weighed_on_the_way_in_in_every_form(M, dtype, E, top, shared):
    """Few pairs (one warp per output), the grouped launch, and (bf16, many pairs) the tensor-core form; expert 1 gets no token; the
    shared expert's gate is open for some tokens and shut for others.  The scores are far from 1, so that a weight on the expert's
    output instead of its input would show."""
    g = gen(6)
    W, ff = 64, 24
    router = bf(torch.randn(E, W, generator=g) * 2.0 * W ** -0.5)
    router[:, 0] = -0.7
    if E > top:
        router[1] = 0.0
        router[1, 0] = -30.0                                           # h[:, 0] > 0 below: expert 1 never wins
    experts = [{"gate": bf(torch.randn(ff, W, generator=g) * 2.0 * W ** -0.5), "up": bf(torch.randn(ff, W, generator=g) * 2.0 * W ** -0.5),
                "down": bf(torch.randn(W, ff, generator=g) * ff ** -0.5)} for _ in range(E)]
    h = bf(torch.randn(M, W, generator=g))
    h[:, 0] = h[:, 0].abs() + 0.5
    w = {"router": router.double()}
    for e, ex in enumerate(experts):
        w.update({f"e{e}.{k}": v.double() for k, v in ex.items()})
    sh, sg = None, None
    if shared:
        sw = {"gate": bf(torch.randn(shared, W, generator=g) * W ** -0.5), "up": bf(torch.randn(shared, W, generator=g) * W ** -0.5),
              "down": bf(torch.randn(W, shared, generator=g) * shared ** -0.5)}
        sg = bf(torch.randn(1, W, generator=g) * 3.0 * W ** -0.5)
        w.update({"shared." + k: v.double() for k, v in sw.items()})
        w["shared.sg"] = sg.double()
        sh = GatedMLP(sw, shared, ops.ACT_SILU, dtype, DEV)
    spec = {"router": {"experts": E, "top": top}, "expert": {"ff": ff}}
    want = O.moe(h.double(), w, "", dict(spec, shared={"ff": shared}) if shared else spec)
    mx = MoEFeedForward(router, experts, top, ff, ops.ACT_SILU, sh, dtype, DEV, renorm=False, score="sigmoid", weigh="input", shared_gate=sg)
    got = mx(h.to(DEV, dtype))
    assert got.dtype == F32 and rel(got, want) < (2e-5 if dtype == F32 else 2e-2)
    mx.weigh_in = False
    assert rel(mx(h.to(DEV, dtype)), want) > 0.05


def test_shared_experts_gate_and_identity_experts_go_together():
    """Options of different designs at once: input-weighed experts beside identity experts (which hand w * h back either way) and a
    gated shared expert, in the three forms."""
    g = gen(7)
    W, ff, E, top = 64, 16, 4, 3
    experts = [{k: bf(torch.randn(s, generator=g) * s[1] ** -0.5) for k, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff)))} for _ in range(E)]
    router, sg = bf(torch.randn(E + 2, W, generator=g) * 0.3), bf(torch.randn(1, W, generator=g) * 0.3)
    sw = {k: bf(torch.randn(s, generator=g) * s[1] ** -0.5) for k, s in (("gate", (8, W)), ("up", (8, W)), ("down", (W, 8)))}
    for M, dtype in ((6, F32), (100, F32), (400, BF16)):
        h = bf(torch.randn(M, W, generator=g))
        mx = MoEFeedForward(router, experts, top, ff, ops.ACT_SILU, GatedMLP(sw, 8, ops.ACT_SILU, dtype, DEV), dtype, DEV, renorm=False, identity=2,
                            score="sigmoid", weigh="input", shared_gate=sg)
        idx, wt = O.route(h.double(), router.double(), top)
        want = torch.sigmoid(h.double() @ sg.double().T) * O.gated(h.double(), {k: v.double() for k, v in sw.items()}, "", O.silu)
        for t in range(M):
            for j in range(top):
                e = int(idx[t, j])
                x = wt[t, j] * h[t].double()
                want[t] += x if e >= E else O.gated(x, {k: v.double() for k, v in experts[e].items()}, "", O.silu)
        assert rel(mx(h.to(DEV, dtype)), want) < (2e-5 if dtype == F32 else 2e-2), M


# ------------------------------------------------------------------------------------------------ the mixer alone
def _weights(H, dim, vdim, rank, W, seed, scale=2.0):
    g = gen(seed)
    w = {k: bf(torch.randn(s, generator=g) * scale * s[1] ** -0.5)
         for k, s in (("q", (H * dim, W)), ("dkv", (rank, W)), ("uk", (H * dim, rank)), ("uv", (H * vdim, rank)), ("o", (W, H * vdim)))}
    w["dkv.norm"] = bf(1.0 + 0.2 * torch.randn(rank, generator=g))
    w["sink"] = bf(2.0 * torch.randn(H, generator=g))
    return w


def _mixer(w, m, dtype=F32, own=True):
    return LatentAttentionMixer(w, m["heads"], m["dim"], 0, m["vdim"], m["kv_rank"], 0, None, m["scale"], 1e-5, dtype, DEV, gate=None,
                                window=m.get("mask", {}).get("size", 0), sink=True, own_latent=own)


def d64(w):
    return {k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("expand", [None, (1, 1000), (20, 2)])
@pytest.mark.parametrize("H,dim,vdim,rank,window,W", [(4, 16, 24, 32, 11, 64), (3, 10, 7, 20, 5, 45), (9, 24, 40, 264, 40, 96), (2, 8, 8, 24, 1, 32),
                                                      (1, 32, 32, 32, 33, 32), (2, 16, 8, 40, 0, 64)])
def test_latent_attention_mixer_alone_and_on_another_layers_latents(H, dim, vdim, rank, window, W, expand, monkeypatch):
    """The mixer with latents of its own, then a second one (other heads, other window) that reads the first one's cache in the same
    steps -- in the latent space throughout, with every portion's latents expanded into keys and values, and with the long
    portions' alone."""
    if expand:
        monkeypatch.setattr(LatentAttentionMixer, "EXPAND_ROWS", expand[0])
        monkeypatch.setattr(LatentAttentionMixer, "EXPAND_RATIO", expand[1])
    m = latent(H, dim, vdim, rank, window)["mixer"]
    m2 = latent(H + 2, dim + 3, vdim + 1, rank, 2 * window + 3 if window else 4)["mixer"]
    w, w2 = _weights(H, dim, vdim, rank, W, 20), _weights(H + 2, dim + 3, vdim + 1, rank, W, 21)
    h, h2 = bf(torch.randn(60, W, generator=gen(22))), bf(torch.randn(60, W, generator=gen(23)))
    c = O.latents(h.double(), d64(w), "", 1e-5)
    want, want2 = O.latent_attention(h.double(), c, d64(w), "", m), O.latent_attention(h2.double(), c, d64(w2), "", m2)
    mx, reader = _mixer(w, m), _mixer({k: v for k, v in w2.items() if not k.startswith("dkv")}, m2, own=False)
    assert (mx.up_k is not None) == (dim + vdim < 2 * rank)
    for label, cuts in CUTS.items():
        slots = SlotState(3, 60, DEV)
        state = mx.new_state(slots)
        state2 = reader.new_state(slots, state)
        a, b, at = [], [], 0
        for n in cuts:
            batch = make_batch([(1, at, n)])
            a.append(mx(h[at:at + n].to(DEV), batch, state).float().cpu())
            b.append(reader(h2[at:at + n].to(DEV), batch, state2).float().cpu())
            at += n
        assert rel(torch.cat(a), want) < 5e-5 and rel(torch.cat(b), want2) < 5e-5, label


@pytest.mark.parametrize("expand", [False, True])
def test_two_sequences_in_one_batch_keep_their_own_state(expand, monkeypatch):
    """Portions side by side; with ``expand`` those of 6 and more rows take expanded keys and values, the rows around them the latent
    space."""
    if expand:
        monkeypatch.setattr(LatentAttentionMixer, "EXPAND_ROWS", 6)
    W = 64
    m = latent(4, 16, 8, 32, 7)["mixer"]
    w = _weights(4, 16, 8, 32, W, 26)
    mx = _mixer(w, m)
    ha, hb = bf(torch.randn(20, W, generator=gen(29))), bf(torch.randn(9, W, generator=gen(30)))
    want_a, want_b = (O.latent_attention(h.double(), O.latents(h.double(), d64(w), "", 1e-5), d64(w), "", m) for h in (ha, hb))
    state = mx.new_state(SlotState(3, 32, DEV))
    got_a, got_b = [], []
    ia = ib = 0
    for na, nb in [(12, 1), (1, 2), (7, 6)]:                          # tokens of a, of b per step; b sits in the rows right after a
        out = mx(torch.cat([ha[ia:ia + na], hb[ib:ib + nb]]).to(DEV), make_batch([(2, ia, na), (0, ib, nb)]), state).cpu()
        got_a.append(out[:na]); got_b.append(out[na:])
        ia += na; ib += nb
    assert rel(torch.cat(got_a), want_a) < 5e-5 and rel(torch.cat(got_b), want_b) < 5e-5


# ------------------------------------------------------------------------------------------------ the model
def build(name, dtype, seed=11, std_scale=1.0, change=None):
    cfg = CASES[name] if isinstance(name, str) else name
    w = O.random_weights(cfg, seed, std_scale)
    if change:
        change(w)
    m = PazivikForCausalLM(PazivikConfig.from_dict(copy.deepcopy(cfg)), DEV, dtype).load_weights(lambda n: w[n])
    return cfg, w, m


def toks_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=gen(seed)).tolist()


def err(got, want, reduce="max"):
    """The measure a serving check would use: rms over the vocabulary of the centred difference, relative to the logits' rms."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    return float(e.max() if reduce == "max" else e.mean())


@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_fp32_and_every_layer(name):
    cfg, w, m = build(name, F32)
    toks = toks_for(cfg, 45, 1)
    trace_o, trace_m = [], []
    want = O.logits_of(cfg, w, toks, trace_o)
    got = Engine(m, 64, 2).step([{"id": 0, "tokens": toks, "want": list(range(45))}], trace=trace_m)
    assert len(trace_m) == len(trace_o) == len(cfg["layers"])
    for r, (a, b) in enumerate(zip(trace_m, trace_o)):
        assert rel(a, b) < 2e-4, f"what layer {r} hands on"
    assert err(got, want) < 2e-4


@pytest.mark.parametrize("name", sorted(CASES))
def test_bf16_model_stays_within_rounding(name):
    cfg, w, m = build(name, BF16)
    toks = toks_for(cfg, 70, 2)
    got = Engine(m, 80, 1).step([{"id": 0, "tokens": toks, "want": list(range(70))}])
    assert err(got, O.logits_of(cfg, w, toks), "mean") < 0.06


@pytest.mark.parametrize("name,dtype", [("even", F32), ("odd", F32), ("wide", F32), ("even", BF16)])
def test_portions_and_decoding_equal_the_whole_prompt(name, dtype):
    cfg, w, m = build(name, dtype)
    n = 75                                                            # long enough for expanded keys and values in the whole prompt
    toks = toks_for(cfg, n, 3)
    eng = Engine(m, 100, 2)
    whole = eng.step([{"id": "w", "tokens": toks, "want": list(range(n))}], end=["w"])
    schedules = {"token by token": [1] * n, "twos": [2] * 37 + [1], "ragged": [31, 1, 1, 2, 30, 3, 7], "stage edges": [32, 32, 8, 1, 1, 1],
                 "prompt then decode": [n - 33] + [1] * 33}
    for label, cuts in schedules.items():
        assert sum(cuts) == n
        outs, at = [], 0
        for c in cuts:
            outs.append(eng.step([{"id": label, "tokens": toks[at:at + c], "want": list(range(c))}]))
            at += c
        eng.step([], end=[label])
        if dtype == F32:
            assert err(torch.cat(outs), whole.double().cpu()) < 1e-4, label
        else:       # bf16: GEMM tiles differ with the row count, so portions differ by rounding
            assert err(torch.cat(outs), whole.double().cpu(), "mean") < 0.08, label
    if dtype == F32:
        assert err(whole, O.logits_of(cfg, w, toks)) < 2e-4


def test_unequal_requests_in_one_step_equal_each_alone():
    cfg, w, m = build("even", F32)
    eng = Engine(m, 64, 4)
    prompts = {"a": toks_for(cfg, 40, 4), "b": toks_for(cfg, 3, 5), "c": toks_for(cfg, 17, 6)}
    alone = {k: eng.step([{"id": k, "tokens": t, "want": list(range(len(t)))}], end=[k]) for k, t in prompts.items()}
    got = {k: [] for k in prompts}
    plan = [{"a": 25, "b": 3, "c": 1}, {"a": 1, "c": 10}, {"a": 14, "c": 6}]
    at = {k: 0 for k in prompts}
    for step in plan:
        entries = [{"id": k, "tokens": prompts[k][at[k]:at[k] + n], "want": list(range(n))} for k, n in step.items()]
        out = eng.step(entries)
        o = 0
        for k, n in step.items():
            got[k].append(out[o:o + n])
            o += n
            at[k] += n
    for k in prompts:
        assert at[k] == len(prompts[k])
        assert err(torch.cat(got[k]), alone[k].double().cpu()) < 1e-4, k
        assert err(alone[k], O.logits_of(cfg, w, prompts[k])) < 2e-4


def test_freed_slots_are_reused_clean_and_passes_cut_long_entries():
    """A 40-token entry runs as passes of 16, 16 and 8 rows (each pass's first bigram reaches into the pass before); a slot's next
    owner starts with the first token's own bigram row, whatever the last owner left."""
    cfg, w, m = build("odd", F32)
    eng = Engine(m, 48, 2, max_rows=16)
    t1, t2, t3 = toks_for(cfg, 40, 7), toks_for(cfg, 33, 8), toks_for(cfg, 9, 9)
    a = eng.step([{"id": 1, "tokens": t1, "want": [0, 15, 16, 39]}], end=[1])
    assert err(a, O.logits_of(cfg, w, t1)[[0, 15, 16, 39]]) < 2e-4
    b = eng.step([{"id": 2, "tokens": t2, "want": [0, 32]}, {"id": 3, "tokens": t3, "want": [8]}], end=[2])
    assert err(b[:2], O.logits_of(cfg, w, t2)[[0, 32]]) < 2e-4 and err(b[2:], O.logits_of(cfg, w, t3)[[8]]) < 2e-4
    c = eng.step([{"id": 4, "tokens": t1[:5], "want": [0, 4]}], end=[3, 4])
    assert err(c, O.logits_of(cfg, w, t1[:5])[[0, 4]]) < 2e-4
    assert eng.slots.live_tokens == 0


def _replay(eng, seq, rid, cuts):
    at = 0
    for c in cuts:
        out = eng.step([{"id": rid, "tokens": seq[at:at + c], "want": [c - 1]}])
        at += c
    eng.step([], end=[rid])
    assert at == len(seq)
    return out


@pytest.mark.parametrize("bigram", [None, (37, 5, 3)])
def test_a_token_just_outside_the_window_changes_nothing_and_just_inside_does(bigram):
    """A model of one layer: the last position's logits depend on the tokens of its window alone (and, through the bigram of the
    window's first token, on the one before).  Replacing the first token inside moves the logits as the oracle says; replacing the last one
    outside leaves them exactly as they were -- in a whole prompt, with the tail decoded, and in portions cut at the window's edge."""
    window, n = 50, 230                                               # the last position, 229, sees positions 180 .. 229
    cfg = config([latent(2, 16, 16, 24, window, scale=0.05)], vocab=50, width=32, bigram=bigram)         # flat scores: every key counts
    _, w, m = build(cfg, F32, seed=12, std_scale=1.5, change=lambda w: w["l0.mix.sink"].mul_(0.2))
    toks = toks_for(cfg, n, 10)
    first = n - window - (1 if bigram else 0)                         # the first token that the last position depends on
    inside, outside = list(toks), list(toks)
    inside[first] = (inside[first] + 7) % cfg["vocab"]
    outside[first - 1] = (outside[first - 1] + 7) % cfg["vocab"]
    base, moved = O.logits_of(cfg, w, toks)[-1:], O.logits_of(cfg, w, inside)[-1:]
    assert err(moved, base) > 1e-3 and err(O.logits_of(cfg, w, outside)[-1:], base) < 1e-12
    eng = Engine(m, n, 1)
    for cuts in ([n], [n - 40] + [1] * 40, [100, 2, 76, 1, 3, 48], [first, 1, n - first - 1], [first, n - first], [first + 1, n - first - 1], [n - 60] + [1] * 60):
        got = {k: _replay(eng, seq, k, cuts) for k, seq in (("base", toks), ("inside", inside), ("outside", outside))}
        assert err(got["base"], base) < 1e-4 and err(got["inside"], moved) < 1e-4, cuts
        assert torch.equal(got["outside"], got["base"]), cuts


@pytest.mark.parametrize("cfg_layers", [[latent(2, 16, 16, 24, 380, scale=1.0)], [latent(2, 16, 16, 24, 130, scale=1.0), latent(3, 16, 8, 24, 380, kv_from=0, scale=1.0)]])
def test_a_far_token_still_moves_the_logits_through_the_model(cfg_layers):
    """Sharp attention scores and a window of 380 (in the second model on another layer's latents, which that layer itself sees 130
    positions far): among the tokens about 350 positions back, the one whose replacement moves the last position's logits most
    (found with the oracle) is replaced; the model follows the oracle with and without the replacement."""
    cfg = config(cfg_layers, vocab=50, width=32)
    _, w, m = build(cfg, F32, seed=12, std_scale=2.0)
    n = 400
    toks = toks_for(cfg, n, 10)
    base = O.logits_of(cfg, w, toks)[-1:]
    best = (0.0, None, None)
    for far in range(n - 366, n - 346):
        variant = list(toks)
        variant[far] = (variant[far] + 7) % cfg["vocab"]
        moved = O.logits_of(cfg, w, variant)[-1:]
        best = max(best, (err(moved, base), variant, moved), key=lambda t: t[0])
    effect, variant, moved = best
    assert effect > 5e-4
    eng = Engine(m, n, 1)
    for seq, want in ((toks, base), (variant, moved)):
        for cuts in ([n], [n - 40] + [1] * 40, [100, 2, 61, 130, 3, 104]):
            assert err(_replay(eng, seq, 0, cuts), want) < 1e-4, cuts


def test_the_sink_takes_its_share_in_prompts_and_in_decoding():
    """Sinks above most scores: the oracle without them (a sink far below every score) gives other logits, with them the model's."""
    cfg = config([latent(3, 16, 16, 24, 20), latent(2, 8, 16, 24, 90, kv_from=0)], vocab=50, width=32)
    _, w, m = build(cfg, F32, seed=8, change=lambda w: (w["l0.mix.sink"].copy_(torch.tensor([3.0, 2.0, 4.0])), w["l1.mix.sink"].fill_(5.0)))
    toks = toks_for(cfg, 150, 9)
    want = O.logits_of(cfg, w, toks)
    without = dict(w, **{k: torch.full_like(v, -1e9) for k, v in w.items() if k.endswith("sink")})
    assert err(O.logits_of(cfg, without, toks), want) > 0.05
    eng = Engine(m, 150, 1)
    got = [eng.step([{"id": 0, "tokens": toks[:110], "want": list(range(110))}])] + [eng.step([{"id": 0, "tokens": [t], "want": [0]}]) for t in toks[110:]]
    assert err(torch.cat(got), want) < 2e-4


def test_long_decoding_keeps_the_state_exact():
    """260 decoded tokens: the history passes the attention kernel's stage and key-range edges and every window several times."""
    cfg, w, m = build("even", F32)
    n = 264
    toks = toks_for(cfg, n, 13)
    eng = Engine(m, n, 1)
    eng.step([{"id": 0, "tokens": toks[:4], "want": []}])
    outs = [eng.step([{"id": 0, "tokens": [t], "want": [0]}]) for t in toks[4:]]
    assert err(torch.cat(outs), O.logits_of(cfg, w, toks)[4:]) < 2e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["even", "wide"])
def test_graphed_decode_passes_equal_eager_ones_bit_for_bit(name, dtype):
    cfg, w, m = build(name, dtype)
    a, b, c = toks_for(cfg, 129, 40), toks_for(cfg, 60, 41), toks_for(cfg, 30, 42)

    def play(graphs):
        eng = Engine(m, 130, 2, graphs=graphs)
        outs = [eng.step([{"id": "a", "tokens": a[:50], "want": [49]}, {"id": "b", "tokens": b[:3], "want": [2]}])]
        for i in range(50):
            want = [] if i % 7 == 3 else [0]
            o = eng.step([{"id": "a", "tokens": [a[50 + i]], "want": want}, {"id": "b", "tokens": [b[3 + i]], "want": want}])
            assert (o is None) == (not want)
            if o is not None:
                outs.append(o)
        eng.step([], end=["b"])
        outs.append(eng.step([{"id": "c", "tokens": c[:1], "want": [0]}]))           # b's slot again; alone in its pass
        for i in range(1, 30):
            outs.append(eng.step([{"id": "c", "tokens": [c[i]], "want": [0]}, {"id": "a", "tokens": [a[99 + i]], "want": [0]}]))
        return torch.cat(outs), eng

    eager, _ = play(False)
    graphed, eng = play(True)
    assert sum(g.graph is not None for g in eng._step_graphs.values()) >= 2           # several shapes were captured and replayed
    assert torch.equal(eager, graphed)
    if dtype == F32:
        la, lc = O.logits_of(cfg, w, a), O.logits_of(cfg, w, c)
        assert err(graphed[-2:-1], lc[29:30]) < 2e-4 and err(graphed[-1:], la[128:129]) < 2e-4


def test_first_tokens_and_single_token_prompts():
    cfg, w, m = build("odd", F32)
    eng = Engine(m, 8, 3)
    for seed in (20, 21, 22):
        t = toks_for(cfg, 1, seed)
        assert err(eng.step([{"id": seed, "tokens": t, "want": [0]}]), O.logits_of(cfg, w, t)) < 2e-4
    t = toks_for(cfg, 5, 23)
    eng.step([], end=[20, 21, 22])
    got = torch.cat([eng.step([{"id": "s", "tokens": [x], "want": [0]}]) for x in t])
    assert err(got, O.logits_of(cfg, w, t)) < 2e-4


def test_sizes_that_are_equal_or_one():
    """What a configuration may make equal or 1: one head, heads and latents as wide as the model, a window of one position, a window
    longer than the sequence, one expert, a router that takes every expert, one bucket, factors of 1, a width of 2's power, no cap."""
    cfg = config([latent(1, 32, 32, 32, 1, mlp=dense(32)), latent(1, 32, 32, 32, 500, kv_from=0, mlp=moe(1, 1, 32, shared=32)),
                  latent(2, 16, 16, 1, 500, mlp=moe(3, 3, 1, shared=1)), latent(32, 1, 1, 32, 2, scale=1.0)], vocab=32, width=32, bigram=(1, 1, 1), softcap=0.0)
    _, w, m = build(cfg, F32, seed=5)
    toks = toks_for(cfg, 40, 24)
    eng = Engine(m, 40, 1)
    got = torch.cat([eng.step([{"id": 0, "tokens": toks[:17], "want": list(range(17))}]), eng.step([{"id": 0, "tokens": toks[17:], "want": list(range(23))}])])
    assert err(got, O.logits_of(cfg, w, toks)) < 2e-4


def _write_checkpoint(tmp_path, cfg, seed):
    w = O.random_weights(cfg, seed)
    d = tmp_path / "ckpt"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), {k: v.to(BF16) for k, v in w.items()})
    return str(d), w


def test_greedy_generation_through_generate_and_from_pretrained(tmp_path):
    cfg = CASES["even"]
    ckpt, w = _write_checkpoint(tmp_path, cfg, 14)
    m = registry.load_model(ckpt, device=DEV, dtype=F32)
    assert isinstance(m, PazivikForCausalLM)
    prompts = torch.tensor([toks_for(cfg, 12, 30), toks_for(cfg, 12, 31)])
    new = 10
    out = m.generate(prompts, max_new_tokens=new)
    out_chunked = m.generate(prompts, max_new_tokens=new, chunk=5)
    assert out.shape == (2, 12 + new) and torch.equal(out[:, :12], prompts)
    for b in range(2):      # teacher-forced against the oracle: every greedy pick is its argmax wherever the top-2 margin is not a near-tie
        lg = O.logits_of(cfg, w, out[b].tolist())
        for t in range(new):
            top = lg[11 + t].topk(2)
            if float(top.values[0] - top.values[1]) > 1e-3:
                assert int(out[b, 12 + t]) == int(top.indices[0]), (b, t)
                assert int(out_chunked[b, 12 + t]) == int(out[b, 12 + t])


def test_trace_runner_and_command_line_as_a_user_calls_them(tmp_path):
    """The two programs a user runs, as child processes on a small checkpoint: the trace runner in both dtypes against the
    oracle, and run.py's generation summary."""
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CASES["even"]
    ckpt, w = _write_checkpoint(tmp_path, cfg, 15)
    a, b = toks_for(cfg, 41, 50), toks_for(cfg, 6, 51)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},              # nothing wanted: no file
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:40], "want": [7]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[40:41], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [5]}], "end": ["b"]}]               # a's slot, handed out again
    la, lb = O.logits_of(cfg, w, a), O.logits_of(cfg, w, b)
    want = {0: la[[0, 29]], 2: la[[39]], 3: la[[40]], 4: lb[[5]]}
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 0.2)):
        out = tmp_path / ("out_" + dtype)
        p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", ckpt, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == ["done %d" % s["step"] for s in steps]
        assert sorted(os.listdir(out)) == ["%d.f32" % k for k in sorted(want)]
        for k, ref in want.items():
            got = torch.from_numpy(np.fromfile(out / ("%d.f32" % k), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
            assert got.shape == ref.shape and err(got, ref) < tol, (dtype, k)
    p = subprocess.run([sys.executable, os.path.join(root, "run.py"), "-m", ckpt, "--dtype", "float32", "--input-tokens", "9", "--max-new-tokens", "5",
                        "--batch-size", "2", "--num-iter", "2", "--num-warmup", "1"], text=True, capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert "Inference latency:" in p.stdout and "Throughput:" in p.stdout and "[5, 5]" in p.stdout
