"""GPU checks of the Sekenex path against the plain float64 oracle (tests/sekenex_oracle.py): every new kernel and every mixer alone,
then the model through the step engine -- whole prompts, token-by-token decoding, portions down to two tokens, unequal requests
in one step, slots that are freed and reused, a far key that takes all the weight, keys at the edges of the attention kernel's own tiles (32
cached positions per stage, 64 per key range), inputs just inside and just outside a convolution's reach, the first tokens, long
decoding through states that hardly decay, sizes that are equal or 1, greedy generation through generate(), the trace runner and the
command line."""
import copy
import json
import os

import pytest
import torch

import lia_b200  # noqa: F401
from lia_b200 import ops, registry
from lia_b200.checkpoint import write_safetensors
from lia_b200.engine import Engine
from lia_b200.modeling_sekenex import SekenexConfig, SekenexForCausalLM
from lia_b200.seq_layers import GatedRecurrentMixer, MoEFeedForward, ParallelMixer, PlainMLP, SinkAttentionMixer, StateSpaceMixer, StepBatch
from lia_b200.seq_state import SlotState

import sekenex_oracle as O
from sekenex_cases import CASES, config, dense, left, mamba, moe, parallel

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


def d64(w):
    return {k: v.double() for k, v in w.items()}


def make_batch(portions):
    """portions: (slot, first position, tokens) in row order."""
    segs, meta, row = [], [], 0
    for slot, p0, n in portions:
        segs.append((slot, p0, row, n))
        meta += [(slot, p0 + i) for i in range(n)]
        row += n
    return StepBatch(row, i32(segs), i32(meta), max(p0 + n for _, p0, n in portions), portions=segs)


CUTS = {"whole": [90], "token by token": [1] * 90, "twos": [2] * 45, "ragged": [31, 1, 1, 2, 22, 3, 30], "stage edges": [8, 16, 8, 32, 1, 7, 18]}


# ------------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("W,S", [(45, 1), (64, 2), (256, 3), (1000, 4), (46, 5), (64, 8), (52, 9), (33, 16)])
def test_residual_streams(W, S):
    """Embedding into S streams, an update by one sublayer's output, one by two normed branches, and the read-out of a few rows; every
    weight differs, so a swapped [from, to] index or an update that reads a stream already written shows."""
    g = gen(0)
    M, V, eps = 7, 20, 1e-5
    table, norm, norm2 = bf(torch.randn(V, W, generator=g)), 1 + 0.3 * torch.randn(W, generator=g), 1 + 0.3 * torch.randn(W, generator=g)
    wy, wy2 = 1 + 0.3 * torch.randn(W, generator=g), 1 + 0.3 * torch.randn(W, generator=g)
    mix, w_out, w_in, w_in2 = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.rand(S, generator=g) + 0.2, torch.rand(S, generator=g) + 0.2
    y, ya, yb = (bf(torch.randn(M, W, generator=g) * 2) for _ in range(3))
    ids = torch.randint(0, V, (M,), generator=g)
    dev = lambda t: t.to(DEV).contiguous()  # noqa: E731
    for dt, ytype, tol in ((F32, F32, 3e-6), (BF16, BF16, 6e-3), (BF16, F32, 6e-3)):
        x, h = torch.empty(M, S, W, device=DEV), torch.empty(M, W, dtype=dt, device=DEV)
        ops.streams_embed(ids.to(DEV), table.to(DEV, dt), x, dev(w_in), dev(norm), h, eps)
        want = [table.double()[ids] for _ in range(S)]
        read = lambda ws, n: O.rms_norm(O.hyper_read(want, ws.double()), n.double(), eps)  # noqa: E731
        assert rel(x, torch.stack(want, 1)) == 0.0 and rel(h, read(w_in, norm)) < tol
        ops.streams_update(x, y.to(DEV, ytype), dev(mix), dev(w_out), dev(w_in2), dev(norm2), h, eps)
        want = O.hyper_write(want, y.double(), mix.double(), w_out.double())
        assert rel(x, torch.stack(want, 1)) < 2e-6 and rel(h, read(w_in2, norm2)) < tol
        ops.streams_update(x, ya.to(DEV, ytype), dev(mix), dev(w_out), dev(w_in), dev(norm), h, eps, branch_norms=(dev(wy), dev(wy2)), y2=yb.to(DEV, ytype), scale=0.5)
        v = 0.5 * (O.rms_norm(ya.double(), wy.double(), eps) + O.rms_norm(yb.double(), wy2.double(), eps))
        want = O.hyper_write(want, v, mix.double(), w_out.double())
        assert rel(x, torch.stack(want, 1)) < 4e-6 and rel(h, read(w_in, norm)) < tol
        ops.streams_update(x, y.to(DEV, ytype), dev(mix), dev(w_out), None, None, None, eps)                  # nothing reads on
        want = O.hyper_write(want, y.double(), mix.double(), w_out.double())
        assert rel(x, torch.stack(want, 1)) < 6e-6
        hn = torch.empty(3, W, dtype=dt, device=DEV)
        ops.streams_gather(x, i32([6, 0, 6]), dev(norm), hn, eps)
        assert rel(hn, O.rms_norm(sum(want), norm.double(), eps)[[6, 0, 6]]) < max(tol, 2e-5)


@pytest.mark.parametrize("F,groups,at", [(96, 1, 0), (96, 4, 8), (45, 5, 3), (2048, 2, 16), (34, 17, 0), (7, 7, 1), (5000, 1, 0)])
def test_gate_before_a_norm_in_groups(F, groups, at):
    g = gen(1)
    o, zz, w = torch.randn(9, F, generator=g) * 2, bf(torch.randn(9, F + 24, generator=g)), 1 + 0.3 * torch.randn(F, generator=g)
    o[:, :F // groups] *= 30.0                                            # the parts have scales of their own
    for dt, tol in ((F32, 3e-6), (BF16, 5e-3)):
        out = torch.empty(9, F, dtype=dt, device=DEV)
        z = zz.to(DEV, dt)[:, at:at + F]
        ops.silu_gate_norm(o.to(DEV), z, w.to(DEV), out, groups, 1e-5)
        assert rel(out, O.gated_group_norm(o.double(), z.double().cpu(), w.double(), groups, 1e-5)) < tol


@pytest.mark.parametrize("C,taps,H", [(40, 4, 3), (33, 1, 0), (300, 2, 5), (17, 3, 0), (24, 5, 2), (24, 16, 0)])
def test_short_convolution_and_step_sizes(C, taps, H):
    """Two sequences cut in every way, with an input bias (which must not appear before the start), an output bias, SiLU or none, beside the
    step sizes and decays; rows enough for the strips that fetch all their inputs together."""
    g = gen(2)
    n, col0, dt_col = 90, 5, C + 9
    y = bf(torch.randn(2, n, C + 9 + max(H, 1), generator=g))
    w, ib, ob = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g)
    dtb, al = torch.randn(H, generator=g), torch.randn(H, generator=g)
    for dt in (F32, BF16):
        for act in (ops.ACT_NONE, ops.ACT_SILU):
            want = torch.stack([O.causal_conv(y[s, :, col0:col0 + C].double() + ib.double(), n, w.double(), ob.double()) for s in range(2)])
            want = O.silu(want) if act == ops.ACT_SILU else want
            step = O.softplus(y[:, :, dt_col:dt_col + H].double() + dtb.double())
            for cuts in CUTS.values():
                state = torch.zeros(3, max(taps - 1, 1), C, device=DEV)
                at, got, gates_got = 0, [], []
                for c in cuts:
                    batch = make_batch([(2, at, c), (0, at, c)])
                    yy = torch.cat([y[0, at:at + c], y[1, at:at + c]]).to(DEV, dt)
                    out = torch.empty(2 * c, C + 3, device=DEV)[:, :C]
                    gates = torch.empty(2 * c, 2 * H, device=DEV) if H else None
                    ops.conv_act(yy, col0, w.to(DEV), out, batch, state=state, in_bias=ib.to(DEV), bias=ob.to(DEV), act=act, dt_col=dt_col,
                                 dt_bias=dtb.to(DEV) if H else None, a_log=al.to(DEV) if H else None, gates=gates)
                    got.append(out.view(2, c, C).cpu() if out.is_contiguous() else out.clone().view(2, c, C).cpu())
                    gates_got.append(gates.view(2, c, 2 * H).cpu() if H else None)
                    at += c
                assert rel(torch.cat(got, 1), want) < 3e-6
                if H:
                    gg = torch.cat(gates_got, 1)
                    assert rel(gg[..., :H], step) < 3e-6 and rel(gg[..., H:], torch.exp(-torch.exp(al.double()) * step)) < 3e-6
                assert not state[1].any()


@pytest.mark.parametrize("taps", [2, 4, 7])
def test_the_convolutions_reach_is_exact(taps):
    """Only the oldest tap has a weight: the output is the input taps - 1 tokens back and nothing else, across portions and in decoding; a
    large number one token further back never shows."""
    n, C = 60, 8
    y = torch.zeros(n, C)
    y[20], y[21] = 1e6, 3.0
    w = torch.zeros(C, taps)
    w[:, 0] = 1.0
    want = torch.cat([torch.zeros(taps - 1, C), y[:n - taps + 1]])
    for cuts in ([n], [1] * n, [20, 2, 38], [21, 1, 38], [22, taps - 2 or 1] + [1] * (n - 22 - (taps - 2 or 1))):
        state, at, got = torch.zeros(1, taps - 1, C, device=DEV), 0, []
        for c in cuts:
            out = torch.empty(c, C, device=DEV)
            ops.conv_act(y[at:at + c].to(DEV), 0, w.to(DEV), out, make_batch([(0, at, c)]), state=state)
            got.append(out.cpu())
            at += c
        assert torch.equal(torch.cat(got), want), cuts


@pytest.mark.parametrize("H,G,N,vd", [(4, 2, 16, 24), (3, 1, 5, 7), (2, 2, 64, 32), (5, 5, 65, 33), (6, 2, 128, 40), (1, 1, 132, 64), (2, 1, 200, 8), (2, 1, 257, 3),
                                      (1, 1, 512, 34), (4, 1, 40, 1)])
def test_state_space_scan(H, G, N, vd):
    """Against the token-by-token recurrence: whole, in portions, two sequences side by side in slots of their own, rows that allow 128-bit
    copies and rows that do not; steps from nearly 0 (the state stays) to large (it is wiped)."""
    g = gen(3)
    n = 90
    C = H * vd + 2 * G * N
    xbc = torch.randn(2, n, C, generator=g)
    dt = torch.rand(2, n, H, generator=g) ** 4 * 3.0
    A, D = torch.rand(H, generator=g) + 0.05, torch.randn(H, generator=g)
    want, last = [], []
    for s in range(2):
        x, B, Cm = torch.split(xbc[s].double(), [H * vd, G * N, G * N], -1)
        y, S = O.ssd(x.reshape(n, H, vd), B.reshape(n, G, N), Cm.reshape(n, G, N), dt[s].double(), A.double(), D.double(), torch.zeros(H, N, vd, dtype=F64))
        want.append(y.reshape(n, H * vd))
        last.append(S.transpose(1, 2))
    gates = torch.cat([dt, torch.exp(-A * dt)], -1)
    for pad in (0, (-C) % 4):
        for cuts in CUTS.values():
            S = torch.zeros(3, H, vd, N, device=DEV)
            at, got = 0, []
            for c in cuts:
                batch = make_batch([(1, at, c), (2, at, c)])
                buf = torch.empty(2 * c, C + pad, device=DEV)[:, :C]
                buf.copy_(torch.cat([xbc[0, at:at + c], xbc[1, at:at + c]]))
                o = torch.empty(2 * c, H * vd, device=DEV)
                ops.ssd_scan(buf, torch.cat([gates[0, at:at + c], gates[1, at:at + c]]).to(DEV).contiguous(), D.to(DEV), S, batch.segs, H, G, N, vd, o)
                got.append(o.view(2, c, H * vd).cpu())
                at += c
            assert rel(torch.cat(got, 1), torch.stack(want)) < 2e-5 and rel(S[1:], torch.stack(last)) < 2e-5 and not S[0].any()


@pytest.mark.parametrize("width,blocks", [(48, 3), (21, 7), (5, 1), (16, 16), (264, 2)])
def test_gated_recurrent_unit_scan(width, blocks):
    """Sweeps of 128 tokens, whole and cut; decays from almost 1 (where 1 - a^2 loses everything if it is taken as it stands) to almost 0."""
    g = gen(4)
    n, per = 300, width // blocks
    u, zr, zi = (torch.randn(n, width, generator=g) for _ in range(3))
    br, bi = torch.randn(width, generator=g), torch.randn(width, generator=g)
    c = -8.0 * O.softplus(torch.linspace(-16.0, 3.0, width).double())
    y, yb = bf(torch.randn(n, width + 8, generator=g)), torch.randn(width, generator=g)
    la = c * torch.sigmoid(zr.double() + br.double())
    b = torch.sqrt(-torch.expm1(2 * la)) * torch.sigmoid(zi.double() + bi.double()) * u.double()
    s, S = torch.zeros(n, width, dtype=F64), torch.zeros(width, dtype=F64)
    for t in range(n):
        S = torch.exp(la[t]) * S + b[t]
        s[t] = S
    want = s * O.gelu_tanh(y[:, 3:3 + width].double() + yb.double())
    z = torch.stack([zr.view(n, blocks, per), zi.view(n, blocks, per)], 2).reshape(n, 2 * width)
    zb = torch.stack([br.view(blocks, per), bi.view(blocks, per)], 1).reshape(-1)
    for dt, tol in ((F32, 1e-5), (BF16, 5e-3)):
        for cuts in ([n], [1] * n, [128, 2, 126, 44], [127, 1, 1, 129, 42]):
            state, at, got = torch.zeros(2, width, device=DEV), 0, []
            for k in cuts:
                out = torch.empty(k, width, dtype=dt, device=DEV)
                ops.rglru_scan(u[at:at + k].to(DEV), z[at:at + k].to(DEV), zb.to(DEV), c.float().to(DEV), y[at:at + k].to(DEV, dt)[:, 3:3 + width], yb.to(DEV), state,
                               make_batch([(1, at, k)]).segs, blocks, out)
                got.append(out)
                at += k
            assert rel(torch.cat(got), want) < tol and rel(state[1], S) < 1e-5 and not state[0].any()
            big = s.abs().amax(0) > 0                                   # the slowest channels on their own scale
            assert float(((state[1].double().cpu() - S).abs() / s.abs().amax(0).clamp_min(1e-30))[big].max()) < 1e-4


@pytest.mark.parametrize("E,top,groups", [(8, 3, (4, 2)), (8, 2, (4, 2)), (6, 3, (2, 1)), (16, 1, (16, 1)), (12, 4, (1, 1)), (70, 5, (7, 3)), (9, 9, (3, 3)), (64, 6, (32, 5))])
def test_router_chooses_among_the_best_groups(E, top, groups):
    g = gen(5)
    M = 65
    z = torch.randn(M, E, generator=g) * 3.0
    idx, wt = torch.empty(M, top, dtype=torch.int32, device=DEV), torch.empty(M, top, device=DEV)
    ops.router_topk(z.to(DEV), top, idx, wt, renorm=False, groups=groups[0], keep=groups[1])
    ref, val = O.route(z.double(), torch.eye(E, dtype=F64), {"top": top, "groups": {"count": groups[0], "keep": groups[1]}})
    assert torch.equal(idx.cpu().long(), ref) and rel(wt, val) < 1e-6
    if groups[1] < groups[0]:
        free, _ = O.route(z.double(), torch.eye(E, dtype=F64), {"top": top})
        assert torch.equal(free, ref) == (top <= groups[1])             # (the best of as many groups are always in the best groups)
    corr = torch.randn(E, generator=g)                                  # with an option of other designs: a group then ranks by its corrected scores
    ops.router_topk(z.to(DEV), top, idx, wt, renorm=True, sigmoid=True, correction=corr.to(DEV), groups=groups[0], keep=groups[1])
    s = torch.sigmoid(z.double())
    ch = (s + corr.double()).view(M, groups[0], -1)
    best = ch.max(-1).values.topk(groups[1], dim=-1).indices
    mask = torch.zeros(M, groups[0], dtype=torch.bool).scatter_(1, best, True)
    ref = ch.masked_fill(~mask[:, :, None], float("-inf")).reshape(M, E).topk(top, dim=-1).indices
    v = s.gather(1, ref)
    assert torch.equal(idx.cpu().long(), ref) and rel(wt, v / v.sum(-1, keepdim=True)) < 1e-5


@pytest.mark.parametrize("M,dtype,E,top,groups,shared", [(5, F32, 6, 3, (3, 2), 16), (5, BF16, 6, 2, (3, 1), 40), (90, F32, 6, 3, (2, 1), 0), (90, BF16, 6, 3, (2, 2), 24),
                                                         (300, BF16, 8, 2, (4, 2), 24), (600, BF16, 3, 1, None, 0), (300, F32, 4, 4, None, 9), (7, F32, 1, 1, (1, 1), 8)])
def test_squared_relu_experts_in_every_form(M, dtype, E, top, groups, shared):
    """Few pairs (one warp per output), the grouped launch, and (bf16, many pairs) the tensor-core form; the first group gets no token."""
    g = gen(6)
    W, ff = 64, 24
    router = bf(torch.randn(E, W, generator=g) * 2.0 * W ** -0.5)
    if groups and groups[1] < groups[0]:
        router[:E // groups[0]] = 0.0
        router[:E // groups[0], 0] = -30.0                                # h[:, 0] > 0 below
    h = bf(torch.randn(M, W, generator=g))
    h[:, 0] = h[:, 0].abs() + 0.5
    names = [f"e{e}." for e in range(E)] + (["shared."] if shared else [])
    w = {"router": router}
    for k in names:
        n = shared if k == "shared." else ff
        w.update({k + "up": bf(torch.randn(n, W, generator=g) * 2.0 * W ** -0.5), k + "down": bf(torch.randn(W, n, generator=g) * n ** -0.5)})
    spec = {"router": {"experts": E, "top": top}, "shared": shared}
    if groups:
        spec["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    want = O.moe(h.double(), d64(w), "", spec)
    sh = PlainMLP({k: w["shared." + k] for k in ("up", "down")}, shared, ops.ACT_RELU_SQUARED, dtype, DEV) if shared else None
    mx = MoEFeedForward(router, [{k: w[f"e{e}." + k] for k in ("up", "down")} for e in range(E)], top, ff, ops.ACT_RELU_SQUARED, sh, dtype, DEV, renorm=False, groups=groups)
    got = mx(h.to(DEV, dtype))
    assert got.dtype == F32 and rel(got, want) < (2e-5 if dtype == F32 else 2e-2)
    if float(O.route(h.double(), router.double(), spec["router"])[1].sum(-1).min()) < 0.8:
        mx.renorm = True
        assert rel(mx(h.to(DEV, dtype)), want) > 0.05                    # renormalised scores would show


# ------------------------------------------------------------------------------------------------ mixers alone
def _group(cfg, seed, prefix, scale=1.0, change=None):
    w = {k[len(prefix):]: v for k, v in O.random_weights(cfg, seed, scale).items() if k.startswith(prefix)}
    if change:
        change(w)
    return w


def _left_mixer(wl, a, dtype=F32, ride_along=()):
    return SinkAttentionMixer(wl, a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], 1e-5, dtype, DEV, taps=a.get("conv"), rot=a.get("rot"), rot_halves=True,
                              gate="channel", sink=False, ride_along=ride_along)


def _run(mx, h, cuts, slot=1, capacity=None):
    state, at, out = mx.new_state(SlotState(3, capacity or h.shape[0], DEV)), 0, []
    for c in cuts:
        y = mx(h[at:at + c].to(DEV), make_batch([(slot, at, c)]), state)
        out.append(tuple(t.float().cpu() for t in y) if isinstance(y, tuple) else y.float().cpu())
        at += c
    return tuple(torch.cat(t) for t in zip(*out)) if isinstance(out[0], tuple) else torch.cat(out)


@pytest.mark.parametrize("heads,vdim,state,groups,norm_groups,conv,W", [(4, 16, 24, 2, 2, 4, 64), (3, 7, 5, 1, 1, 5, 45), (2, 40, 132, 1, 4, 2, 32), (6, 8, 64, 3, 6, 1, 40)])
def test_state_space_mixer_alone(heads, vdim, state, groups, norm_groups, conv, W):
    l = mamba(heads, vdim, state, groups, norm_groups, conv)
    w = _group(config([l], 10, W), 20, "l0.mix.", 1.5)
    h = bf(torch.randn(90, W, generator=gen(21)))
    want = O.mamba2(h.double(), d64(w), "", l["mixer"], 1e-5, {})
    mx = StateSpaceMixer(w, heads, vdim, state, groups, norm_groups, conv, 1e-5, F32, DEV)
    for label, cuts in CUTS.items():
        assert rel(_run(mx, h, cuts), want) < 5e-5, label


@pytest.mark.parametrize("shared", [True, False])
@pytest.mark.parametrize("a,width,blocks,conv,W", [(left(4, 2, 16, 24, rot=8), 48, 3, 4, 64), (left(3, 3, 10, 7, conv=None), 21, 7, 1, 45), (left(6, 2, 6, 11, rot=6, conv=6), 30, 1, 6, 33),
                                                   (left(9, 1, 40, 72, rot=20), 264, 2, 3, 96), (left(1, 1, 8, 8, rot=2, conv=1), 16, 16, 2, 16)])
def test_attention_and_recurrent_block_alone_and_side_by_side(a, width, blocks, conv, W, shared):
    """Both mixers, in one projection and in two, under every way of cutting; the sum of their normed outputs through the stream update."""
    l = parallel(a, width, blocks, conv)
    cfg = config([l], 10, W)
    wl, wr = _group(cfg, 22, "l0.mix.left.", 1.5), _group(cfg, 22, "l0.mix.right.", 1.5)
    h = bf(torch.randn(90, W, generator=gen(23)))
    want_l, want_r = O.attention(h.double(), d64(wl), "", a, {}), O.recurrent_block(h.double(), d64(wr), "", l["mixer"]["right"], {})
    ride = GatedRecurrentMixer.ride_along(wr) if shared else ()
    mx = ParallelMixer(_left_mixer(wl, a, ride_along=ride), GatedRecurrentMixer(wr, width, blocks, conv, F32, DEV, projected=shared), wl["out"], wr["out"], DEV,
                       shared_projection=shared)
    for label, cuts in CUTS.items():
        got_l, got_r = _run(mx, h, cuts)
        assert rel(got_l, want_l) < 5e-5 and rel(got_r, want_r) < 5e-5, label
    one = torch.ones(1, device=DEV)
    x = torch.zeros(90, 1, W, device=DEV)
    ops.streams_update(x, got_l.to(DEV), one, one, None, None, None, 1e-5, branch_norms=mx.branch_norms, y2=got_r.to(DEV), scale=mx.branch_scale)
    both = {"left." + k: v.double() for k, v in wl.items()} | {"right." + k: v.double() for k, v in wr.items()}
    assert rel(x[:, 0], O.parallel(h.double(), both, "", l["mixer"], 1e-5, {})) < 1e-4


def test_a_far_key_takes_all_the_weight():
    """Every query and one key (position 7) are made to score far above everything else: each later position, hundreds of tokens on, returns that
    key's value behind its gate -- in a prompt, in portions cut at stage and key-range edges, and row by row; the position before
    does not see it."""
    W, n, star = 32, 420, 7
    a = left(3, 1, 16, 16, rot=8, conv=None, scale=1.0)
    a["rot"]["base"] = 1e9                                              # (slow angles: the marked direction survives the distance)
    wl = _group(config([parallel(a, 8, 1)], 10, W), 30, "l0.mix.left.", 0.3)
    for k in ("q", "k"):
        wl[k][15::16] = 0.0                                             # the last channel of every head, beyond the rotated ones
    wl["q"][15::16, 0], wl["k"][15::16, 1] = 8.0, 8.0
    h = bf(torch.randn(n, W, generator=gen(31)) * 0.3)
    h[:, 0], h[:, 1] = 1.0, 0.0
    h[star, 1] = 1.0
    want = O.attention(h.double(), d64(wl), "", a, {})
    v = h[star].double() @ wl["v"].double().T
    gate = torch.sigmoid(h.double() @ wl["g"].double().T)
    only = (v.repeat(3) * gate) @ wl["o"].double().T
    assert rel(want[star:], only[star:]) < 1e-9 and rel(want[star - 1], only[star - 1]) > 0.1
    mx = _left_mixer(wl, a)
    for cuts in ([n], [1] * n, [6, 1, 1, 2, 54, 64, 1, 127, 164], [star, 2] + [1] * (n - star - 2)):
        assert rel(_run(mx, h, cuts), want) < 2e-5, cuts[:3]


def test_recurrences_carry_a_far_token():
    """Steps and gates that hardly decay: what token 3 wrote is still read 500 tokens later, in prompts, portions and decoding; with the
    state of the last owner left in the slot it would not agree."""
    W, n = 32, 520
    l = mamba(2, 16, 24, conv=2)
    w = _group(config([l], 10, W), 32, "l0.mix.", 1.0, lambda w: (w["A_log"].fill_(-9.0), w["dt_bias"].fill_(-1.0)))
    r = {"width": 24, "blocks": 2, "conv": 3}
    wr = _group(config([parallel(left(1, 1, 4, 4), 24, 2, 3)], 10, W), 33, "l0.mix.right.", 1.0, lambda w: w["lam"].fill_(-10.0))
    h = bf(torch.randn(n, W, generator=gen(34)) * 0.2)
    h[3] *= 100.0
    without = h.clone()
    without[3] = 0.0
    for mx, f in ((StateSpaceMixer(w, 2, 16, 24, 1, 1, 2, 1e-5, F32, DEV), lambda h: O.mamba2(h.double(), d64(w), "", l["mixer"], 1e-5, {})),
                  (GatedRecurrentMixer(wr, 24, 2, 3, F32, DEV), lambda h: O.recurrent_block(h.double(), d64(wr), "", r, {}))):
        want = f(h)
        assert rel(f(without)[-1], want[-1]) > 0.05
        for cuts in ([n], [2, 2, 2] + [1] * (n - 6), [100, 2, 3, 260, 155]):
            assert rel(_run(mx, h, cuts), want) < 5e-5, cuts[:3]


def test_two_sequences_in_one_batch_keep_their_own_state():
    W = 64
    l, m = parallel(left(4, 2, 16, 24, rot=8), 48, 3, 4), mamba(4, 16, 24, 2, 2, 4)
    cfg = config([l, m], 10, W)
    wl, wr, ws = _group(cfg, 22, "l0.mix.left."), _group(cfg, 22, "l0.mix.right."), _group(cfg, 22, "l1.mix.")
    par = ParallelMixer(_left_mixer(wl, l["mixer"]["left"], ride_along=GatedRecurrentMixer.ride_along(wr)), GatedRecurrentMixer(wr, 48, 3, 4, F32, DEV, projected=True),
                        wl["out"], wr["out"], DEV)
    ss = StateSpaceMixer(ws, 4, 16, 24, 2, 2, 4, 1e-5, F32, DEV)
    ha, hb = bf(torch.randn(40, W, generator=gen(29))), bf(torch.randn(19, W, generator=gen(30)))
    fs = (lambda h: O.attention(h.double(), d64(wl), "", l["mixer"]["left"], {}), lambda h: O.recurrent_block(h.double(), d64(wr), "", l["mixer"]["right"], {}),
          lambda h: O.mamba2(h.double(), d64(ws), "", m["mixer"], 1e-5, {}))
    sp, st = par.new_state(SlotState(3, 40, DEV)), ss.new_state(SlotState(3, 40, DEV))
    got = [([], []) for _ in range(3)]
    ia = ib = 0
    for na, nb in [(1, 1), (12, 1), (1, 2), (7, 6), (1, 1), (18, 8)]:                          # b sits in the rows right after a
        hh, batch = torch.cat([ha[ia:ia + na], hb[ib:ib + nb]]).to(DEV), make_batch([(2, ia, na), (0, ib, nb)])
        for i, y in enumerate((*par(hh, batch, sp), ss(hh, batch, st))):
            got[i][0].append(y[:na].cpu())
            got[i][1].append(y[na:].cpu())
        ia += na; ib += nb
    assert (ia, ib) == (40, 19)
    for i, f in enumerate(fs):
        assert rel(torch.cat(got[i][0]), f(ha)) < 5e-5 and rel(torch.cat(got[i][1]), f(hb)) < 5e-5, i


# ------------------------------------------------------------------------------------------------ the model
def build(name, dtype, seed=11, std_scale=1.0, change=None):
    cfg = CASES[name] if isinstance(name, str) else name
    w = O.random_weights(cfg, seed, std_scale)
    if change:
        change(w)
    m = SekenexForCausalLM(SekenexConfig.from_dict(copy.deepcopy(cfg)), DEV, dtype).load_weights(lambda n: w[n])
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
        assert rel(a, b) < 2e-4, f"the streams after layer {r}"
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
    n = 90
    toks = toks_for(cfg, n, 3)
    eng = Engine(m, 100, 2)
    whole = eng.step([{"id": "w", "tokens": toks, "want": list(range(n))}], end=["w"])
    for label, cuts in dict(CUTS, **{"prompt then decode": [n - 33] + [1] * 33}).items():
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
    plan = [{"a": 25, "b": 2, "c": 1}, {"a": 1, "b": 1, "c": 1}, {"a": 1, "c": 9}, {"a": 13, "c": 6}]
    at = {k: 0 for k in prompts}
    for step in plan:
        out = eng.step([{"id": k, "tokens": prompts[k][at[k]:at[k] + n], "want": list(range(n))} for k, n in step.items()])
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
    """A 40-token entry runs as passes of 16, 16 and 8 rows; a slot's next owner starts with empty states and convolutions, whatever the last
    owner left."""
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


@pytest.mark.parametrize("layers", [[parallel(left(2, 1, 16, 16, rot=8, scale=1.0), 32, 2)], [mamba(2, 16, 24)]])
def test_a_far_token_still_moves_the_logits_through_the_model(layers):
    """Sharp attention scores without the recurrent branch (its norm weight is 0), and slow decays: among five tokens about 350 positions back,
    the one whose replacement moves the last position's logits most (found with the oracle) is replaced; the model follows the
    oracle with and without the replacement."""
    cfg = config(layers, vocab=50, width=32)

    def change(w):
        for k, v in w.items():
            if k.endswith("right.out"):
                v.zero_()
            elif k.endswith("A_log"):
                v.fill_(-7.0)
    _, w, m = build(cfg, F32, seed=15, std_scale=2.0, change=change)
    n = 400
    toks = toks_for(cfg, n, 10)
    base = O.logits_of(cfg, w, toks)[-1:]
    best = (0.0, None, None)
    for far in range(n - 360, n - 340, 4):
        variant = list(toks)
        variant[far] = (variant[far] + 7) % cfg["vocab"]
        moved = O.logits_of(cfg, w, variant)[-1:]
        best = max(best, (err(moved, base), variant, moved), key=lambda t: t[0])
    effect, variant, moved = best
    assert effect > 5e-4
    eng = Engine(m, n, 1)
    for seq, want in ((toks, base), (variant, moved)):
        for cuts in ([n], [n - 40] + [1] * 40, [100, 2, 61, 130, 3, 104]):
            at = 0
            for c in cuts:
                out = eng.step([{"id": 0, "tokens": seq[at:at + c], "want": [c - 1]}])
                at += c
            eng.step([], end=[0])
            assert err(out, want) < 1e-4, cuts


def test_long_decoding_keeps_the_state_exact():
    """220 decoded tokens: the history passes the attention kernel's stage and key-range edges several times."""
    cfg, w, m = build("even", F32)
    n = 224
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
    t = toks_for(cfg, 7, 23)
    eng.step([], end=[20, 21, 22])
    got = torch.cat([eng.step([{"id": "s", "tokens": [x], "want": [0]}]) for x in t])
    assert err(got, O.logits_of(cfg, w, t)) < 2e-4


def test_sizes_that_are_equal_or_one():
    """What a configuration may make equal or 1: one stream, one head of one channel, states of one number, one tap, one block and blocks of one
    channel, one expert, a router that takes every expert, groups of one expert, mixers as wide as the model."""
    cfg = config([mamba(1, 32, 32, mlp=dense(32)), parallel(left(1, 1, 32, 32, rot=32, conv=1), 32, 1, 1, mlp=moe(1, 1, 32, shared=32, groups=(1, 1))),
                  mamba(32, 1, 1, groups=32, norm_groups=32, conv=1, mlp=moe(3, 3, 1, shared=1, groups=(3, 3))),
                  parallel(left(32, 32, 2, 1, rot=2, conv=2), 32, 32, 2, mlp=moe(4, 2, 8, groups=(4, 2))), mamba(2, 16, 1, norm_groups=1, conv=2)], vocab=32, width=32, streams=1)
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
    assert isinstance(m, SekenexForCausalLM)
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
