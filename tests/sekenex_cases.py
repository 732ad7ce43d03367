"""Small Sekenex configurations for the tests (none of them a real model's sizes): odd head counts and widths, sizes that are not
multiples of 8 or 32, states above and below the scan's row tiles, one to five residual streams, convolutions of one to six taps, attention with and
without rotation and convolution, dense layers, routers over one, some or all groups of experts, with and without a shared expert, layers
without a feed-forward."""


def mamba(heads, vdim, state, groups=1, norm_groups=1, conv=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def left(heads, kv_heads, dim, vdim, rot=None, conv=3, scale=None, base=10000.0):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if conv:
        a["conv"] = conv
    if rot:
        a["rot"] = {"base": base, "dims": rot}
    return a


def parallel(l, width, blocks, conv=4, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": l, "right": {"width": width, "blocks": blocks, "conv": conv}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, groups=None):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if groups:
        d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def config(layers, vocab, width, streams=2, eps=1e-5):
    return {"architecture": "Sekenex", "vocab": vocab, "width": width, "streams": streams, "layers": layers, "norm": {"eps": eps}}


CASES = {
    # sizes that are multiples of 8: bf16 projections run on the tensor-core GEMM (the state-space projection's width is not: 3 step sizes)
    "even": config([parallel(left(4, 2, 16, 24, rot=8), 48, 3, mlp=moe(8, 2, 24, shared=16, groups=(4, 2))), mamba(6, 16, 24, groups=3, norm_groups=2, mlp=dense(40)),
                    mamba(3, 24, 16, mlp=moe(6, 3, 16, groups=(2, 1))), parallel(left(2, 1, 32, 16, rot=32, conv=4), 64, 1, conv=2), mamba(4, 8, 64, groups=2, norm_groups=4)],
                   vocab=120, width=64, streams=2),
    # nothing divides by 8, the width is odd: every projection takes the plain kernel; three streams; no rotation, no convolution, one tap
    "odd": config([mamba(3, 7, 5, conv=5, mlp=moe(3, 1, 9, groups=(3, 3))), parallel(left(3, 3, 10, 7, conv=None), 21, 7, conv=1, mlp=dense(13)),
                   mamba(5, 3, 9, norm_groups=5, conv=1), parallel(left(6, 2, 6, 11, rot=2, conv=6, base=300.0), 30, 5, conv=6, mlp=moe(5, 5, 11, shared=3))],
                  vocab=61, width=45, streams=3, eps=1e-6),
    # wide states and heads, states that fill a row tile and states that pass it by a little, nine heads, five streams
    "wide": config([mamba(2, 40, 132, mlp=moe(6, 2, 16, shared=8, groups=(3, 1))), parallel(left(9, 3, 40, 72, rot=20), 264, 2, conv=3, mlp=dense(80)),
                    mamba(4, 72, 128, groups=4, norm_groups=3, conv=2, mlp=dense(24)), mamba(1, 34, 260, norm_groups=17)],
                   vocab=90, width=96, streams=5),
}
