"""Small Pazivik configurations for the tests (none of them a real model's sizes): odd head counts and widths, sizes that are not
multiples of 8 or 32, latents above and below 256 numbers, windows from one position to more than the sequence, layers that read
an earlier layer's latents (one or several per source, with other windows and heads than the source), dense layers, routers that
take one expert of one, some or all of them, with and without a shared expert, layers without a feed-forward, no bigram table, no
soft cap."""


def latent(heads, dim, vdim, kv_rank, window, kv_from=None, scale=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def config(layers, vocab, width, bigram=(37, 5, 3), eps=1e-5, softcap=20.0):
    c = {"architecture": "Pazivik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if bigram:
        c["embedding"] = {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}
    if softcap:
        c["logit_softcap"] = softcap
    return c


CASES = {
    # sizes that are multiples of 8: bf16 projections run on the tensor-core GEMM; two layers read the latents of layer 0 with
    # other heads and other windows; one layer without a feed-forward; routers with and without a shared expert
    "even": config([latent(4, 16, 24, 32, 11, mlp=dense(48)), latent(2, 8, 16, 32, 20, kv_from=0, mlp=moe(6, 2, 24, shared=16)),
                    latent(3, 24, 16, 40, 33, mlp=moe(4, 1, 16)), latent(4, 16, 8, 40, 7, kv_from=2),
                    latent(1, 8, 40, 32, 64, kv_from=0, mlp=moe(3, 3, 8, shared=24))], vocab=120, width=64),
    # nothing divides by 8, the width is odd (the last channel of the positions is a lone sine): every projection takes the plain
    # kernel; one expert of one; no soft cap; a bigram hash with large factors
    "odd": config([latent(3, 10, 7, 20, 5, mlp=moe(1, 1, 9, shared=5)), latent(5, 6, 11, 20, 9, kv_from=0, mlp=dense(13)),
                   latent(1, 12, 10, 17, 31, mlp=moe(5, 3, 11))], vocab=61, width=45, bigram=(23, 1000003, 998244353), eps=1e-6, softcap=0.0),
    # wide heads, a latent above 256 numbers, nine heads (two blocks of heads), a window of one position, a layer that sees its
    # whole history, no bigram table
    "wide": config([latent(9, 40, 72, 264, 40, mlp=moe(4, 4, 16, shared=8)), latent(2, 72, 136, 264, 0, kv_from=0, mlp=dense(80)),
                    latent(6, 24, 8, 48, 1, mlp=moe(7, 2, 24)), latent(10, 8, 24, 264, 100, kv_from=0, mlp=dense(16))], vocab=90, width=96, bigram=None,
                   softcap=6.0),
}
