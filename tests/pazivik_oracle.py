"""Plain, slow restatement of the Pazivik design, one function per mechanism, in float64 PyTorch on the CPU.  It shares no code
with the product: every cached latent is expanded into per-head keys and values, the attention builds the full score matrix
over the whole history with an explicit mask and an explicit sink column, experts are visited token by token, and state is the
history itself (latents per layer, the previous token's id).

Weights: dict name -> tensor ('l<i>.mix.q', ...), config: the dict of config.json.
"""
import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norm and activations
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------ embedding
def bigram_rows(tokens, before, b):
    """The bigram table's row of every token; ``before``: the id of the token ahead of the first one (None: there is none)."""
    rows = []
    for t in tokens:
        rows.append(b["buckets"] if before is None else (before * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"])
        before = t
    return rows


def sinusoid(pos, width):
    """[T, width]: sine and cosine of pos * 10000^(-2i/width) side by side."""
    out = torch.zeros(len(pos), width, dtype=F64)
    for t, p in enumerate(pos):
        for j in range(width):
            a = p * 10000.0 ** (-2.0 * (j // 2) / width)
            out[t, j] = math.sin(a) if j % 2 == 0 else math.cos(a)
    return out


# ------------------------------------------------------------------------------------------------ attention
def window_mask(P, T, size):
    """mask [T, P + T]: new token t (position P + t) sees the ``size`` positions that end with its own (0: all before it)."""
    i = (P + torch.arange(T))[:, None]
    j = torch.arange(P + T)[None, :]
    m = j <= i
    return m & (i - j < size) if size else m


def sink_softmax(s, mask, sink):
    """Weights over the visible keys; the sink takes its share of the denominator and is dropped."""
    s = torch.cat([s.masked_fill(~mask, float("-inf")), torch.full((s.shape[0], 1), float(sink), dtype=F64)], 1)
    return torch.softmax(s, -1)[:, :-1]


def latents(h, w, p, eps):
    return rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)


def latent_attention(h, c_all, w, p, m):
    """``c_all``: latents of the whole history, the new tokens' included."""
    T, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d)
    k = (c_all @ w[p + "uk"].T).view(-1, H, d)
    v = (c_all @ w[p + "uv"].T).view(-1, H, vd)
    mask = window_mask(c_all.shape[0] - T, T, (m.get("mask") or {}).get("size", 0))
    out = torch.zeros(T, H, vd, dtype=F64)
    for a in range(H):
        out[:, a] = sink_softmax(q[:, a] @ k[:, a].T * m["scale"], mask, w[p + "sink"][a]) @ v[:, a]
    return out.reshape(T, H * vd) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w_router, top):
    """The ``top`` largest sigmoid scores as they are."""
    s = torch.sigmoid(h @ w_router.T)
    val, idx = torch.topk(s, top, dim=-1)
    return idx, val


def moe(h, w, p, cfg):
    idx, wt = route(h, w[p + "router"], cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            out[t] += gated(wt[t, j] * h[t], w, p + f"e{int(idx[t, j])}.", silu)      # the score weighs what goes INTO the expert
    if cfg.get("shared"):
        out += torch.sigmoid(h @ w[p + "shared.sg"].T) * gated(h, w, p + "shared.", silu)
    return out


# ------------------------------------------------------------------------------------------------ the model
class Oracle:
    """Feeds portions of one sequence; keeps the sequence's state between calls."""

    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: v.to(F64) for k, v in weights.items()}
        self.c = [None] * len(cfg["layers"])           # latents of every layer that makes its own
        self.last = None
        self.n = 0

    def embed(self, tokens):
        cfg, w = self.cfg, self.w
        x = w["embed"][torch.tensor(tokens)]
        b = (cfg.get("embedding") or {}).get("bigram")
        if b:
            x = x + w["bigram"][torch.tensor(bigram_rows(tokens, self.last, b))]
        x = x + sinusoid(range(self.n, self.n + len(tokens)), cfg["width"])
        self.last = tokens[-1]
        self.n += len(tokens)
        return x

    def forward(self, tokens, trace=None):
        """logits [T, vocab] of the next ``tokens``; ``trace`` receives the stream after every layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = self.embed([int(t) for t in tokens])
        for i, l in enumerate(cfg["layers"]):
            p, m = f"l{i}.", l["mixer"]
            h = rms_norm(x, w[p + "norm1"], eps)
            src = m.get("kv_from")
            if src is None:
                c = latents(h, w, p + "mix.", eps)
                self.c[i] = c if self.c[i] is None else torch.cat([self.c[i], c], 0)
                src = i
            x = x + latent_attention(h, self.c[src], w, p + "mix.", m)
            mlp = l.get("mlp")
            if mlp is not None:
                h = rms_norm(x, w[p + "norm2"], eps)
                x = x + (gated(h, w, p + "mlp.", gelu_tanh) if mlp["kind"] == "dense" else moe(h, w, p + "mlp.", mlp))
            if trace is not None:
                trace.append(x.clone())
        z = rms_norm(x, w["final.norm"], eps) @ w["embed"].T
        cap = cfg.get("logit_softcap")
        return cap * torch.tanh(z / cap) if cap else z


# ------------------------------------------------------------------------------------------------ weights for the tests
def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        out["bigram"] = (b["buckets"] + 1, W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, v, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        out[p + "norm1"] = (W,)
        for k, shp in (("q", (H * d, W)), ("uk", (H * d, r)), ("uv", (H * v, r)), ("sink", (H,)), ("o", (W, H * v))):
            out[p + "mix." + k] = shp
        if m.get("kv_from") is None:
            out[p + "mix.dkv"], out[p + "mix.dkv.norm"] = (r, W), (r,)
        mlp = l.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = (W,)

        def ff(q, n):
            out[q + "gate"], out[q + "up"], out[q + "down"] = (n, W), (n, W), (W, n)

        if mlp["kind"] == "dense":
            ff(p + "mlp.", mlp["ff"])
            continue
        out[p + "mlp.router"] = (mlp["router"]["experts"], W)
        for e in range(mlp["router"]["experts"]):
            ff(p + f"mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            ff(p + "mlp.shared.", mlp["shared"]["ff"])
            out[p + "mlp.shared.sg"] = (1, W)
    return out


def random_weights(cfg, seed, std_scale=1.0):
    """bf16-representable fp32 tensors: projections N(0, std_scale / sqrt(inputs)), norm weights around 1, sinks around 0, routers
    sharp enough that choices are no close calls."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in tensor_shapes(cfg).items():
        if name in ("embed", "bigram"):
            t = torch.randn(shp, generator=g) * (1.0 if name == "embed" else 0.7)
        elif name.endswith(".router"):
            t = 3.0 * torch.randn(shp, generator=g) * shp[1] ** -0.5
        elif name.endswith(".sink"):
            t = torch.randn(shp, generator=g)
        elif len(shp) == 2:
            t = torch.randn(shp, generator=g) * std_scale * shp[1] ** -0.5
        else:
            t = 1.0 + 0.2 * torch.randn(shp, generator=g)
        out[name] = t.to(torch.bfloat16).float()
    return out


def logits_of(cfg, weights, tokens, trace=None):
    with torch.no_grad():
        return Oracle(cfg, weights).forward(tokens, trace)
