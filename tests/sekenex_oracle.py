"""Plain, slow restatement of the Sekenex design, one function per mechanism, in float64 PyTorch on the CPU.  It shares no code with
the product: convolutions visit their taps over the whole history, the attention builds the full score matrix, both recurrences
go token by token and head by head, experts are visited token by token, and the residual streams are a Python list.

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


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ------------------------------------------------------------------------------------------------ short convolution
def causal_conv(history, T, w, bias=None):
    """The convolved last ``T`` rows of ``history`` [P + T, channels] (all rows of the sequence so far); the last column of ``w``
    [channels, taps] belongs to the current row."""
    taps = w.shape[1]
    out = torch.zeros(T, history.shape[1], dtype=F64)
    first = history.shape[0] - T
    for t in range(T):
        for back in range(taps):
            if first + t - back >= 0:
                out[t] += w[:, taps - 1 - back] * history[first + t - back]
    return out if bias is None else out + bias


# ------------------------------------------------------------------------------------------------ attention
def rotate_halves(x, pos, dims, base):
    """x [T, heads, dim]: channel i of the first ``dims`` turns with channel i + dims/2."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = pos.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = u * c - v * s, v * c + u * s
    return out


def softmax_attention(q, k, v, scale):
    """q [T, H, d] are the last T positions of k [P + T, G, d], v [P + T, G, vd]; causal."""
    T, H, n, rep = q.shape[0], q.shape[1], k.shape[0], q.shape[1] // k.shape[1]
    seen = torch.arange(n)[None, :] <= (n - T + torch.arange(T))[:, None]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T * scale).masked_fill(~seen, float("-inf"))
        out[:, h] = torch.softmax(s, -1) @ v[:, h // rep]
    return out


def attention(h, w, p, m, hist):
    """``hist``: dict with the projected rows so far (before their convolutions), and the keys and values as they are attended to."""
    T, H, G, d, vd = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    pos = hist.setdefault("n", 0) + torch.arange(T)
    hist["n"] += T
    rows = {}
    for name in ("q", "k", "v"):
        raw = h @ w[p + name].T
        if m.get("conv"):
            extend(hist, "raw " + name, raw)
            rows[name] = causal_conv(hist["raw " + name], T, w[p + name + ".conv"])
        else:
            rows[name] = raw
    q, k, v = rows["q"].view(T, H, d), rows["k"].view(T, G, d), rows["v"].view(T, G, vd)
    if m.get("rot"):
        q, k = (rotate_halves(t, pos, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    extend(hist, "k", k)
    extend(hist, "v", v)
    o = softmax_attention(q, hist["k"], hist["v"], m["scale"]).reshape(T, H * vd)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def extend(hist, key, rows):
    hist[key] = rows if key not in hist else torch.cat([hist[key], rows], 0)


# ------------------------------------------------------------------------------------------------ the gated linear recurrent unit
def rglru(u, w, p, blocks, state):
    """u [T, width] -> the state after every token [T, width] and the last state."""
    T, width = u.shape
    n = width // blocks
    out = torch.zeros(T, width, dtype=F64)
    for t in range(T):
        r, i = torch.zeros(width, dtype=F64), torch.zeros(width, dtype=F64)
        for b in range(blocks):
            s = slice(b * n, (b + 1) * n)
            r[s] = torch.sigmoid(w[p + "ra"][b] @ u[t, s] + w[p + "ra.b"][b])
            i[s] = torch.sigmoid(w[p + "ri"][b] @ u[t, s] + w[p + "ri.b"][b])
        a = torch.exp(-8.0 * r * softplus(w[p + "lam"]))
        state = a * state + torch.sqrt(1.0 - a * a) * i * u[t]
        out[t] = state
    return out, state


def recurrent_block(h, w, p, m, hist):
    T = h.shape[0]
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    extend(hist, "x", h @ w[p + "x"].T + w[p + "x.b"])
    u = causal_conv(hist["x"], T, w[p + "conv"], w[p + "conv.b"])
    s, hist["S"] = rglru(u, w, p, m["blocks"], hist.get("S", torch.zeros(m["width"], dtype=F64)))
    return (s * y) @ w[p + "o"].T


def parallel(h, w, p, m, eps, hist):
    left = attention(h, w, p + "left.", m["left"], hist.setdefault("left", {}))
    right = recurrent_block(h, w, p + "right.", m["right"], hist.setdefault("right", {}))
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


# ------------------------------------------------------------------------------------------------ state-space duality
def ssd(x, B, C, dt, A, D, state):
    """x [T, H, vd], B and C [T, G, N], dt [T, H]; state [H, N, vd].  Returns y [T, H, vd] and the last state."""
    T, H, rep = x.shape[0], x.shape[1], x.shape[1] // B.shape[1]
    y = torch.zeros_like(x)
    state = state.clone()
    for t in range(T):
        for h in range(H):
            g = h // rep
            state[h] = torch.exp(-A[h] * dt[t, h]) * state[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = state[h].T @ C[t, g] + D[h] * x[t, h]
    return y, state


def gated_group_norm(y, z, w, groups, eps):
    g = (y * silu(z)).view(y.shape[0], groups, -1)
    return (g / torch.sqrt((g * g).mean(-1, keepdim=True) + eps)).reshape(y.shape) * w


def mamba2(h, w, p, m, eps, hist):
    T, H, vd, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    extend(hist, "xbc", xbc)
    xbc = silu(causal_conv(hist["xbc"], T, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    y, hist["S"] = ssd(x.view(T, H, vd), B.view(T, G, N), C.view(T, G, N), softplus(dt + w[p + "dt_bias"]), torch.exp(w[p + "A_log"]), w[p + "D"],
                       hist.get("S", torch.zeros(H, N, vd, dtype=F64)))
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


def route(h, w_router, r):
    """The ``top`` largest softmax scores (as they are) among the experts of the ``keep`` best groups."""
    s = torch.softmax(h @ w_router.T, -1)
    T, E = s.shape
    allowed = torch.ones(T, E, dtype=torch.bool)
    g = r.get("groups")
    if g:
        per = E // g["count"]
        best = s.view(T, g["count"], per).max(-1).values.topk(g["keep"], dim=-1).indices
        allowed = torch.zeros(T, E, dtype=torch.bool)
        for t in range(T):
            for b in best[t].tolist():
                allowed[t, b * per:(b + 1) * per] = True
    idx = s.masked_fill(~allowed, -1.0).topk(r["top"], dim=-1).indices
    return idx, s.gather(1, idx)


def moe(h, w, p, cfg):
    idx, wt = route(h, w[p + "router"], cfg["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            out[t] += wt[t, j] * expert(h[t], w, p + f"e{int(idx[t, j])}.")
    return out + expert(h, w, p + "shared.") if cfg.get("shared") else out


# ------------------------------------------------------------------------------------------------ residual streams
def hyper_read(streams, w_in):
    return sum(w_in[s] * x for s, x in enumerate(streams))


def hyper_write(streams, y, mix, w_out):
    return [sum(mix[s, t] * x for s, x in enumerate(streams)) + w_out[t] * y for t in range(len(streams))]


# ------------------------------------------------------------------------------------------------ the model
class Oracle:
    """Feeds portions of one sequence; keeps the sequence's state between calls."""

    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: v.to(F64) for k, v in weights.items()}
        self.hist = [{} for _ in cfg["layers"]]

    def sublayer(self, streams, hc, norm, f):
        w = self.w
        u = hyper_read(streams, w[hc + ".in"])
        return hyper_write(streams, f(rms_norm(u, w[norm], self.cfg["norm"]["eps"])), w[hc + ".mix"], w[hc + ".out"])

    def forward(self, tokens, trace=None):
        """logits [T, vocab] of the next ``tokens``; ``trace`` receives the sum of the streams after every layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][torch.tensor([int(t) for t in tokens])]
        streams = [x.clone() for _ in range(cfg["streams"])]
        for i, l in enumerate(cfg["layers"]):
            p, m, mlp = f"l{i}.", l["mixer"], l.get("mlp")
            mixer = parallel if l["type"] == "parallel" else mamba2
            streams = self.sublayer(streams, p + "hc1", p + "norm1", lambda h: mixer(h, w, p + "mix.", m, eps, self.hist[i]))
            if mlp is not None:
                ff = (lambda h: dense(h, w, p + "mlp.")) if mlp["kind"] == "dense" else (lambda h: moe(h, w, p + "mlp.", mlp))
                streams = self.sublayer(streams, p + "hc2", p + "norm2", ff)
            if trace is not None:
                trace.append(sum(streams))
        return rms_norm(sum(streams), w["final.norm"], eps) @ w["head"].T


# ------------------------------------------------------------------------------------------------ weights for the tests
def tensor_shapes(cfg):
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, l in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", l["mixer"], l.get("mlp")
        for q in (1, 2) if mlp is not None else (1,):
            out.update({f"{p}norm{q}": (W,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        x = p + "mix."
        if l["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            out.update({x + "in": (2 * inner + 2 * gn + m["heads"], W), x + "conv": (inner + 2 * gn, m["conv"]), x + "conv.b": (inner + 2 * gn,),
                        x + "norm": (inner,), x + "o": (W, inner)})
            out.update({x + k: (m["heads"],) for k in ("dt_bias", "A_log", "D")})
        else:
            a, r = m["left"], m["right"]
            H, G, d, v = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a.get("vdim", a["dim"])
            for k, n in (("q", H * d), ("k", G * d), ("v", G * v)):
                out[x + "left." + k] = (n, W)
                if a.get("conv"):
                    out[x + f"left.{k}.conv"] = (n, a["conv"])
            out.update({x + "left.g": (H * v, W), x + "left.o": (W, H * v)})
            n, b = r["width"], r["blocks"]
            for k in ("y", "x"):
                out[x + "right." + k], out[x + f"right.{k}.b"] = (n, W), (n,)
            for k in ("ra", "ri"):
                out[x + "right." + k], out[x + f"right.{k}.b"] = (b, n // b, n // b), (b, n // b)
            out.update({x + "right.conv": (n, r["conv"]), x + "right.conv.b": (n,), x + "right.lam": (n,), x + "right.o": (W, n),
                        x + "left.out": (W,), x + "right.out": (W,)})
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
            continue
        out[p + "mlp.router"] = (mlp["router"]["experts"], W)
        parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + ([("shared.", mlp["shared"]["ff"])] if mlp.get("shared") else [])
        for k, n in parts:
            out[p + "mlp." + k + "up"], out[p + "mlp." + k + "down"] = (n, W), (W, n)
    return out


def random_weights(cfg, seed, std_scale=1.0):
    """bf16-representable fp32 tensors: projections N(0, std_scale / sqrt(inputs)), norm weights around 1, biases around 0, decays
    from fast to slow, streams that stay apart without growing, routers sharp enough that choices are no close calls."""
    g = torch.Generator().manual_seed(seed)
    S = cfg["streams"]
    out = {}
    for name, shp in tensor_shapes(cfg).items():
        n = torch.randn(shp, generator=g)
        if name == "embed":
            t = n
        elif name.endswith(".mix"):
            t = 0.8 * torch.eye(S) + 0.2 / S + 0.05 * n
        elif name.endswith((".hc1.in", ".hc2.in")):
            t = 1.0 / S + 0.2 * n
        elif name.endswith((".hc1.out", ".hc2.out")):
            t = 1.0 + 0.3 * n
        elif name.endswith("conv"):
            t = 0.6 * n
        elif name.endswith(".router"):
            t = 3.0 * n * shp[1] ** -0.5
        elif name.endswith(".A_log"):
            t = 0.7 * n
        elif name.endswith(".dt_bias"):
            t = n - 2.0
        elif name.endswith(".lam"):
            t = 1.5 * n - 2.5
        elif name.endswith(".b"):
            t = 0.3 * n
        elif len(shp) >= 2:
            t = n * std_scale * shp[-1] ** -0.5
        else:
            t = 1.0 + 0.2 * n
        out[name] = t.to(torch.bfloat16).float()
    return out


def logits_of(cfg, weights, tokens, trace=None):
    with torch.no_grad():
        return Oracle(cfg, weights).forward(tokens, trace)
