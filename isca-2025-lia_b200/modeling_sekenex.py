"""Sekenex: a decoder-only language model that keeps several residual streams per token ("hyper-connections") and interleaves two
kinds of layer: state-space mixers (Mamba-2) and layers that run softmax attention and Griffin's recurrent block side by side on the
same input.

    x_1 = .. = x_S = embed[token]
    per sublayer, with its own ``in`` [S], ``mix`` [S, S], ``out`` [S] (hc1 for a layer's mixer, hc2 for its feed-forward):
        y   = sublayer(N(sum_s in[s] x_s; norm_q))
        x_t = sum_s mix[s, t] x_s + out[t] y          (all t from the old streams)
    logits = head N(sum_s x_s; final.norm)            N(z; w) = w z / rms(z)

Mixers: ``mamba2`` (``seq_layers.StateSpaceMixer``); ``parallel`` (``seq_layers.ParallelMixer``): left, causal attention over the whole history
with grouped key/value heads behind a short convolution of q, k, v and a rotation of channel pairs (i, i + dims/2), with an output gate
per channel (``SinkAttentionMixer`` without a sink); right, a gated linear recurrent unit (``GatedRecurrentMixer``); half the sum of
their normed outputs.  Feed-forwards: dense SiLU-gated, or a routed mixture of experts with a squared ReLU, chosen among the best
groups of experts by softmax scores that are not renormalised, with a shared expert (``MoEFeedForward``).

``config.json`` gives every size and constant (``SekenexConfig``); tensor names are ``embed``, ``l<i>.norm1|norm2``,
``l<i>.hc1|hc2.in|mix|out``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.  Per-sequence state lives in a
``seq_state.SlotState``; serving goes through ``engine.Engine`` (the model only implements ``new_state`` and ``forward_rows``).

dtype bfloat16: projections, caches and activations of the feed-forwards in bf16 with fp32 accumulation; the streams, norms, positions and
angles, attention scores and weights, routers, convolutions on the way into a recurrence, its gates, step sizes, decays and state in
fp32.  dtype float32: everything in true fp32.
"""
import json
import os
from dataclasses import dataclass, field

import torch

from . import _lib, ops
from .seq_layers import GatedMLP, GatedRecurrentMixer, Linear, MoEFeedForward, ParallelMixer, PlainMLP, SinkAttentionMixer, StateSpaceMixer
from .seq_state import SlotState

BF16, F32 = torch.bfloat16, torch.float32
MIXERS = ("parallel", "mamba2")
MLP_KINDS = ("dense", "moe")


def _check_layer(i, l):
    if l.get("type") not in MIXERS:
        raise ValueError(f"layer {i}: unknown mixer type {l.get('type')!r} (known: {MIXERS})")
    m = l["mixer"]
    if l["type"] == "parallel":
        a, r = m["left"], m["right"]
        a.setdefault("vdim", a["dim"])                       # value heads as wide as query/key heads unless said otherwise
        a.setdefault("kv_heads", a["heads"])                 # ungrouped unless said otherwise
        if a["heads"] % a["kv_heads"]:
            raise ValueError(f"layer {i}: {a['heads']} heads do not divide into {a['kv_heads']} groups")
        rot = a.get("rot")
        if rot is not None and (rot["dims"] % 2 or not 0 < rot["dims"] <= a["dim"]):
            raise ValueError(f"layer {i}: cannot rotate {rot['dims']} of {a['dim']} channels")
        if r["width"] % r["blocks"]:
            raise ValueError(f"layer {i}: {r['width']} channels do not divide into {r['blocks']} blocks")
    else:
        m.setdefault("groups", 1)
        m.setdefault("norm_groups", 1)
        if m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ValueError(f"layer {i}: {m['heads']} heads of {m['vdim']} in {m['groups']} groups, {m['norm_groups']} parts of the norm")
    mlp = l.get("mlp")
    if mlp is None:
        return
    mlp.setdefault("kind", "moe" if "router" in mlp else "dense")
    if mlp["kind"] not in MLP_KINDS:
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r} (known: {MLP_KINDS})")
    if mlp["kind"] == "moe":
        r = mlp["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        if r["experts"] < 1 or r["experts"] % g["count"] or not 1 <= g["keep"] <= g["count"] or not 1 <= r["top"] <= g["keep"] * (r["experts"] // g["count"]):
            raise ValueError(f"layer {i}: router takes {r['top']} of {r['experts']} experts in {g['keep']} of {g['count']} groups")


@dataclass
class SekenexConfig:
    vocab: int = 0
    width: int = 0
    streams: int = 1
    layers: list = field(default_factory=list)          # dicts: type, mixer {...}, mlp {...} | None
    norm_eps: float = 1e-6
    name: str = "sekenex"
    architectures: list = field(default_factory=lambda: ["Sekenex"])
    eos_token_id: int = -1

    @classmethod
    def from_dict(cls, c, name="sekenex"):
        for i, l in enumerate(c["layers"]):
            _check_layer(i, l)
        streams = int(c["streams"])
        if not 1 <= streams <= 16:
            raise ValueError(f"{streams} residual streams (1 to 16)")
        return cls(vocab=int(c["vocab"]), width=int(c["width"]), streams=streams, layers=c["layers"], norm_eps=float(c["norm"]["eps"]), name=name)

    def to_dict(self):
        return {"architecture": "Sekenex", "vocab": self.vocab, "width": self.width, "streams": self.streams, "layers": self.layers,
                "norm": {"eps": self.norm_eps}}

    def tensor_shapes(self):
        """name -> shape of every tensor of a checkpoint of this configuration."""
        W, V, S = self.width, self.vocab, self.streams
        out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
        for i, l in enumerate(self.layers):
            p, m, mlp = f"l{i}.", l["mixer"], l.get("mlp")
            for q in ("1", "2")[:1 if mlp is None else 2]:
                out.update({p + "norm" + q: (W,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,), p + f"hc{q}.mix": (S, S)})
            if l["type"] == "mamba2":
                H, inner, C = m["heads"], m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
                out.update({p + "mix.in": (inner + C + H, W), p + "mix.conv": (C, m["conv"]), p + "mix.conv.b": (C,), p + "mix.dt_bias": (H,),
                            p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (inner,), p + "mix.o": (W, inner)})
            else:
                a, r = m["left"], m["right"]
                q, L, R = a["heads"] * a["vdim"], p + "mix.left.", p + "mix.right."
                for k, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                    out[L + k] = (n, W)
                    if a.get("conv"):
                        out[L + k + ".conv"] = (n, a["conv"])
                n, b = r["width"], r["blocks"]
                out.update({L + "g": (q, W), L + "o": (W, q), L + "out": (W,), R + "out": (W,), R + "y": (n, W), R + "y.b": (n,), R + "x": (n, W), R + "x.b": (n,),
                            R + "conv": (n, r["conv"]), R + "conv.b": (n,), R + "ra": (b, n // b, n // b), R + "ra.b": (b, n // b),
                            R + "ri": (b, n // b, n // b), R + "ri.b": (b, n // b), R + "lam": (n,), R + "o": (W, n)})
            if mlp is None:
                continue
            if mlp["kind"] == "dense":
                f = mlp["ff"]
                out.update({p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
            else:
                out[p + "mlp.router"] = (mlp["router"]["experts"], W)
                parts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
                if mlp.get("shared") is not None:
                    parts.append(("shared", mlp["shared"]["ff"]))
                for k, f in parts:
                    out.update({p + f"mlp.{k}.up": (f, W), p + f"mlp.{k}.down": (W, f)})
        return out


class _Connection:
    """The weights with which a sublayer reads, mixes and writes the residual streams."""

    def __init__(self, w_in, mix, w_out, norm):
        self.w_in, self.mix, self.w_out, self.norm = w_in, mix, w_out, norm


class _Layer:
    def __init__(self, mixer, mlp, hc1, hc2):
        self.mixer, self.mlp, self.hc1, self.hc2 = mixer, mlp, hc1, hc2


class SekenexForCausalLM:
    step_serving = True          # served through engine.Engine (requests, slots, portions)

    def __init__(self, config, device="cuda", dtype=BF16):
        _lib.load()
        if dtype not in (BF16, F32):
            raise ValueError("dtype must be torch.bfloat16 or torch.float32")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        self.layers = []
        self.embed = self.head = self.final_norm = None

    # ---- weights
    def load_weights(self, get):
        """``get(name)`` -> CPU tensor (checkpoint dtype).  Projection weights take the model's dtype; norm weights, biases, convolutions,
        decays and the streams' weights stay fp32."""
        cfg, dev, dt = self.config, self.device, self.dtype
        shapes = cfg.tensor_shapes()

        def fetch(name):
            t = get(name)
            if tuple(t.shape) != tuple(shapes[name]):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration needs {tuple(shapes[name])}")
            return t.float()

        def vec(name):
            return fetch(name).to(dev).contiguous()

        def group(prefix):
            return {k[len(prefix):]: fetch(k) for k in shapes if k.startswith(prefix)}

        def connection(p, q):
            return _Connection(vec(p + f"hc{q}.in"), vec(p + f"hc{q}.mix"), vec(p + f"hc{q}.out"), vec(p + f"norm{q}"))

        self.embed = fetch("embed").to(device=dev, dtype=dt).contiguous()
        self.head = Linear([fetch("head")], dt, dev)
        self.final_norm = vec("final.norm")
        self.layers = []
        for i, l in enumerate(cfg.layers):
            p, m, spec = f"l{i}.", l["mixer"], l.get("mlp")
            if l["type"] == "mamba2":
                mixer = StateSpaceMixer(group(p + "mix."), m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"], m["conv"], cfg.norm_eps, dt, dev)
            else:
                a, r, wl, wr = m["left"], m["right"], group(p + "mix.left."), group(p + "mix.right.")
                left = SinkAttentionMixer(wl, a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], cfg.norm_eps, dt, dev, taps=a.get("conv"),
                                          rot=a.get("rot"), rot_halves=True, gate="channel", sink=False, ride_along=GatedRecurrentMixer.ride_along(wr))
                right = GatedRecurrentMixer(wr, r["width"], r["blocks"], r["conv"], dt, dev, projected=True)
                mixer = ParallelMixer(left, right, wl["out"], wr["out"], dev)
            mlp = None
            if spec is not None and spec["kind"] == "dense":
                mlp = GatedMLP(group(p + "mlp."), spec["ff"], ops.ACT_SILU, dt, dev)
            elif spec is not None:
                q, r, shared = p + "mlp.", spec["router"], spec.get("shared")
                experts = [{k: fetch(q + f"e{e}." + k) for k in ("up", "down")} for e in range(r["experts"])]
                g = r.get("groups")
                mlp = MoEFeedForward(fetch(q + "router"), experts, r["top"], spec["expert"]["ff"], ops.ACT_RELU_SQUARED,
                                     PlainMLP(group(q + "shared."), shared["ff"], ops.ACT_RELU_SQUARED, dt, dev) if shared is not None else None, dt, dev,
                                     renorm=False, groups=(g["count"], g["keep"]) if g else None)
            self.layers.append(_Layer(mixer, mlp, connection(p, 1), connection(p, 2) if mlp is not None else None))
        return self

    def init_weights(self, seed=0, std=None):
        """Random weights (bf16-representable) for tests and benchmarks: N(0, K^-1/2) projections, norm weights near 1, decays from fast to
        slow, streams that stay apart without growing."""
        g = torch.Generator().manual_seed(seed)
        shapes, S = self.config.tensor_shapes(), self.config.streams

        def make(name):
            shp = shapes[name]
            n = torch.randn(shp, generator=g)
            if name.endswith(".hc1.mix") or name.endswith(".hc2.mix"):
                t = 0.8 * torch.eye(S) + 0.2 / S + 0.05 * n
            elif name.endswith((".hc1.in", ".hc2.in")):
                t = 1.0 / S + 0.1 * n
            elif name.endswith("conv"):
                t = 0.5 * n
            elif name.endswith(".A_log"):
                t = 0.7 * n
            elif name.endswith((".dt_bias", ".lam")):
                t = n - 2.0
            elif name.endswith(".b"):
                t = 0.2 * n
            elif len(shp) >= 2:
                t = n * (std if std is not None else shp[-1] ** -0.5)
            else:
                t = 1.0 + 0.1 * n
            return t.to(BF16)

        cache = {}
        return self.load_weights(lambda n: cache.setdefault(n, make(n)))

    @classmethod
    def from_pretrained(cls, path, device="cuda", dtype=BF16, **unused):
        from .checkpoint import SafetensorsFile
        cfg = SekenexConfig.from_dict(json.load(open(os.path.join(path, "config.json"))), name=os.path.basename(os.path.abspath(path)) or "sekenex")
        f = SafetensorsFile(os.path.join(path, "model.safetensors"))
        try:
            return cls(cfg, device, dtype).load_weights(f.get)
        finally:
            f.close()

    def eval(self):
        return self

    # ---- serving interface (engine.Engine)
    def new_state(self, n_slots, capacity):
        slots = SlotState(n_slots, capacity, self.device)
        slots.layer_state = [layer.mixer.new_state(slots) for layer in self.layers]
        return slots

    def forward_rows(self, ids, batch, want, slots, trace=None):
        """One step: ``ids`` int64 [rows] on the device, ``batch`` a StepBatch, ``want`` int32 row indices (device) whose
        logits are returned as fp32 [len(want), vocab] (None when empty).  ``trace``: a list that receives the sum of the
        residual streams after every layer."""
        cfg, dev, dt = self.config, self.device, self.dtype
        M, W, eps = batch.rows, cfg.width, cfg.norm_eps
        x = torch.empty(M, cfg.streams, W, dtype=F32, device=dev)
        h = torch.empty(M, W, dtype=dt, device=dev)
        first = self.layers[0].hc1 if self.layers else None
        ops.streams_embed(ids, self.embed, x, first.w_in if first else None, first.norm if first else None, h if first else None, eps)
        for i, layer in enumerate(self.layers):
            # a sublayer's update of the streams also makes what the next sublayer reads
            nxt = self.layers[i + 1].hc1 if i + 1 < len(self.layers) else None
            y, after = layer.mixer(h, batch, slots.layer_state[i]), layer.hc2 if layer.mlp is not None else nxt
            self._update(x, y, layer.mixer, layer.hc1, after, h)
            if layer.mlp is not None:
                self._update(x, layer.mlp(h), None, layer.hc2, nxt, h)
            if trace is not None:
                trace.append(x.sum(1))
        if want is None or want.numel() == 0:
            return None
        n = want.numel()
        hn = torch.empty(n, W, dtype=dt, device=dev)
        ops.streams_gather(x, want, self.final_norm, hn, eps)
        logits = torch.empty(n, cfg.vocab, dtype=F32, device=dev)
        ops.linear_plain(hn, self.head.weight, logits)
        return logits

    def _update(self, x, y, mixer, hc, nxt, h):
        y2, kw = None, {}
        if isinstance(mixer, ParallelMixer):
            y, y2 = y
            kw = dict(branch_norms=mixer.branch_norms, y2=y2, scale=mixer.branch_scale)
        ops.streams_update(x, y, hc.mix, hc.w_out, nxt.w_in if nxt else None, nxt.norm if nxt else None, h if nxt else None, self.config.norm_eps, **kw)

    def graph_class(self, max_ctx):
        """What a decode pass's launches depend on besides the contents of the static buffers: the number of key ranges the
        attention splits the longest history into."""
        return ops.window_attn_split_class(max_ctx, 1 << 30) if any(l["type"] == "parallel" for l in self.config.layers) else 0

    def generate(self, input_ids, max_new_tokens=32, chunk=None, **unused):
        """Greedy generation of a batch of prompts through the step engine; returns ids [B, S + new] on the input's device."""
        from .engine import Engine
        prompts = [[int(t) for t in row] for row in input_ids.tolist()]
        eng = Engine(self, max_tokens=len(prompts[0]) + max_new_tokens, max_requests=len(prompts))
        out = eng.generate(prompts, max_new_tokens, chunk=chunk)
        return torch.tensor(out, dtype=torch.int64, device=input_ids.device)
