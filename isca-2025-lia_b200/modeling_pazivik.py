"""Pazivik: a pre-norm decoder-only language model of latent-attention layers without rotation, under a sliding window with a
sink in the softmax, some of which read an earlier layer's latent cache instead of making latents of their own; dense
(GELU-gated) or mixture-of-experts feed-forwards whose sigmoid routing scores weigh the experts' inputs, with a gated shared
expert; an embedding that adds a hashed bigram table and sine / cosine positions; the output projection is the embedding table.

    x = embed[token] + bigram[hash(previous token, token)] + wave(position)
    per layer:  x += mixer(N(x));   if the layer has a feed-forward:  x += ff(N(x))
    logits = cap * tanh(embed Nf(x) / cap)                 N(x) = w * x / rms(x)

``config.json`` gives every size and constant (``PazivikConfig``); tensor names are ``embed``, ``bigram``, ``l<i>.norm1|norm2``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.  The mixer and the feed-forwards are the general ones of ``seq_layers``;
per-sequence state (latent caches, the ids of the sequence for the bigram of a portion's first token) lives in a
``seq_state.SlotState``; serving goes through ``engine.Engine`` (the model only implements ``new_state`` and ``forward_rows``).

dtype bfloat16: projections and their activations in bf16 with fp32 accumulation; positions and angles, norms, routers, attention
scores, weights and sums, and the residual stream in fp32.  dtype float32: everything in true fp32.
"""
import json
import os
from dataclasses import dataclass, field

import torch

from . import _lib, ops
from .seq_layers import GatedMLP, LatentAttentionMixer, Linear, MoEFeedForward
from .seq_state import SlotState

BF16, F32 = torch.bfloat16, torch.float32
MIXERS = ("latent_attention",)
MLP_KINDS = ("dense", "moe")
WAVE_BASE = 10000.0             # the longest wave of the positions: fixed by the design


@dataclass
class PazivikConfig:
    vocab: int = 0
    width: int = 0
    layers: list = field(default_factory=list)          # dicts: type, mixer {...}, mlp {...} | None
    bigram: tuple = None                                # (buckets, mul_prev, mul_cur); None: no bigram table
    norm_eps: float = 1e-6
    logit_softcap: float = 0.0                          # 0: none
    name: str = "pazivik"
    architectures: list = field(default_factory=lambda: ["Pazivik"])
    eos_token_id: int = -1

    @classmethod
    def from_dict(cls, c, name="pazivik"):
        layers = c["layers"]
        for i, l in enumerate(layers):
            if l.get("type") not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {l.get('type')!r} (known: {MIXERS})")
            m, mlp = l["mixer"], l.get("mlp")
            src = m.get("kv_from")
            if src is not None:
                if not 0 <= src < i:
                    raise ValueError(f"layer {i}: kv_from names layer {src}, which does not come before it")
                other = layers[src]["mixer"]
                if other.get("kv_from") is not None or other["kv_rank"] != m["kv_rank"]:
                    raise ValueError(f"layer {i}: layer {src} has no latents of {m['kv_rank']} numbers of its own")
            if mlp is not None:
                mlp.setdefault("kind", "moe" if "router" in mlp else "dense")
                if mlp["kind"] not in MLP_KINDS:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r} (known: {MLP_KINDS})")
        b = (c.get("embedding") or {}).get("bigram")
        bigram = (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None
        return cls(vocab=int(c["vocab"]), width=int(c["width"]), layers=layers, bigram=bigram, norm_eps=float(c["norm"]["eps"]),
                   logit_softcap=float(c.get("logit_softcap") or 0.0), name=name)

    def to_dict(self):
        d = {"architecture": "Pazivik", "vocab": self.vocab, "width": self.width, "layers": self.layers, "norm": {"eps": self.norm_eps}}
        if self.bigram:
            d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d

    def tensor_shapes(self):
        """name -> shape of every tensor of a checkpoint of this configuration."""
        W, V = self.width, self.vocab
        out = {"embed": (V, W), "final.norm": (W,)}
        if self.bigram:
            out["bigram"] = (self.bigram[0] + 1, W)
        for i, l in enumerate(self.layers):
            p, m, mlp = f"l{i}.", l["mixer"], l.get("mlp")
            H, d, v, c = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            out.update({p + "norm1": (W,), p + "mix.q": (H * d, W), p + "mix.uk": (H * d, c), p + "mix.uv": (H * v, c), p + "mix.sink": (H,),
                        p + "mix.o": (W, H * v)})
            if m.get("kv_from") is None:
                out.update({p + "mix.dkv": (c, W), p + "mix.dkv.norm": (c,)})
            if mlp is None:
                continue
            out[p + "norm2"] = (W,)
            parts = [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            if mlp["kind"] == "moe":
                out[p + "mlp.router"] = (mlp["router"]["experts"], W)
                if mlp.get("shared") is not None:
                    parts.append(("shared.", mlp["shared"]["ff"]))
                    out[p + "mlp.shared.sg"] = (1, W)
            for q, f in parts:
                out.update({p + "mlp." + q + "gate": (f, W), p + "mlp." + q + "up": (f, W), p + "mlp." + q + "down": (W, f)})
        return out


class _Layer:
    def __init__(self, mixer, kv_from, mlp, norm1, norm2):
        self.mixer, self.kv_from, self.mlp, self.norm1, self.norm2 = mixer, kv_from, mlp, norm1, norm2


class PazivikForCausalLM:
    step_serving = True          # served through engine.Engine (requests, slots, portions)

    def __init__(self, config, device="cuda", dtype=BF16):
        _lib.load()
        if dtype not in (BF16, F32):
            raise ValueError("dtype must be torch.bfloat16 or torch.float32")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        self.layers = []
        self.embed = self.bigram = self.final_norm = self.wave_freq = None

    # ---- weights
    def load_weights(self, get):
        """``get(name)`` -> CPU tensor (checkpoint dtype).  Projection weights and the embedding tables take the model's dtype; norm
        weights and sinks stay fp32, the frequencies of the position waves float64."""
        cfg, dev, dt = self.config, self.device, self.dtype
        shapes = cfg.tensor_shapes()

        def fetch(name):
            t = get(name)
            if tuple(t.shape) != tuple(shapes[name]):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration needs {tuple(shapes[name])}")
            return t.float()

        def norm(name):
            return fetch(name).to(dev).contiguous()

        def gated(q, ff, act):
            return GatedMLP({k: fetch(q + k) for k in ("gate", "up", "down")}, ff, act, dt, dev)

        self.embed = fetch("embed").to(device=dev, dtype=dt).contiguous()
        self.bigram = fetch("bigram").to(device=dev, dtype=dt).contiguous() if cfg.bigram else None
        i = torch.arange((cfg.width + 1) // 2, dtype=torch.float64)
        self.wave_freq = (WAVE_BASE ** (-2.0 * i / cfg.width)).to(dev)
        self.final_norm = norm("final.norm")
        self.layers = []
        for i, l in enumerate(cfg.layers):
            p, m, spec = f"l{i}.", l["mixer"], l.get("mlp")
            w = {k[len(p) + 4:]: fetch(k) for k in shapes if k.startswith(p + "mix.")}
            src = m.get("kv_from")
            mixer = LatentAttentionMixer(w, m["heads"], m["dim"], 0, m["vdim"], m["kv_rank"], 0, None, m["scale"], cfg.norm_eps, dt, dev, gate=None,
                                         window=(m.get("mask") or {}).get("size", 0), sink=True, own_latent=src is None)
            mlp, n2 = None, None
            if spec is not None:
                q = p + "mlp."
                if spec["kind"] == "dense":
                    mlp = gated(q, spec["ff"], ops.ACT_GELU_TANH)
                else:
                    shared = spec.get("shared")
                    experts = [{k: fetch(q + f"e{e}." + k) for k in ("gate", "up", "down")} for e in range(spec["router"]["experts"])]
                    mlp = MoEFeedForward(fetch(q + "router"), experts, spec["router"]["top"], spec["expert"]["ff"], ops.ACT_SILU,
                                         gated(q + "shared.", shared["ff"], ops.ACT_SILU) if shared is not None else None, dt, dev, renorm=False,
                                         score="sigmoid", weigh="input", shared_gate=fetch(q + "shared.sg") if shared is not None else None)
                n2 = norm(p + "norm2")
            self.layers.append(_Layer(mixer, src, mlp, norm(p + "norm1"), n2))
        return self

    def init_weights(self, seed=0, std=None):
        """Random weights (bf16-representable) for tests and benchmarks: N(0, K^-1/2) projections, norm weights near 1, sinks
        near 0."""
        g = torch.Generator().manual_seed(seed)
        shapes = self.config.tensor_shapes()

        def make(name):
            shp = shapes[name]
            if name in ("embed", "bigram"):
                t = torch.randn(shp, generator=g)
            elif len(shp) == 2:
                t = torch.randn(shp, generator=g) * (std if std is not None else shp[1] ** -0.5)
            elif name.endswith(".sink"):
                t = 0.5 * torch.randn(shp, generator=g)
            else:
                t = 1.0 + 0.1 * torch.randn(shp, generator=g)
            return t.to(BF16)

        cache = {}
        return self.load_weights(lambda n: cache.setdefault(n, make(n)))

    @classmethod
    def from_pretrained(cls, path, device="cuda", dtype=BF16, **unused):
        from .checkpoint import SafetensorsFile
        cfg = PazivikConfig.from_dict(json.load(open(os.path.join(path, "config.json"))), name=os.path.basename(os.path.abspath(path)) or "pazivik")
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
        slots.tokens = slots.add_rows(1, torch.int32) if self.bigram is not None else None
        slots.layer_state = []
        for l in self.layers:              # a layer with kv_from has no rows of its own: it reads that layer's
            slots.layer_state.append(l.mixer.new_state(slots, None if l.kv_from is None else slots.layer_state[l.kv_from]))
        return slots

    def forward_rows(self, ids, batch, want, slots, trace=None):
        """One step: ``ids`` int64 [rows] on the device, ``batch`` a StepBatch, ``want`` int32 row indices (device) whose
        logits are returned as fp32 [len(want), vocab] (None when empty).  ``trace``: a list that receives a copy of the
        residual stream after every layer."""
        cfg, dev, dt = self.config, self.device, self.dtype
        M, W, eps = batch.rows, cfg.width, cfg.norm_eps
        x = torch.empty(M, W, dtype=F32, device=dev)
        h = torch.empty(M, W, dtype=dt, device=dev)
        first = self.layers[0].norm1 if self.layers else None
        ops.embed_bigram_pos(ids, self.embed, batch.meta, x, bigram=self.bigram, hashing=cfg.bigram, tokens=slots.tokens, freq=self.wave_freq,
                             norm_w=first, h=h if first is not None else None, eps=eps)
        for i, layer in enumerate(self.layers):
            y = layer.mixer(h, batch, slots.layer_state[i])
            if layer.mlp is not None:
                ops.residual_norm(x, y, layer.norm2, h, eps)
                y = layer.mlp(h)
            # the layer's last residual update also makes what the next layer reads: its first norm
            nxt = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            ops.residual_norm(x, y, nxt, h if nxt is not None else None, eps)
            if trace is not None:
                trace.append(x.clone())
        if want is None or want.numel() == 0:
            return None
        n = want.numel()
        hn = torch.empty(n, W, dtype=dt, device=dev)
        ops.rms_gather(x, want, self.final_norm, hn, eps)
        logits = torch.empty(n, cfg.vocab, dtype=F32, device=dev)
        ops.linear_plain(hn, self.embed, logits)
        if cfg.logit_softcap > 0:
            ops.softcap(logits, cfg.logit_softcap)
        return logits

    def graph_class(self, max_ctx):
        """What a decode pass's launches depend on besides the contents of the static buffers: the number of key ranges each
        layer splits the longest history's window into."""
        return tuple(sorted({ops.latent_attn_split_class(min(max_ctx, l.mixer.window) if l.mixer.window else max_ctx) for l in self.layers}))

    def generate(self, input_ids, max_new_tokens=32, chunk=None, **unused):
        """Greedy generation of a batch of prompts through the step engine; returns ids [B, S + new] on the input's device."""
        from .engine import Engine
        prompts = [[int(t) for t in row] for row in input_ids.tolist()]
        eng = Engine(self, max_tokens=len(prompts[0]) + max_new_tokens, max_requests=len(prompts))
        out = eng.generate(prompts, max_new_tokens, chunk=chunk)
        return torch.tensor(out, dtype=torch.int64, device=input_ids.device)
