"""Nuderax: a decoder-only model with latent attention (queries direct or through a latent of their own, some
layers reading an earlier layer's cache), a grouped mixture of clamped-gate experts with a shared expert, and
parallel layers on an fp32 residual: x <- x + mixer(norm1(x)) + mlp(norm2(x)).

config.json gives every size, the order of the layers and the constants; the tensor names are
embed, embed.norm, final.norm, l<i>.norm1, l<i>.norm2, l<i>.mix.{q | dq, dq.norm, uq}, l<i>.mix.{dkv, dkv.norm, uk, uv, o},
l<i>.mlp.{router, correction}, l<i>.mlp.{e<j>, shared}.{gate, up, down}.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from .. import ops
from . import register
from .layers import Cache, GroupedSigmoidRouter, LatentAttention, MixtureOfExperts, Rows

_MIXERS = {"latent_attention": False, "latent_attention_2": True}  # name -> queries through a latent


@dataclass
class MixerConfig:
    low_rank_q: bool
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    q_rank: Optional[int]
    kv_from: Optional[int]


@dataclass
class MlpConfig:
    experts: int
    top: int
    groups: int
    keep: int
    router_scale: float
    ff: int
    limit: float
    shared_ff: Optional[int]
    shared_limit: float


@dataclass
class LayerConfig:
    mixer: MixerConfig
    mlp: Optional[MlpConfig]


@dataclass
class NuderaxConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerConfig]

    @classmethod
    def parse(cls, config: dict) -> "NuderaxConfig":
        layers = []
        for i, entry in enumerate(config["layers"]):
            if entry["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            m = entry["mixer"]
            mixer = MixerConfig(_MIXERS[entry["type"]], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]),
                                int(m["kv_rank"]), float(m["scale"]), float(m["rot"]["base"]), int(m["rot"]["dims"]),
                                m.get("q_rank"), m.get("kv_from"))
            if mixer.low_rank_q and mixer.q_rank is None:
                raise ValueError(f"layer {i}: q_rank missing")
            if mixer.rot_dims % 2 or mixer.rot_dims > mixer.rot_dim:
                raise ValueError(f"layer {i}: rot.dims {mixer.rot_dims} does not fit rot_dim {mixer.rot_dim}")
            if mixer.kv_from is not None:
                if not 0 <= mixer.kv_from < i or layers[mixer.kv_from].mixer.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {mixer.kv_from} is not an earlier layer with a latent of its own")
                src = layers[mixer.kv_from].mixer
                if (src.kv_rank, src.rot_dim) != (mixer.kv_rank, mixer.rot_dim):
                    raise ValueError(f"layer {i}: latent sizes differ from layer {mixer.kv_from}")
            mlp = None
            if entry.get("mlp") is not None:
                f = entry["mlp"]
                if f.get("kind") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {f.get('kind')!r}")
                r, groups, shared = f["router"], f["router"].get("groups") or {}, f.get("shared")
                mlp = MlpConfig(int(r["experts"]), int(r["top"]), int(groups.get("count", 1)), int(groups.get("keep", 1)),
                                float(r["scale"]), int(f["expert"]["ff"]), float(f["expert"]["limit"]),
                                int(shared["ff"]) if shared else None, float(shared["limit"]) if shared else 0.0)
            layers.append(LayerConfig(mixer, mlp))
        return cls(int(config["vocab"]), int(config["width"]), float(config["norm"]["eps"]), layers)


def tensor_shapes(cfg: NuderaxConfig):
    """(name, shape) of every tensor a model of this configuration has."""
    width = cfg.width
    yield "embed", (cfg.vocab, width)
    yield "embed.norm", (width,)
    yield "final.norm", (width,)
    for i, layer in enumerate(cfg.layers):
        m, f, p = layer.mixer, layer.mlp, f"l{i}."
        q = m.heads * (m.dim + m.rot_dim)
        yield p + "norm1", (width,)
        if m.low_rank_q:
            yield p + "mix.dq", (m.q_rank, width)
            yield p + "mix.dq.norm", (m.q_rank,)
            yield p + "mix.uq", (q, m.q_rank)
        else:
            yield p + "mix.q", (q, width)
        if m.kv_from is None:
            yield p + "mix.dkv", (m.kv_rank + m.rot_dim, width)
            yield p + "mix.dkv.norm", (m.kv_rank,)
        yield p + "mix.uk", (m.heads * m.dim, m.kv_rank)
        yield p + "mix.uv", (m.heads * m.vdim, m.kv_rank)
        yield p + "mix.o", (width, m.heads * m.vdim)
        if f is None:
            continue
        yield p + "norm2", (width,)
        yield p + "mlp.router", (f.experts, width)
        yield p + "mlp.correction", (f.experts,)
        forms = [(f"e{j}", f.ff) for j in range(f.experts)]
        if f.shared_ff is not None:
            forms.append(("shared", f.shared_ff))
        for name, ff in forms:
            yield f"{p}mlp.{name}.gate", (ff, width)
            yield f"{p}mlp.{name}.up", (ff, width)
            yield f"{p}mlp.{name}.down", (width, ff)


@register("Nuderax")
class Nuderax:
    config_class = NuderaxConfig
    kernel_sources = ("moe.cu", "moe_umma.cu")
    state_shapes = ()  # no recurrent layers

    def __init__(self, cfg: NuderaxConfig, weights, dtype=torch.bfloat16, device="cuda"):
        self.cfg, self.dtype, self.device, self.vocab = cfg, dtype, torch.device(device), cfg.vocab

        def get(name, *shape, to=dtype):
            t = weights[name]
            if tuple(t.shape) != shape:
                raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {shape}")
            return t.to(device=self.device, dtype=to).contiguous()

        self.embed = get("embed", cfg.vocab, cfg.width)
        self.embed_norm, self.final_norm = get("embed.norm", cfg.width), get("final.norm", cfg.width)
        self.layers, self.cache_rows, cache_of = [], [], {}
        for i, layer in enumerate(cfg.layers):
            if layer.mixer.kv_from is None:
                cache_of[i] = len(self.cache_rows)
                self.cache_rows.append(layer.mixer.kv_rank + layer.mixer.rot_dim)
            else:
                cache_of[i] = cache_of[layer.mixer.kv_from]
            norm2 = get(f"l{i}.norm2", cfg.width) if layer.mlp is not None else None
            self.layers.append((get(f"l{i}.norm1", cfg.width), norm2, self._mixer(get, f"l{i}.mix.", layer.mixer, cache_of[i]),
                                self._mlp(get, f"l{i}.mlp.", layer.mlp) if layer.mlp is not None else None))

    def _mixer(self, get, p, m: MixerConfig, cache_layer):
        width, q = self.cfg.width, m.heads * (m.dim + m.rot_dim)
        kw = {}
        if m.low_rank_q:
            kw = dict(wdq=get(p + "dq", m.q_rank, width), dq_norm=get(p + "dq.norm", m.q_rank), wuq=get(p + "uq", q, m.q_rank))
        else:
            kw = dict(wq=get(p + "q", q, width))
        if m.kv_from is None:
            kw.update(wdkv=get(p + "dkv", m.kv_rank + m.rot_dim, width), dkv_norm=get(p + "dkv.norm", m.kv_rank))
        return LatentAttention(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.rot_base, m.rot_dims // 2, self.cfg.eps,
                               get(p + "uk", m.heads * m.dim, m.kv_rank), get(p + "uv", m.heads * m.vdim, m.kv_rank),
                               get(p + "o", width, m.heads * m.vdim), cache_layer, **kw)

    def _mlp(self, get, p, f: MlpConfig):
        width = self.cfg.width

        def pack(names, ff):
            gate_up = torch.empty((len(names), 2, ff, width), dtype=self.dtype, device=self.device)
            down = torch.empty((len(names), width, ff), dtype=self.dtype, device=self.device)
            for j, name in enumerate(names):
                gate_up[j, 0] = get(f"{p}{name}.gate", ff, width)
                gate_up[j, 1] = get(f"{p}{name}.up", ff, width)
                down[j] = get(f"{p}{name}.down", width, ff)
            return gate_up, down

        router = GroupedSigmoidRouter(get(p + "router", f.experts, width), get(p + "correction", f.experts, to=torch.float32),
                                      f.groups, f.keep, f.top, f.router_scale)
        gate_up, down = pack([f"e{j}" for j in range(f.experts)], f.ff)
        shared = pack(["shared"], f.shared_ff) if f.shared_ff is not None else (None, None)
        return MixtureOfExperts(router, gate_up, down, f.limit, *shared, f.shared_limit)

    def takes_segment(self, n: int) -> bool:
        """Whether a portion of n tokens of one sequence should go through attention's expanded form."""
        return all(mixer.takes_segment(n) for _, _, mixer, _ in self.layers)

    def forward(self, tokens, rows: Rows, cache: Cache, want, trace=None):
        """tokens int64 (rows) on the device; cache.pages[c]: pool of cache layer c; want: int64 row indices whose logits
        are computed, or None for all.  Returns fp32 logits (wanted, vocab), or None when nothing is wanted.
        trace: list that receives a copy of the residual after every layer."""
        eps = self.cfg.eps
        x = ops.embed_layer_norm(tokens, self.embed, self.embed_norm, eps)
        pending = {}
        for i, (norm1, norm2, mixer, mlp) in enumerate(self.layers):
            h1, h2 = ops.residual_layer_norm(x, norm1, norm2, eps, **pending)
            if trace is not None and i:
                trace.append(x.clone())
            pending = {"a": mixer.forward(h1, rows, cache)}
            if mlp is not None:
                pending["experts"], pending["b"] = mlp.forward(h2)
        h, _ = ops.residual_layer_norm(x, self.final_norm, None, eps, **pending)
        if trace is not None:
            trace.append(x.clone())
        if want is not None:
            if want.numel() == 0:
                return None
            h = ops.embedding(want, h)
        return ops.linear(h, self.embed, out_dtype=torch.float32)

    def weight_bytes(self) -> float:
        n = 0
        for t in self._tensors():
            n += t.numel() * t.element_size()
        return float(n)

    def _tensors(self):
        yield from (self.embed, self.embed_norm, self.final_norm)
        for norm1, norm2, mixer, mlp in self.layers:
            for part in (norm1, norm2):
                if part is not None:
                    yield part
            for obj in (mixer, mlp, mlp.router if mlp is not None else None):
                if obj is not None:
                    yield from (v for v in vars(obj).values() if isinstance(v, torch.Tensor))
