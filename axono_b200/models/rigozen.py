"""Rigozen: a decoder-only model whose layers mix by a gated delta rule, by latent attention without positions (sliding
window, sinks) or by grouped attention whose values are the raw keys (sliding window), with a dense gated feed-forward
and norms on the sublayers' outputs, on an fp32 residual:

    x <- x + norm1(mixer(x)),   x <- x + norm2(ff(x)),   logits = embed . norm(x).

A layer may use an earlier layer's weights with a cache or state of its own.  config.json gives every size, the order of
the layers and the constants; the tensor names are embed, final.norm, l<i>.norm1, l<i>.norm2, l<i>.mlp.{gate, up, down} and
  delta             l<i>.mix.{q, k, v, b, a, g, o}, .{q, k, v}.conv, .A_log, .dt_bias, .norm
  latent_attention  l<i>.mix.{q, dkv, uk, uv, o}, .dkv.norm, .sink
  attention         l<i>.mix.{q, k, o}, .q.norm, .k.norm
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Union

import torch

from .. import ops
from . import register
from .layers import Cache, GatedDelta, GatedMLP, LatentAttention, Rows, SharedKVAttention

NORM_OFFSET = 1.0  # the residual's norm weights are stored around zero


@dataclass
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def shapes(self, width):
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        return {"q": (qk, width), "k": (qk, width), "v": (v, width), "b": (self.heads, width), "a": (self.heads, width),
                "g": (v, width), "o": (width, v), "q.conv": (qk, self.conv), "k.conv": (qk, self.conv), "v.conv": (v, self.conv),
                "A_log": (self.heads,), "dt_bias": (self.heads,), "norm": (self.vdim,)}


@dataclass
class LatentConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int

    def shapes(self, width):
        return {"q": (self.heads * self.dim, width), "dkv": (self.kv_rank, width), "dkv.norm": (self.kv_rank,),
                "uk": (self.heads * self.dim, self.kv_rank), "uv": (self.heads * self.vdim, self.kv_rank), "sink": (self.heads,),
                "o": (width, self.heads * self.vdim)}


@dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int

    def shapes(self, width):
        q, k = self.heads * self.dim, self.kv_heads * self.dim
        return {"q": (q, width), "k": (k, width), "q.norm": (q,), "k.norm": (k,), "o": (width, q)}


@dataclass
class LayerConfig:
    mixer: Union[DeltaConfig, LatentConfig, AttentionConfig]
    ff: Optional[int]
    weights_of: int  # the layer whose tensors this one uses (itself, unless it shares)


def _positive(i, m, *names):
    for name in names:
        if int(m[name]) <= 0:
            raise ValueError(f"layer {i}: {name} must be positive")
    return [int(m[name]) for name in names]


def _window(i, m) -> int:
    """How many tokens a row sees; 0 for all."""
    if m.get("mask") is None:
        return 0
    return _positive(i, m["mask"], "size")[0]


def _mixer(i, kind, m):
    if kind == "delta":
        c = DeltaConfig(*_positive(i, m, "heads", "kv_heads", "dim", "vdim", "conv"))
        if c.dim > 256:
            raise ValueError(f"layer {i}: dim above 256")
    elif kind == "latent_attention":
        return LatentConfig(*_positive(i, m, "heads", "dim", "vdim", "kv_rank"), float(m["scale"]), _window(i, m))
    elif kind == "attention":
        c = AttentionConfig(*_positive(i, m, "heads", "kv_heads", "dim"), float(m["scale"]), _window(i, m))
        if int(m.get("vdim", c.dim)) != c.dim:
            raise ValueError(f"layer {i}: vdim differs from dim, but the values are the keys")
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if c.heads % c.kv_heads:
        raise ValueError(f"layer {i}: heads is not a multiple of kv_heads")
    return c


@dataclass
class RigozenConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerConfig]

    @classmethod
    def parse(cls, config: dict) -> "RigozenConfig":
        entries, layers = config["layers"], []
        for i, entry in enumerate(entries):
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            ff = _positive(i, mlp, "ff")[0] if mlp is not None else None
            src = i
            for _ in range(len(entries)):
                if entries[src].get("weights_of") is None:
                    break
                src = int(entries[src]["weights_of"])
                if not 0 <= src < len(entries):
                    raise ValueError(f"layer {i}: weights_of {src} is no layer")
            else:
                raise ValueError(f"layer {i}: weights_of leads nowhere")
            layers.append(LayerConfig(_mixer(i, entry["type"], entry["mixer"]), ff, src))
        for i, layer in enumerate(layers):
            other = layers[layer.weights_of]
            if (layer.mixer.shapes(1), type(layer.mixer), layer.ff) != (other.mixer.shapes(1), type(other.mixer), other.ff):
                raise ValueError(f"layer {i}: differs from layer {layer.weights_of}, whose weights it uses")
        return cls(int(config["vocab"]), int(config["width"]), float(config["norm"]["eps"]), layers)


def tensor_shapes(cfg: RigozenConfig):
    """(name, shape) of every tensor a model of this configuration has."""
    width = cfg.width
    yield "embed", (cfg.vocab, width)
    yield "final.norm", (width,)
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of != i:
            continue
        yield f"l{i}.norm1", (width,)
        for name, shape in layer.mixer.shapes(width).items():
            yield f"l{i}.mix.{name}", shape
        if layer.ff is not None:
            yield f"l{i}.norm2", (width,)
            yield f"l{i}.mlp.gate", (layer.ff, width)
            yield f"l{i}.mlp.up", (layer.ff, width)
            yield f"l{i}.mlp.down", (width, layer.ff)


@register("Rigozen")
class Rigozen:
    config_class = RigozenConfig
    kernel_sources = ("delta.cu", "delta_chunk.cu", "shared_kv.cu")

    def __init__(self, cfg: RigozenConfig, weights, dtype=torch.bfloat16, device="cuda"):
        self.cfg, self.dtype, self.device, self.vocab = cfg, dtype, torch.device(device), cfg.vocab
        shapes = dict(tensor_shapes(cfg))

        def get(name):
            t = weights[name]
            if tuple(t.shape) != shapes[name]:
                raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {shapes[name]}")
            return t.to(device=self.device, dtype=dtype).contiguous()

        self.embed, self.final_norm = get("embed"), get("final.norm")
        self.layers, self.cache_rows, self.state_shapes = [], [], []
        parts = {}  # layer -> its norms, the function that makes its mixer, its feed-forward
        for i, layer in enumerate(cfg.layers):
            src = layer.weights_of
            if src not in parts:
                p, full = f"l{src}.", layer.ff is not None
                w = {name: get(f"{p}mix.{name}") for name in layer.mixer.shapes(cfg.width)}
                mlp = GatedMLP(get(p + "mlp.gate"), get(p + "mlp.up"), get(p + "mlp.down")) if full else None
                parts[src] = (get(p + "norm1"), self._mixer(layer.mixer, w), get(p + "norm2") if full else None, mlp)
            norm1, mixer, norm2, mlp = parts[src]
            self.layers.append((norm1, self._placed(mixer, layer.mixer), norm2, mlp))

    def _mixer(self, m, w):
        eps = self.cfg.eps
        if isinstance(m, DeltaConfig):
            return GatedDelta(m.heads, m.kv_heads, m.dim, m.vdim, eps, w["q"], w["k"], w["v"], w["g"], w["a"], w["b"], w["q.conv"],
                              w["k.conv"], w["v.conv"], w["A_log"], w["dt_bias"], w["norm"], w["o"], 0)
        if isinstance(m, LatentConfig):
            return LatentAttention(m.heads, m.dim, 0, m.vdim, m.kv_rank, m.scale, 1.0, 0, eps, w["uk"], w["uv"], w["o"], 0, wq=w["q"],
                                   wdkv=w["dkv"], dkv_norm=w["dkv.norm"], window=m.window, sink=w["sink"])
        return SharedKVAttention(m.heads, m.kv_heads, m.dim, m.scale, eps, w["q"], w["k"], w["q.norm"], w["k.norm"], w["o"], 0, m.window)

    def _placed(self, mixer, m):
        """The mixer with a cache or state layer of its own; the weights stay shared."""
        own = object.__new__(type(mixer))
        vars(own).update(vars(mixer))
        if isinstance(m, DeltaConfig):
            own.state_layer = len(self.state_shapes)
            self.state_shapes.append(own.state_shapes(self.dtype))
        else:
            own.cache_layer = len(self.cache_rows)
            own.window, own.scale = m.window, m.scale
            self.cache_rows.append(m.kv_rank if isinstance(m, LatentConfig) else own.row_elems)
        return own

    def takes_segment(self, n: int) -> bool:
        """Whether a portion of n tokens of one sequence should go through attention's expanded form."""
        return all(mixer.takes_segment(n) for _, mixer, _, _ in self.layers if not isinstance(mixer, GatedDelta))

    def forward(self, tokens, rows: Rows, cache: Cache, want, trace=None):
        """tokens int64 (rows) on the device; cache: what the runner keeps for the sequences; want: int64 row indices
        whose logits are computed, or None for all.  Returns fp32 logits (wanted, vocab), or None when nothing is wanted.
        trace: list that receives a copy of the residual after every layer."""
        eps = self.cfg.eps
        x, h = ops.embed_residual(tokens, self.embed)
        subs = []
        for i, (norm1, mixer, norm2, mlp) in enumerate(self.layers):
            subs.append((norm1, lambda h, mixer=mixer: mixer.forward(h, rows, cache), mlp is None))
            if mlp is not None:
                subs.append((norm2, mlp.forward, True))
        for i, (norm, sub, ends_layer) in enumerate(subs):
            final = self.final_norm if i == len(subs) - 1 else None
            h = ops.residual_post_norm(x, sub(h), norm, eps, NORM_OFFSET, final)
            if trace is not None and ends_layer:
                trace.append(x.clone())
        if want is not None:
            if want.numel() == 0:
                return None
            h = ops.embedding(want, h)
        return ops.linear(h, self.embed, out_dtype=torch.float32)

    def weight_bytes(self) -> float:
        seen = {}
        for obj in (self, *(part for layer in self.layers for part in layer)):
            for t in ([obj] if isinstance(obj, torch.Tensor) else vars(obj).values() if obj is not None else []):
                if isinstance(t, torch.Tensor):
                    seen[t.data_ptr()] = t.numel() * t.element_size()
        return float(sum(seen.values()))
