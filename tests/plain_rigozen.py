"""A plain, slow evaluation of the Rigozen design on the CPU: one function per mechanism, whole sequences, no cache,
one token or head at a time where that keeps the equation visible.  It shares no code with the product path and
checks it.

Everything runs in the dtype of the weights it is given (float64 in the tests)."""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def post_norm(x, y, w, eps):
    """Residual after a sublayer whose output y is normed; the stored weight is around zero."""
    return x + rms(y, eps) * (1 + w)


def causal_conv(x, w):
    """x (tokens, channels), w (channels, taps) with the current token's tap last; zeros before the start; then silu."""
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            if t - j >= 0:
                out[t] += w[:, taps - 1 - j] * x[t - j]
    return silu(out)


def unit(x):
    """Unit vectors over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def log_decay(a, a_log, dt_bias):
    return -torch.exp(a_log) * softplus(a + dt_bias)


def delta_rule(q, k, v, g, beta, state=None):
    """One head: q, k (tokens, dim), v (tokens, vdim), g and beta (tokens) -> outputs (tokens, vdim), last state."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        s = s * g[t]
        u = beta[t] * (v[t] - s.T @ k[t])
        s = s + torch.outer(k[t], u)
        out.append(s.T @ q[t])
    return torch.stack(out), s


def delta(w, p, h, m, eps):
    n, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(n, groups, dim)
    k = causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(n, groups, dim)
    v = causal_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(n, heads, vdim)
    q, k = unit(q) * dim ** -0.5, unit(k)
    beta = 1 / (1 + torch.exp(-(h @ w[p + "b"].T)))
    g = torch.exp(log_decay(h @ w[p + "a"].T, w[p + "A_log"], w[p + "dt_bias"]))
    gate = silu(h @ w[p + "g"].T).view(n, heads, vdim)
    outs = []
    for hd in range(heads):
        src = hd // (heads // groups)
        o, _ = delta_rule(q[:, src], k[:, src], v[:, hd], g[:, hd], beta[:, hd])
        outs.append(rms(o, eps) * w[p + "norm"] * gate[:, hd])
    return torch.cat(outs, -1) @ w[p + "o"].T


def attend_row(q, k, v, i, scale, window, sink=None):
    """Row i of one head over keys j with 0 <= i - j < window; a sink takes part in the denominator only."""
    lo = max(0, i - window + 1) if window else 0
    s = (k[lo:i + 1] @ q[i]) * scale
    top = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - top)
    total = e.sum() if sink is None else e.sum() + torch.exp(sink - top)
    return (e / total) @ v[lo:i + 1]


def window_of(m):
    return m["mask"]["size"] if m.get("mask") else 0


def latent_attention(w, p, h, m, eps):
    n, dim, vdim = h.shape[0], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(n, m["heads"], dim)
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    outs = []
    for hd in range(m["heads"]):
        k = c @ w[p + "uk"][hd * dim:(hd + 1) * dim].T
        v = c @ w[p + "uv"][hd * vdim:(hd + 1) * vdim].T
        outs.append(torch.stack([attend_row(q[:, hd], k, v, i, m["scale"], window_of(m), w[p + "sink"][hd]) for i in range(n)]))
    return torch.cat(outs, -1) @ w[p + "o"].T


def attention(w, p, h, m, eps):
    """Grouped attention whose values are the keys before their norm."""
    n, heads, groups, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(n, heads, dim)
    raw = h @ w[p + "k"].T
    k = (rms(raw, eps) * w[p + "k.norm"]).view(n, groups, dim)
    v = raw.view(n, groups, dim)
    outs = []
    for hd in range(heads):
        src = hd // (heads // groups)
        outs.append(torch.stack([attend_row(q[:, hd], k[:, src], v[:, src], i, m["scale"], window_of(m)) for i in range(n)]))
    return torch.cat(outs, -1) @ w[p + "o"].T


def dense(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"delta": delta, "latent_attention": latent_attention, "attention": attention}


def source_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, trace=None):
    """Logits (tokens, vocab) of one sequence; trace receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{source_layer(cfg, i)}."
        x = post_norm(x, MIXERS[layer["type"]](w, p + "mix.", x, layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = post_norm(x, dense(w, p + "mlp.", x), w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * (1 + w["final.norm"])) @ w["embed"].T


def greedy(cfg, w, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]


def random_weights(cfg, seed):
    """Weights as a file holds them (bfloat16), on the scale at which every mechanism shows."""
    gen = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, gain=None, mean=0.0, std=0.1):
        t = torch.randn(*shape, generator=gen, dtype=torch.float64)
        w[name] = (mean + std * t if len(shape) == 1 else t * (gain or 1 / math.sqrt(shape[1]))).to(torch.bfloat16)

    width = cfg["width"]
    put("embed", cfg["vocab"], width, gain=1.0)
    put("final.norm", width)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}."
        put(p + "norm1", width)
        if layer["type"] == "delta":
            qk, vv = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, rows in (("q", qk), ("k", qk), ("v", vv)):
                put(p + f"mix.{name}", rows, width)
                put(p + f"mix.{name}.conv", rows, m["conv"], gain=0.7)
            put(p + "mix.b", m["heads"], width, gain=2 / math.sqrt(width))
            put(p + "mix.a", m["heads"], width)
            put(p + "mix.A_log", m["heads"], mean=-1.5, std=1.0)
            put(p + "mix.dt_bias", m["heads"], mean=-1.0, std=0.5)
            put(p + "mix.norm", m["vdim"], mean=1.0)
            put(p + "mix.g", vv, width)
            put(p + "mix.o", width, vv)
        elif layer["type"] == "latent_attention":
            put(p + "mix.q", m["heads"] * m["dim"], width, gain=2 / math.sqrt(width))
            put(p + "mix.dkv", m["kv_rank"], width)
            put(p + "mix.dkv.norm", m["kv_rank"], mean=1.0)
            put(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"])
            put(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
            put(p + "mix.sink", m["heads"], mean=1.5, std=1.0)
            put(p + "mix.o", width, m["heads"] * m["vdim"])
        else:
            put(p + "mix.q", m["heads"] * m["dim"], width)
            put(p + "mix.k", m["kv_heads"] * m["dim"], width)
            put(p + "mix.q.norm", m["heads"] * m["dim"], mean=1.0, std=0.3)
            put(p + "mix.k.norm", m["kv_heads"] * m["dim"], mean=1.0, std=0.3)
            put(p + "mix.o", width, m["heads"] * m["dim"])
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            put(p + "norm2", width)
            put(p + "mlp.gate", ff, width)
            put(p + "mlp.up", ff, width)
            put(p + "mlp.down", width, ff)
    return w
