"""A plain, slow evaluation of the Nuderax design on the CPU: one function per mechanism, whole sequences,
no cache, no absorbed products, one token or head at a time where that keeps the equation visible.  It
shares no code with the product path and checks it.

Everything runs in the dtype of the weights it is given (float64 in the tests)."""
import math

import torch


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w over the last axis."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_interleaved(x, positions, base, dims):
    """x (tokens, ..., n): pairs (2i, 2i+1), i < dims/2, turned by position * base^(-2i/dims); the rest stays."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a), torch.sin(a)
        shape = (-1,) + (1,) * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_of(w, prefix, h, m, eps):
    """The cached part of a layer: normed latent c (tokens, kv_rank), rotated shared key (tokens, rot_dim)."""
    down = h @ w[prefix + "dkv"].T
    rank = m["kv_rank"]
    c = rms_norm(down[:, :rank], w[prefix + "dkv.norm"], eps)
    kr = rotate_interleaved(down[:, rank:], torch.arange(h.shape[0]), m["rot"]["base"], m["rot"]["dims"])
    return c, kr


def queries_of(w, prefix, h, m, eps, low_rank):
    if low_rank:
        q = rms_norm(h @ w[prefix + "dq"].T, w[prefix + "dq.norm"], eps) @ w[prefix + "uq"].T
    else:
        q = h @ w[prefix + "q"].T
    q = q.view(h.shape[0], m["heads"], m["dim"] + m["rot_dim"])
    q_plain, q_rot = q[..., :m["dim"]], q[..., m["dim"]:]
    return q_plain, rotate_interleaved(q_rot, torch.arange(h.shape[0]), m["rot"]["base"], m["rot"]["dims"])


def latent_attention(w, prefix, h, m, eps, low_rank, latent):
    """Causal attention whose keys and values are expanded from the latent, head by head and row by row."""
    c, kr = latent
    n = h.shape[0]
    q_plain, q_rot = queries_of(w, prefix, h, m, eps, low_rank)
    heads = []
    for hd in range(m["heads"]):
        k = c @ w[prefix + "uk"][hd * m["dim"]:(hd + 1) * m["dim"]].T
        v = c @ w[prefix + "uv"][hd * m["vdim"]:(hd + 1) * m["vdim"]].T
        rows = []
        for i in range(n):
            s = (k[:i + 1] @ q_plain[i, hd] + kr[:i + 1] @ q_rot[i, hd]) * m["scale"]
            p = torch.exp(s - s.max())
            rows.append((p / p.sum()) @ v[:i + 1])
        heads.append(torch.stack(rows))
    return torch.cat(heads, -1) @ w[prefix + "o"].T


def gated_expert(w, prefix, h, limit):
    g = torch.clamp(h @ w[prefix + "gate"].T, max=limit)
    u = torch.clamp(h @ w[prefix + "up"].T, min=-limit, max=limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w[prefix + "down"].T


def route_token(z, correction, top, groups, keep, scale):
    """Router logits of ONE token -> (expert ids in choice order, weights)."""
    s = 1 / (1 + torch.exp(-z))
    choice = (s + correction).tolist()
    n = len(choice)
    size = n // groups
    group_score = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -group_score[g])[:keep]
    open_ids = [e for e in range(n) if e // size in kept]
    ids = sorted(open_ids, key=lambda e: -choice[e])[:top]
    return ids, [float(s[e]) * scale for e in ids]


def mixture(w, prefix, h, mlp):
    r = mlp["router"]
    z = h @ w[prefix + "router"].T
    rows = []
    for t in range(h.shape[0]):
        ids, weights = route_token(z[t], w[prefix + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])
        y = gated_expert(w, prefix + "shared.", h[t], mlp["shared"]["limit"])
        for e, wt in zip(ids, weights):
            y = y + wt * gated_expert(w, f"{prefix}e{e}.", h[t], mlp["expert"]["limit"])
        rows.append(y)
    return torch.stack(rows)


def forward(cfg, w, tokens, layers_out=None):
    """tokens: list of ids -> logits (tokens, vocab).  cfg: the parsed config.json; w: name -> tensor."""
    eps = cfg["norm"]["eps"]
    x = layer_norm(w["embed"][torch.tensor(tokens)], w["embed.norm"], eps)
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, w[p + "norm1"], eps)
        src = m.get("kv_from")
        latents[i] = latents[src] if src is not None else latent_of(w, p + "mix.", h, m, eps)
        y = latent_attention(w, p + "mix.", h, m, eps, layer["type"] == "latent_attention_2", latents[i])
        if layer["mlp"] is not None:
            y = y + mixture(w, p + "mlp.", layer_norm(x, w[p + "norm2"], eps), layer["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, w, tokens, n):
    """n greedy tokens, the whole sequence evaluated anew for each."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(torch.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(tokens):]


def random_weights(cfg, seed, dtype=torch.bfloat16):
    """Random weights of a configuration, name -> tensor; scaled so that activations stay near 1 and the
    router's choices, the clamps and the attention's scores all vary."""
    g = torch.Generator().manual_seed(seed)
    width, w = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = (gain * torch.randn(rows, cols, generator=g) / math.sqrt(cols)).to(dtype)

    def vec(name, n, center=1.0, spread=0.1):
        w[name] = (center + spread * torch.randn(n, generator=g)).to(dtype)

    mat("embed", cfg["vocab"], width, math.sqrt(width))
    vec("embed.norm", width)
    vec("final.norm", width)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        qk = m["heads"] * (m["dim"] + m["rot_dim"])
        vec(p + "norm1", width)
        if layer["type"] == "latent_attention_2":
            mat(p + "mix.dq", m["q_rank"], width)
            vec(p + "mix.dq.norm", m["q_rank"])
            mat(p + "mix.uq", qk, m["q_rank"], 1.5)
        else:
            mat(p + "mix.q", qk, width, 1.5)
        if m.get("kv_from") is None:
            mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], width)
            vec(p + "mix.dkv.norm", m["kv_rank"])
        mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"])
        mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "mix.o", width, m["heads"] * m["vdim"])
        mlp = layer["mlp"]
        if mlp is None:
            continue
        vec(p + "norm2", width)
        mat(p + "mlp.router", mlp["router"]["experts"], width)
        vec(p + "mlp.correction", mlp["router"]["experts"], 0.0, 0.3)
        forms = [(f"e{e}", mlp["expert"]) for e in range(mlp["router"]["experts"])] + [("shared", mlp["shared"])]
        for name, form in forms:
            mat(f"{p}mlp.{name}.gate", form["ff"], width)
            mat(f"{p}mlp.{name}.up", form["ff"], width)
            mat(f"{p}mlp.{name}.down", width, form["ff"])
    return w
