"""Configurations of the Rigozen tests.  Sizes differ from layer to layer and are awkward on purpose in `odd`, which also
has windows of one and a few tokens, convolutions of one and three taps and layers that share weights; `fast` has the
sizes the tensor-core kernels take, and `tiles` some that end inside their tiles."""


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def latent(heads, dim, vdim, kv_rank, scale, window):
    return "latent_attention", dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=scale, mask=dict(size=window))


def attention(heads, kv_heads, dim, scale, window):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=dict(size=window))


def config(vocab, width, eps, layers):
    """layers: (mixer, ff or None), or the number of an earlier layer whose weights are used."""
    entries = []
    for layer in layers:
        if isinstance(layer, int):
            entries.append(dict(entries[layer], weights_of=layer))
        else:
            (kind, mixer), ff = layer
            entries.append(dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None))
    return dict(architecture="Rigozen", vocab=vocab, width=width, norm=dict(eps=eps), layers=entries)


def odd():
    return config(211, 76, 1e-4, [
        (delta(6, 2, 20, 12, 3), 44),
        (attention(6, 3, 20, 0.3, 17), 52),
        (latent(3, 20, 28, 44, 0.21, 5), None),
        0,
        2,
        (delta(3, 3, 33, 7, 1), 12),
        (attention(2, 2, 9, 0.5, 1), 20),
        1,
    ])


def tiles():
    return config(300, 200, 1e-6, [
        (latent(5, 24, 40, 136, 0.2, 70), 72),
        (delta(4, 1, 72, 136, 4), 136),
        (attention(12, 2, 40, 0.16, 65), 72),
        (delta(2, 2, 136, 40, 5), None),
        0,
    ])


def fast():
    return config(512, 384, 1e-5, [
        (delta(8, 4, 128, 128, 4), 512),
        (latent(16, 128, 128, 512, 0.09, 200), 320),
        (attention(32, 4, 128, 0.09, 129), 512),
        0,
        (latent(40, 64, 64, 256, 0.12, 333), 192),
        (delta(6, 2, 64, 96, 2), 256),
        (attention(10, 1, 56, 0.14, 64), 192),
    ])


def recurrent():
    """No attention at all: nothing grows with the sequence."""
    return config(97, 64, 1e-5, [(delta(2, 1, 16, 32, 4), 48), 0])
