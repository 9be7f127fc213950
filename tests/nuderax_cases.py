"""Configurations of the Nuderax tests.  Sizes differ from layer to layer and
are awkward on purpose in `odd`; `fast` has the sizes the tensor-core kernels take, and `tiles` some that end
inside their tiles."""

def _mixer(low_rank_q, heads, dim, rot_dim, rot_dims, vdim, kv_rank, scale, base, q_rank=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dims))
    if low_rank_q:
        m["q_rank"] = q_rank
    if kv_from is not None:
        m["kv_from"] = kv_from
    return ("latent_attention_2" if low_rank_q else "latent_attention"), m


def _moe(experts, top, count, keep, scale, ff, limit, shared_ff, shared_limit):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), shared=dict(ff=shared_ff, limit=shared_limit),
                router=dict(experts=experts, top=top, scale=scale, groups=dict(count=count, keep=keep)))


def _config(vocab, width, eps, layers):
    return dict(architecture="Nuderax", vocab=vocab, width=width, norm=dict(eps=eps),
                layers=[dict(type=t, mixer=m, mlp=mlp) for (t, m), mlp in layers])


def odd():
    moe = _moe(6, 3, 3, 2, 1.7, 44, 0.9, 36, 1.3)
    return _config(211, 76, 1e-4, [
        (_mixer(True, 3, 20, 12, 8, 28, 44, 0.21, 500.0, q_rank=36), moe),
        (_mixer(False, 5, 12, 8, 8, 20, 60, 0.3, 9000.0), _moe(5, 1, 1, 1, 2.5, 20, 2.0, 52, 0.4)),
        (_mixer(False, 2, 28, 8, 8, 12, 60, 0.17, 9000.0, kv_from=1), None),
        (_mixer(False, 1, 16, 12, 8, 16, 44, 0.4, 500.0, kv_from=0), _moe(4, 4, 4, 4, 0.6, 12, 0.5, 8, 3.0)),
    ])


def tiles():
    moe = _moe(12, 3, 4, 2, 1.2, 72, 1.1, 136, 1.6)
    return _config(300, 200, 1e-6, [
        (_mixer(False, 5, 24, 16, 16, 40, 136, 0.16, 3000.0), moe),
        (_mixer(True, 3, 64, 32, 24, 72, 64, 0.11, 700.0, q_rank=88), moe),
        (_mixer(False, 4, 40, 16, 16, 24, 136, 0.14, 3000.0, kv_from=0), moe),
    ])


def fast():
    moe = _moe(16, 4, 4, 2, 1.4, 192, 1.2, 320, 1.5)
    return _config(512, 384, 1e-5, [
        (_mixer(False, 16, 128, 64, 64, 128, 512, 0.06, 10000.0), moe),
        (_mixer(True, 32, 64, 64, 64, 64, 256, 0.08, 40000.0, q_rank=192), moe),
        (_mixer(False, 20, 128, 64, 64, 128, 512, 0.07, 10000.0, kv_from=0), moe),
    ])
