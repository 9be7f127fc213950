"""What of the Rigozen models needs no GPU: configuration, state of slots, and the plain evaluation against itself."""
import copy

import pytest
import torch

import plain_rigozen as plain
import rigozen_cases as cases


@pytest.mark.parametrize("make", [cases.odd, cases.tiles, cases.fast, cases.recurrent])
def test_registry_and_tensor_names(make):
    from axono_b200 import models
    from axono_b200.models.rigozen import tensor_shapes

    assert "Rigozen" in models.architectures() and "Nuderax" in models.architectures()
    cfg = make()
    shapes = dict(tensor_shapes(models.config_of(cfg)))
    assert shapes == {k: tuple(v.shape) for k, v in plain.random_weights(cfg, 0).items()}


def test_configuration_is_read_from_the_entries():
    from axono_b200 import models

    cfg = cases.odd()
    odd = models.config_of(cfg)
    assert [layer.weights_of for layer in odd.layers] == [0, 1, 2, 0, 2, 5, 6, 1]
    assert odd.layers[2].ff is None and odd.layers[1].ff == 52 and odd.eps == 1e-4
    assert odd.layers[1].mixer.window == 17 and odd.layers[2].mixer.window == 5 and odd.layers[6].mixer.window == 1
    assert odd.layers[5].mixer.conv == 1 and odd.layers[1].mixer.scale == 0.3
    # a chain of layers that share, and a source that comes later
    cfg["layers"][7]["weights_of"], cfg["layers"][1]["weights_of"] = 1, 7
    with pytest.raises(ValueError):
        models.config_of(cfg)
    del cfg["layers"][7]["weights_of"]
    assert [layer.weights_of for layer in models.config_of(cfg).layers] == [0, 7, 2, 0, 2, 5, 6, 7]


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="convolution"),
    lambda c: c["layers"][0]["mixer"].update(heads=7),               # no multiple of kv_heads
    lambda c: c["layers"][1]["mixer"].update(vdim=24),               # values are keys
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][5]["mixer"].update(conv=0),
    lambda c: c["layers"][5]["mixer"].update(dim=300),
    lambda c: c["layers"][3].update(weights_of=8),
    lambda c: c["layers"][3].update(weights_of=1),                   # another kind of layer
    lambda c: c["layers"][3].update(weights_of=3),                   # itself
    lambda c: c["layers"][0].update(mlp=dict(kind="moe", ff=8)),
])
def test_configurations_that_make_no_sense_are_refused(change):
    from axono_b200 import models

    cfg = copy.deepcopy(cases.odd())
    change(cfg)
    with pytest.raises(ValueError):
        models.config_of(cfg)


def test_arena_with_state_and_without_rows():
    from axono_b200.kv_cache import KVArena

    a = KVArena.of_rows([40], num_pages=3, max_seqs=2, max_seq_len=128, device_memory=False)
    assert a.add_state((3, 5, 7), torch.float32) is None and a.stats()["device_bytes"] == 0
    a.close()
    a = KVArena.of_rows([], num_pages=3, max_seqs=2, max_seq_len=128, device_memory=False)
    a.add_state((2, 4), torch.bfloat16)
    s = a.alloc_seq(100)
    assert len(a.seq_pages(s)) == 2
    with pytest.raises(RuntimeError):
        a.reserve(s, 300)
    a.free_seq(s)
    assert a.stats()["pages_free"] == 3
    a.close()


def test_a_design_names_the_sources_it_needs():
    import os

    from axono_b200 import build, models

    for design in models.architectures():
        for name in (*build.SERVING_SOURCES, *models.model_class(design).kernel_sources):
            assert os.path.exists(os.path.join(build.CSRC, name)), name
        assert design.lower() in build.serving_lib(design)


# ---- the plain evaluation itself ---------------------------------------------------------------------------
def test_plain_windows_end_exactly():
    """With window n a row's output depends on the key n - 1 before it and not on the one before that."""
    q, k, v = (torch.randn(9, 4, dtype=torch.float64) for _ in range(3))
    for window in (1, 2, 5):
        base = plain.attend_row(q, k, v, 8, 0.5, window)
        for j in range(9):
            k2 = k.clone()
            k2[j] += 3
            assert torch.equal(plain.attend_row(q, k2, v, 8, 0.5, window), base) == (8 - j >= window or window == 1)
        v2 = v.clone()
        v2[8 - window + 1] += 1
        assert not torch.equal(plain.attend_row(q, k, v2, 8, 0.5, window), base)


def test_plain_sink_joins_the_denominator_once():
    q, k, v = (torch.randn(6, 4, dtype=torch.float64) for _ in range(3))
    s = (k @ q[5]) * 0.7
    sink = torch.tensor(1.3, dtype=torch.float64)
    want = (torch.exp(s) @ v) / (torch.exp(s).sum() + torch.exp(sink))
    assert torch.allclose(plain.attend_row(q, k, v, 5, 0.7, 0, sink), want)
    assert torch.allclose(plain.attend_row(q, k, v, 5, 0.7, 0, torch.tensor(-1e9, dtype=torch.float64)), plain.attend_row(q, k, v, 5, 0.7, 0))


def test_plain_convolution_and_rule():
    x = torch.arange(1.0, 5.0, dtype=torch.float64)[:, None]
    w = torch.tensor([[0.5, 2.0, 3.0]], dtype=torch.float64)  # oldest tap first
    want = torch.tensor([[3.0], [2 + 6.0], [0.5 + 4 + 9], [1 + 6 + 12]], dtype=torch.float64)
    assert torch.allclose(plain.causal_conv(x, w), plain.silu(want))
    # beta 1 and a unit key: the value written is read back exactly, whatever the state held
    k = torch.tensor([[0.6, 0.8]], dtype=torch.float64)
    v = torch.tensor([[2.0, -1.0, 5.0]], dtype=torch.float64)
    one = torch.ones(1, dtype=torch.float64)
    o, _ = plain.delta_rule(k, k, v, 0.3 * one, one, torch.randn(2, 3, dtype=torch.float64))
    assert torch.allclose(o, v)
    # beta 0 only decays
    _, s = plain.delta_rule(k, k, v, 0.5 * one, 0 * one, torch.ones(2, 3, dtype=torch.float64))
    assert torch.allclose(s, 0.5 * torch.ones(2, 3, dtype=torch.float64))


def test_plain_model_shares_weights_but_not_layers():
    cfg = cases.recurrent()
    w = {k: v.double() for k, v in plain.random_weights(cfg, 3).items()}
    copied = dict(w, **{"l1" + k[2:]: v for k, v in w.items() if k.startswith("l0.")})
    apart = dict(cfg, layers=[cfg["layers"][0], dict(cfg["layers"][0])])
    assert torch.equal(plain.forward(cfg, w, [5, 6, 7]), plain.forward(apart, copied, [5, 6, 7]))
    assert not torch.allclose(plain.forward(cfg, w, [5, 6, 7]), plain.forward(dict(cfg, layers=cfg["layers"][:1]), w, [5, 6, 7]))
