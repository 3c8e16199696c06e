"""Sevelorn without a GPU: its configuration and errors, the model as data (tensor names against the plain
implementation's table, what every layer keeps per request, layers that read another's pages and keep a state of their
own), and the cache's views of such layers."""
import copy

import pytest
import torch

import plain_sevelorn as ps
from nano_vllm_cpp_b200.cache import DeviceCache
from nano_vllm_cpp_b200.config import ConfigError, get_architecture
from nano_vllm_cpp_b200.parts import Model, CompositeCacheSpec, KVCacheSpec, SharedCacheSpec, StateCacheSpec

CFG = ps.model_config(
    [ps.attention_layer(heads=4, kv_heads=2, dim=32, vdim=48, mlp=ps.moe(6, 2, 24)),
     ps.retention_layer(heads=3, dim=32, vdim=40, rot_dims=20, decay=[0.5, 0.9, 0.995], mlp=ps.dense(72)),
     ps.attention_layer(heads=6, kv_heads=2, dim=32, vdim=48, kv_from=0, mlp=ps.dense(40)),
     ps.retention_layer(heads=2, dim=48, vdim=16, rot_dims=0, decay=[0.98, 0.75], mlp=None, type="retention_2")],
    width=96, vocab=210, streams=3, taps=4, embed_scale=3.0)


def build(cfg):
    arch = get_architecture("Sevelorn")
    typed = arch.config_from_dict(cfg)
    return typed, Model(arch.build_model(typed))


def test_tensor_names_and_shapes_are_the_plain_table():
    _, model = build(CFG)
    specs, table = model.tensor_specs(), ps.tensor_table(CFG)
    assert set(specs) == set(table)
    for name, (shape, _) in table.items():
        assert tuple(specs[name].shape) == tuple(shape), name
    assert "l2.mix.k" not in specs and "l2.mix.k.norm" not in specs and tuple(specs["l2.mix.q.norm"].shape) == (6 * 32,)
    assert "l3.norm2" not in specs and "l3.hc2.in" not in specs


def test_what_every_layer_keeps_per_request():
    typed, model = build(CFG)
    assert (typed.streams, typed.taps, typed.embed_scale, typed.num_hidden_layers) == (3, 4, 3.0, 4)
    tail = StateCacheSpec((3, 96))
    assert model.cache_specs() == [
        CompositeCacheSpec((KVCacheSpec(2, 32, 0, 48), tail)), CompositeCacheSpec((StateCacheSpec((3, 32, 40)), tail)),
        CompositeCacheSpec((SharedCacheSpec(0, 0), tail)), CompositeCacheSpec((StateCacheSpec((2, 48, 16)), tail))]
    assert model.layers[3].feed_forward is None and [c.cache_of for c in model.calls] == [None, None, 0, None]
    # with one tap the convolution keeps nothing, and a layer that borrows keeps nothing at all
    one = copy.deepcopy(CFG)
    one["canon"]["taps"] = 1
    specs = build(one)[1].cache_specs()
    assert specs == [KVCacheSpec(2, 32, 0, 48), StateCacheSpec((3, 32, 40)), ("shared", 0), StateCacheSpec((2, 48, 16))]


def test_views_of_a_layer_that_borrows_pages_and_keeps_a_state():
    _, model = build(CFG)
    cache = DeviceCache(model.cache_specs(), 16, 3, "cpu", torch.float32)
    assert cache.windows == [0]
    assert cache.bytes_per_page() == [2 * 16 * (32 + 48) * 4]            # one layer's pages: the reader takes none
    cache.allocate(5)
    owner, reader = cache.view(0), cache.view(2)
    assert reader.parts[0].k.data_ptr() == owner.parts[0].k.data_ptr() and owner.parts[0].write and not reader.parts[0].write
    assert reader.parts[1].state.shape == (3, 3, 96) and reader.parts[1].write
    assert reader.parts[1].state.data_ptr() != owner.parts[1].state.data_ptr()
    # every state is a slice of one buffer, so that one launch zeroes a request's whole state
    n = 4 * 3 * 96 + 3 * 32 * 40 + 2 * 48 * 16
    assert cache.state_buffers[torch.float32].shape == (3, n)
    assert cache.has_state


def test_configuration_errors_name_the_key():
    arch = get_architecture("Sevelorn")
    for path, value, drop, word in [
            (("layers", 0, "mixer", "heads"), 5, False, "kv_heads"),
            (("layers", 0, "mixer", "scale"), None, True, "scale"),
            (("layers", 1, "mixer", "decay"), [0.5, 0.9], False, "decay"),
            (("layers", 1, "mixer", "decay"), None, True, "decay"),
            (("layers", 1, "mixer", "rot", "dims"), 34, False, "rot.dims"),
            (("layers", 1, "mixer", "rot", "dims"), 7, False, "rot.dims"),
            (("layers", 2, "mixer", "kv_from"), 1, False, "kv_from"),
            (("layers", 2, "mixer", "kv_from"), 2, False, "kv_from"),
            (("layers", 2, "mixer", "kv_from"), -1, False, "kv_from"),
            (("layers", 2, "mixer", "dim"), 16, False, "kv_from"),
            (("layers", 0, "mlp", "router", "top"), 7, False, "router.top"),
            (("layers", 0, "mlp", "kind"), "sparse", False, "mlp.kind"),
            (("layers", 1, "type"), "conv", False, "type"),
            (("canon", "taps"), 0, False, "canon.taps"),
            (("norm",), None, True, "norm"),
            (("width",), None, True, "width"),
            (("streams",), 0, False, "streams")]:
        d = copy.deepcopy(CFG)
        node = d
        for k in path[:-1]:
            node = node[k]
        if drop:
            del node[path[-1]]
        else:
            node[path[-1]] = value
        with pytest.raises(ConfigError) as e:
            arch.config_from_dict(d)
        assert word in str(e.value), (path, str(e.value))


def test_parts_a_file_leaves_out_are_switched_off():
    d = copy.deepcopy(CFG)
    del d["streams"], d["canon"], d["embedding"]
    typed, model = build(d)
    assert (typed.streams, typed.taps, typed.embed_scale) == (1, 0, 1.0)
    assert model.layers[0].input_filter is None and "l0.canon1" not in model.tensor_specs()
    assert model.layers[3].mixer.position.rotary_dim == 0 and model.layers[1].mixer.position.rotary_dim == 20
    assert model.cache_specs()[2] == ("shared", 0)


def test_the_plain_chunk_rule_is_the_recurrence():
    """The rule that the chunked kernels follow, written out in float64, against the row-by-row recurrence."""
    g = torch.Generator().manual_seed(4)
    T, D, V, d, C = 37, 6, 5, 0.93, 8
    q, k, v = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    S, want = torch.zeros(D, V, dtype=torch.float64), []
    for t in range(T):
        S = d * S + torch.outer(k[t], v[t])
        want.append(S.T @ q[t])
    S2, got = torch.zeros(D, V, dtype=torch.float64), []
    for c in range(0, T, C):
        n = min(C, T - c)
        for i in range(n):
            o = d ** (i + 1) * (S2.T @ q[c + i])
            for j in range(i + 1):
                o = o + d ** (i - j) * float(q[c + i] @ k[c + j]) * v[c + j]
            got.append(o)
        S2 = d ** n * S2 + sum(d ** (n - 1 - j) * torch.outer(k[c + j], v[c + j]) for j in range(n))
    assert torch.allclose(torch.stack(got), torch.stack(want), rtol=0, atol=1e-12) and torch.allclose(S, S2, rtol=0, atol=1e-12)
