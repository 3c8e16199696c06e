"""Dubarax without a GPU: its configuration and errors, the model as data (tensor names against the plain implementation's
table, the order of layer runs, what every run keeps per request), page groups of chunks, the learned distance table's
rows, and the chunk rule with row decays against the recurrence."""
import copy
import math
import random

import pytest
import torch

import plain_dubarax as pd
import plain_host as ph
from nano_vllm_cpp_b200.cache import CacheManager, DeviceCache
from nano_vllm_cpp_b200.config import ConfigError, get_architecture
from nano_vllm_cpp_b200.models.dubarax import linear_slopes
from nano_vllm_cpp_b200.parts import Model, CompositeCacheSpec, KVCacheSpec, StateCacheSpec
from nano_vllm_cpp_b200.parts.attention import distance_buckets
from nano_vllm_cpp_b200.parts.base import BranchSum

CFG = pd.model_config(
    [pd.window_layer(heads=4, kv_heads=2, dim=32, vdim=48, size=24, rows=10, mlp=pd.moe(8, 2, 24, 4, 2, 40)),
     pd.parallel_layer(pd.chunk_part(6, 3, 16, 24, size=20), pd.lightning_part(3, 24, 40, [0.5, 0.9, 1.0]), mlp=pd.moe(6, 3, 16, 2, 1, 0)),
     pd.mamba_layer(heads=6, vdim=8, state=20, groups=3, conv=3, norm_groups=4, mlp=None),
     pd.window_layer(heads=2, kv_heads=1, dim=40, size=9, rows=7, type="attention_2")],
    width=96, vocab=210, embed_scale=3.0, loop=(1, 3, 3))


def build(cfg):
    arch = get_architecture("Dubarax")
    typed = arch.config_from_dict(cfg)
    return typed, Model(arch.build_model(typed))


def test_tensor_names_and_shapes_are_the_plain_table():
    _, model = build(CFG)
    table = pd.tensor_table(CFG)
    for specs in (model.tensor_specs(), model.tensor_specs(lambda n: n in table)):
        assert set(specs) == set(table)
        for name, (shape, _) in table.items():
            want = tuple(specs[name].shape)
            if name.endswith(".rel"):          # the number of rows is the file's
                want, shape = want[1:], shape[1:]
            assert want == tuple(shape), name
    assert model.tensor_specs(lambda n: n in table)["l0.mix.rel"].shape[0] is None
    assert "l2.norm2" not in table and "l1.mlp.shared.up" not in table


def test_the_order_of_layer_runs_and_what_each_keeps():
    typed, model = build(CFG)
    assert (typed.eps, typed.embed_scale, typed.num_hidden_layers) == (1e-5, 3.0, 4)
    assert [(c.layer, c.pass_index) for c in model.calls] == pd.layer_runs(CFG)
    assert [(c.layer, c.pass_index) for c in model.calls] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    first, last = KVCacheSpec(2, 32, 24, 48), KVCacheSpec(1, 40, 9)
    both = CompositeCacheSpec((KVCacheSpec(3, 16, 0, 24, chunk=20), StateCacheSpec((3, 24, 40))))
    memory = CompositeCacheSpec((StateCacheSpec((6, 20, 8)), StateCacheSpec((2, 48 + 2 * 60))))
    assert model.cache_specs() == [first, both, memory, both, memory, both, memory, last]
    cache = DeviceCache(model.cache_specs(), 16, 2, "cpu", torch.float32)
    assert cache.windows == [24, ("chunk", 20), 9]
    cache.allocate(5)
    views = [cache.view(i).parts[0].k for i in (1, 3, 5)]
    assert len({v.data_ptr() for v in views}) == 3            # every pass has pages of its own in the same group
    assert cache.view(1).parts[0].group == cache.view(5).parts[0].group == 1
    assert len({cache.view(i).parts[1].state.data_ptr() for i in (1, 2, 3, 4, 5, 6)}) == 6
    # without a loop every layer runs once; a loop over everything opens its passes at layer 0
    flat = copy.deepcopy(CFG)
    del flat["loop"]
    assert [(c.layer, c.pass_index) for c in build(flat)[1].calls] == [(i, None) for i in range(4)] and build(flat)[1].pass_input is None
    flat["loop"] = {"start": 0, "stop": 4, "times": 2}
    assert [c.pass_index for c in build(flat)[1].calls] == [0, None, None, None, 1, None, None, None]
    flat["loop"] = {"start": 3, "stop": 4, "times": 1}
    assert [c.pass_index for c in build(flat)[1].calls] == [None, None, None, 0]


def test_parts_a_file_leaves_out_are_switched_off():
    d = copy.deepcopy(CFG)
    del d["loop"], d["embedding"], d["layers"][0]["mixer"]["softcap"], d["layers"][0]["mlp"]["router"]["groups"], d["layers"][0]["mlp"]["shared"]
    typed, model = build(d)
    assert typed.loop is None and typed.embed_scale == 1.0
    ff = model.layers[0].feed_forward
    assert model.layers[0].mixer.softcap == 0.0 and ff.groups is None and ff.shared_inter == 0
    assert model.layers[2].feed_forward is None and model.layers[2].norm2 is None
    assert not any(n.startswith("loop.") or ".shared." in n for n in model.tensor_specs())


def test_configuration_errors_name_the_key():
    arch = get_architecture("Dubarax")
    for path, value, drop, word in [
            (("layers", 0, "mixer", "heads"), 5, False, "kv_heads"),
            (("layers", 0, "mixer", "scale"), None, True, "scale"),
            (("layers", 0, "mixer", "mask"), None, True, "mask"),
            (("layers", 0, "mixer", "mask", "size"), 0, False, "mask.size"),
            (("layers", 0, "mixer", "bias_max"), None, True, "bias_max"),
            (("layers", 0, "mixer", "softcap"), -1.0, False, "softcap"),
            (("layers", 1, "mixer", "left"), None, True, "left"),
            (("layers", 1, "mixer", "left_scale"), None, True, "left_scale"),
            (("layers", 1, "mixer", "right", "decay"), [0.5, 0.9], False, "decay"),
            (("layers", 1, "mixer", "right", "decay"), None, True, "decay"),
            (("layers", 2, "mixer", "groups"), 4, False, "groups"),
            (("layers", 2, "mixer", "norm_groups"), 5, False, "norm_groups"),
            (("layers", 2, "mixer", "state"), None, True, "state"),
            (("layers", 0, "mlp", "router", "top"), 9, False, "router.top"),
            (("layers", 0, "mlp", "router", "top"), 5, False, "groups.keep"),
            (("layers", 0, "mlp", "router", "groups", "count"), 3, False, "groups.count"),
            (("layers", 0, "mlp", "router", "groups", "keep"), 5, False, "groups.keep"),
            (("layers", 0, "mlp", "kind"), "dense", False, "mlp.kind"),
            (("layers", 1, "type"), "conv", False, "type"),
            (("loop", "stop"), 5, False, "loop.stop"),
            (("loop", "start"), 3, False, "loop.start"),
            (("loop", "times"), 0, False, "loop.times"),
            (("norm",), None, True, "norm"),
            (("width",), None, True, "width")]:
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


def test_slopes_and_rows_of_the_distance_table():
    for H in (1, 2, 6, 8, 20):
        assert linear_slopes(H) == pd.linear_bias(H)
    for rows, far in ((12, 40), (16, 128), (32, 128), (7, 20), (2, 9), (9, 5), (64, 4096)):
        b = distance_buckets(rows, far)
        assert b[:rows // 2] == list(range(rows // 2)) and b[-1] == rows - 1 and b == sorted(b)
        for n in range(2 * far + 5):
            assert b[min(n, len(b) - 1)] == pd.bucket_of(n, rows, far), (rows, far, n)
    assert distance_buckets(1, 10) == [0] and distance_buckets(8, 3)[-1] == 7


def test_pages_of_chunks_are_given_back_when_the_chunk_has_passed():
    """Chunks of 40 positions on pages of 16: a page goes back once the next row lies in a later chunk than all of it; a page
    that two chunks share stays for the second."""
    m = CacheManager([("chunk", 40), 0], [6, 20], 16, max_requests=2)
    m.open("a")
    at = 0
    for n in (38, 1, 1, 1, 20, 30, 25):
        m.extend("a", at, at + n)
        at += n
        m.commit("a", at)
        start = at // 40 * 40
        chunk, whole = m.get("a").tables
        last_run = at - n                      # pages are given back when the rows are about to run
        gone = last_run // 40 * 40 // 16
        assert all(p == -1 for p in chunk[:gone]) and all(p >= 0 for p in chunk[gone:]), (at, chunk)
        assert all(p >= 0 for p in whole)
        m.check()
    assert at == 116 and not m.prefix_caching
    assert not CacheManager([("chunk", 64)], 4, 16, max_requests=1, prefix_caching=True).prefix_caching


def test_the_native_manager_and_its_plain_twin_agree_on_chunks():
    rng = random.Random(5)
    for case in range(60):
        windows = rng.choice([[("chunk", 24)], [0, ("chunk", 33)], [("chunk", 16), 12], [("chunk", 7), ("chunk", 50), (20, 3)]])
        pages = rng.choice([5, 8, 14])
        a = CacheManager(windows, pages, 16, max_requests=3)
        b = ph.CacheManager(windows, pages, 16, max_requests=3)
        at = {}
        for _ in range(60):
            rid = rng.randrange(4)
            if rid not in at:
                if len(at) == 3:
                    continue
                a.open(rid), b.open(rid)
                at[rid] = 0
            elif rng.random() < 0.1:
                a.close(rid), b.close(rid)
                del at[rid]
                continue
            n = rng.choice([1, 1, 2, 5, 17, 40])
            assert a.pages_needed(rid, at[rid], at[rid] + n) == b.pages_needed(rid, at[rid], at[rid] + n)
            can = a.can_extend(rid, at[rid], at[rid] + n)
            assert can == b.can_extend(rid, at[rid], at[rid] + n)
            if can:
                a.extend(rid, at[rid], at[rid] + n), b.extend(rid, at[rid], at[rid] + n)
                at[rid] += n
                a.commit(rid, at[rid]), b.commit(rid, at[rid])
            assert a.get(rid).tables == b.get(rid).tables if can else True
            a.check()


def test_a_scaled_sum_of_branches():
    a, b = torch.randn(3, 5, dtype=torch.float64), torch.randn(3, 5, dtype=torch.float64)
    assert torch.allclose(BranchSum(a.clone(), b, 0.7, -1.3).sum(), 0.7 * a - 1.3 * b, rtol=0, atol=1e-15)
    assert torch.equal(BranchSum(a.clone(), b).sum(), a + b)


def test_the_plain_chunk_rule_with_row_decays_is_the_recurrence():
    """The rule that the chunked kernels follow when every row has a decay of its own, with running sums of logarithms,
    written out in float64, against the row-by-row recurrence."""
    g = torch.Generator().manual_seed(4)
    T, D, V, C = 37, 6, 5, 8
    q, k, v = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    dt = torch.rand(T, generator=g, dtype=torch.float64) * 2
    log = -0.7 * dt
    S, want = torch.zeros(D, V, dtype=torch.float64), []
    for t in range(T):
        S = math.exp(log[t]) * S + dt[t] * torch.outer(k[t], v[t])
        want.append(S.T @ q[t])
    S2, got = torch.zeros(D, V, dtype=torch.float64), []
    for c in range(0, T, C):
        n = min(C, T - c)
        L = torch.cumsum(log[c:c + n], 0)
        for i in range(n):
            o = torch.exp(L[i]) * (S2.T @ q[c + i])
            for j in range(i + 1):
                o = o + torch.exp(L[i] - L[j]) * dt[c + j] * float(q[c + i] @ k[c + j]) * v[c + j]
            got.append(o)
        S2 = torch.exp(L[-1]) * S2 + sum(torch.exp(L[-1] - L[j]) * dt[c + j] * torch.outer(k[c + j], v[c + j]) for j in range(n))
    assert torch.allclose(torch.stack(got), torch.stack(want), rtol=0, atol=1e-12) and torch.allclose(S, S2, rtol=0, atol=1e-12)


def test_the_plain_routing_keeps_the_best_groups():
    s = [0.1, 0.3, 0.02, 0.05, 0.25, 0.01, 0.2, 0.07]
    r = {"experts": 8, "top": 3, "groups": {"count": 4, "keep": 2}}
    assert pd.route(s, r) == [(1, 0.3), (4, 0.25), (0, 0.1)]          # groups {0, 1} and {4, 5}: expert 6 is out
    assert [e for e, _ in pd.route(s, dict(r, groups={"count": 4, "keep": 4}))] == [1, 4, 6]
    assert [e for e, _ in pd.route(s, dict(r, groups=None))] == [1, 4, 6]
    assert [e for e, _ in pd.route([0.25] * 4, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})] == [0, 1]
