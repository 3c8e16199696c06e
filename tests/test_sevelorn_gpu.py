"""The Sevelorn decoder and its mechanisms against the plain implementation (tests/plain_sevelorn.py): every part alone,
then whole models through the engine's step function, cache manager and scheduler, for every way of cutting the work into
steps.  The configurations are small and of this file's own making; weights are random, and where random weights would
hide a fault (a far key, a far token in a decaying state, a tap) they are shaped so that it shows."""
import json
import math
import random

import pytest
import torch

import plain_sevelorn as ps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

CONFIGS = {
    # both mixers with two sets of sizes, values wider and narrower than keys, part of a retention head turned and
    # nothing turned, two layers that read another's keys and values (one of them with other query heads), a layer
    # without a feed-forward, both feed-forwards behind both mixers
    "M": ps.model_config(
        [ps.attention_layer(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.2, mlp=ps.moe(6, 2, 24)),
         ps.retention_layer(heads=3, dim=32, vdim=40, rot_dims=20, base=500.0, decay=[0.5, 0.9, 0.995], mlp=ps.dense(72)),
         ps.attention_layer(heads=6, kv_heads=2, dim=32, vdim=48, scale=0.15, kv_from=0, mlp=ps.dense(40)),
         ps.retention_layer(heads=2, dim=48, vdim=16, rot_dims=0, decay=[0.98, 0.75], mlp=None, type="retention_2"),
         ps.attention_layer(heads=3, kv_heads=3, dim=40, vdim=24, scale=0.11, mlp=ps.moe(5, 3, 20), type="attention_2"),
         ps.attention_layer(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.25, kv_from=0, mlp=None)],
        width=96, vocab=210, streams=3, taps=4, eps=1e-5, embed_scale=3.0),
    # sizes of one and values that other models make equal: one copy of the stream, one head everywhere, a convolution
    # of one tap, one expert, every expert chosen, a decay of one, no scale on the embedding
    "N": ps.model_config(
        [ps.retention_layer(heads=1, dim=16, vdim=16, rot_dims=2, base=20.0, decay=[1.0], mlp=ps.moe(1, 1, 16)),
         ps.attention_layer(heads=1, kv_heads=1, dim=24, vdim=8, scale=0.3, mlp=ps.moe(4, 4, 24)),
         ps.retention_layer(heads=2, dim=8, vdim=24, rot_dims=8, base=50.0, decay=[0.8, 0.95], mlp=ps.dense(48)),
         ps.attention_layer(heads=5, kv_heads=1, dim=24, vdim=8, scale=0.3, kv_from=None, mlp=None),
         ps.attention_layer(heads=1, kv_heads=1, dim=24, vdim=8, scale=0.4, kv_from=3, mlp=ps.dense(20))],
        width=64, vocab=130, streams=1, taps=1, embed_scale=1.0),
    # sizes that the tensor-core kernels take: heads of 64 and 128, experts of 64, a width of 128
    "R": ps.model_config(
        [ps.retention_layer(heads=2, dim=64, vdim=64, rot_dims=64, base=1e4, decay=[0.97, 0.999], mlp=ps.dense(256)),
         ps.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, mlp=ps.moe(8, 3, 64)),
         ps.retention_layer(heads=1, dim=128, vdim=128, rot_dims=64, base=1e5, decay=[0.99], mlp=ps.moe(8, 2, 64)),
         ps.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.2, kv_from=1, mlp=ps.moe(4, 1, 32))],
        width=128, vocab=344, streams=4, taps=3, eps=1e-6, embed_scale=8.0),
}
SEEDS = {"M": 3, "N": 5, "R": 7}
NAMES = ["M", "N", "R"]
TOL = {"float32": 1e-4, "bfloat16": 4e-2}
# A bfloat16 row may exceed the tolerance as far as the plain implementation says that roundings move it (NOISE_FACTOR
# times the worst of a few draws of noise of a bfloat16 rounding's size on everything a sublayer reads and gives).  It may
# also rightly choose another expert where the last chosen and the first left-out router logits are closer than EDGE, and
# then a few of the rows behind it, which read what it left in the cache and the states, may be off too.
NOISE, NOISE_FACTOR, EDGE, MAX_BEHIND = 2.0 ** -9, 4.0, 0.02, 0.25


def ids_for(name, n, salt=0):
    g = torch.Generator().manual_seed(1000 * ord(name) + 7 * n + salt)
    return [int(t) for t in torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g)]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        W = ps.make_weights(cfg, SEEDS[name])
        out[name] = (cfg, W, ps.write_folder(cfg, W, str(tmp_path_factory.mktemp("sevelorn_" + name))))
    return out


_plain = {}


def plain_logits(models, name, ids):
    """(logits, per row the smallest router margin of any layer)"""
    key = (name, tuple(ids))
    if key not in _plain:
        cfg, W, _ = models[name]
        margins = []
        lg = ps.forward(cfg, W, ids, margins=margins)
        _plain[key] = (lg, torch.stack(margins).min(dim=0).values if margins else torch.full((len(ids),), math.inf))
    return _plain[key]


_errors = {}


def rounding_errors(models, name, ids):
    key = (name, tuple(ids))
    if key not in _errors:
        _errors[key] = ps.rounding_errors(*models[name][:2], ids, NOISE)
    return _errors[key]


def close(got, want, rel, what, margins=None, errors=None):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    err = (got - want).abs().reshape(got.shape[0], -1).max(dim=1).values
    bound = rel * max(1e-3, float(want.abs().max()))
    bad = err > bound
    if errors is not None and bool(bad.any()):
        bad &= err > NOISE_FACTOR * (errors() if callable(errors) else errors)
    if margins is not None:
        edge = margins < EDGE
        if bool(edge.any()):
            first = int(torch.nonzero(edge)[0])
            behind = int((bad[first:] & ~edge[first:]).sum())
            assert behind <= max(3, MAX_BEHIND * (len(bad) - first)), f"{what}: {behind} rows behind the first edge row are off"
            bad[first:] = False
    assert not bool(torch.isnan(err).any()), f"{what}: not a number"
    if bool(bad.any()):
        row = int(torch.nonzero(bad)[0])
        raise AssertionError(f"{what}: error {float(err[row]):.3g} > {bound:.3g} at row {row} (first of {int(bad.sum())})")


def make_runner(folder, dtype, max_tokens, max_requests=4, **kw):
    from nano_vllm_cpp_b200.engine.runner import ModelRunner
    return ModelRunner(folder, dtype=dtype, max_tokens=max_tokens, max_requests=max_requests, **kw)


class Steps:
    """Feeds requests through ``ModelRunner.step`` and keeps the logits per (request, position)."""

    def __init__(self, runner):
        from nano_vllm_cpp_b200.engine.batch import StepEntry
        self.runner, self.StepEntry, self.fed, self.logits = runner, StepEntry, {}, {}

    def step(self, parts, end=()):
        entries = [self.StepEntry(rid, list(toks), list(range(len(toks)))) for rid, toks in parts]
        out = self.runner.step(entries).float().cpu()
        r = 0
        for e in entries:
            base = self.fed.get(e.rid, 0)
            for w in e.want:
                self.logits[(e.rid, base + w)] = out[r]
                r += 1
            self.fed[e.rid] = base + len(e.tokens)
        for rid in end:
            self.runner.close(rid)
            self.fed.pop(rid, None)
        self.runner.manager.check()

    def rows(self, rid, n):
        return torch.stack([self.logits[(rid, p)] for p in range(n)])


def check_rows(st, models, name, rid, ids, dtype, what):
    want, margins = plain_logits(models, name, ids)
    half = dtype == "bfloat16"
    close(st.rows(rid, len(ids)), want, TOL[dtype], what, margins if half else None,
          (lambda: rounding_errors(models, name, ids)) if half else None)


# ------------------------------------------------------------------------------- the parts alone
def ctx_for(dtype, fast=True):
    from nano_vllm_cpp_b200.csrc import ops
    from nano_vllm_cpp_b200.parts import RunContext
    return RunContext(device=torch.device(DEV), act_dtype=dtype, err=ops.ErrorFlag(DEV), page_size=16, fast_kernels=fast)


class Fetch:
    VECTORS = ("q.norm", "k.norm", "router.b", "canon1")

    def __init__(self, tensors, prefix, dtype):
        self.t, self.p, self.dtype = tensors, prefix, dtype

    def __call__(self, name):
        t = self.t[self.p + name]
        vector = t.dim() <= 1 or name in self.VECTORS
        return t.to(torch.float32 if vector else self.dtype).to(DEV)

    def has(self, name):
        return (self.p + name) in self.t


def rnd(seed, *shape):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def dev32(t):
    return t.float().to(DEV).contiguous()


def inputs(width, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(n, width, generator=g).to(torch.bfloat16).double() for n in lengths]


def weights_of(layer, width, seed, what="mix"):
    cfg = ps.model_config([layer], width=width, vocab=8)
    W = ps.make_weights(cfg, seed)
    return {k.replace(f"l0.{what}.", "m."): v for k, v in W.items() if k.startswith(f"l0.{what}.")}


@pytest.mark.parametrize("H", [64, 50, 256, 1100, 2500, 5001])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 7])
def test_copies_of_the_stream_under_an_rms_norm(S, H):
    """One launch brings the copies up to date, reads them and norms what it read: with a dense pending output, with a
    weighted sum of rows that has not been taken yet, with nothing pending, and the closing sum; rows longer than a
    block's first pass; only the float32 rows, only the rows in bfloat16."""
    from nano_vllm_cpp_b200.csrc import ops
    T, R, P, eps = 9, 5, 23, 1e-3
    X, y = rnd(7 * S + H, T, S, H), rnd(8 * S + H, T, H)
    M = torch.eye(S, dtype=F64) + 0.3 * rnd(1 + S, S, S)
    w, r, gain = rnd(2 + S, S), rnd(3 + S, S), 1 + 0.2 * rnd(4 + H, H)
    norm = ("rms", dev32(gain), eps)
    rms = lambda u: ps.unit_rms(u, eps) * gain
    x = dev32(X.reshape(T, S * H))
    out, out32 = torch.empty(T, H, dtype=torch.bfloat16, device=DEV), torch.empty(T, H, dtype=torch.float32, device=DEV)
    ops.stream_mix_norm(x, S, branch=dev32(y), carry=dev32(M), write=dev32(w), read=dev32(r), norm=norm, out=out, out32=out32)
    Xn = torch.einsum("cd,tcw->tdw", M, X) + w[None, :, None] * y[:, None, :]
    u = torch.einsum("c,tcw->tw", r, Xn)
    close(x.view(T, S, H), Xn, 1e-6, "copies after a dense output")
    close(out32, rms(u), 1e-5, "normed rows")
    close(out, rms(u), 2 ** -7, "normed rows, bfloat16")
    rows, dense, index, weight = rnd(5, P, H), rnd(6, T, H), torch.arange(T * R).reshape(T, R) * 7 % P, rnd(9, T, R)
    y2 = dense + torch.einsum("tr,trw->tw", weight, rows[index])
    x = dev32(X.reshape(T, S * H))
    out32.zero_()
    ops.stream_mix_norm(x, S, mix=(dev32(rows), index.int().to(DEV), dev32(weight), dev32(dense), None), carry=dev32(M),
                        write=dev32(w), read=dev32(r), norm=norm, out32=out32)
    Xn = torch.einsum("cd,tcw->tdw", M, X) + w[None, :, None] * y2[:, None, :]
    close(x.view(T, S, H), Xn, 1e-5, "copies after a sum of rows")
    close(out32, rms(torch.einsum("c,tcw->tw", r, Xn)), 1e-5, "float32 rows alone")
    x = dev32(X.reshape(T, S * H))
    out.zero_()
    ops.stream_mix_norm(x, S, norm=norm, out=out)
    close(x.view(T, S, H), X.float(), 0.0, "copies with nothing pending")
    close(out, rms(X.sum(dim=1)), 2 ** -7, "the closing sum")


def batch_of(parts, tables=None, width=1):
    """``parts``: (slot, first position, rows) per entry."""
    from nano_vllm_cpp_b200.engine.batch import StepEntry, EntryInfo
    from batch_builder import build_batch
    ses, infos, row0 = [], [], 0
    for i, (slot, pos0, n) in enumerate(parts):
        ses.append(StepEntry(i, [0] * n, []))
        infos.append(EntryInfo(i, slot, pos0, n, row0))
        row0 += n
    return build_batch(ses, infos, [tables] if tables is not None else [], width, DEV)


def run_cut(forward, xs, cuts, slots, tables=None):
    """``xs``: one [T_i, width] input per request; ``cuts``: per step, the rows every request runs ((lo, hi) or None);
    ``forward(rows float64, batch)``.  Returns per request the float32 outputs of all its rows."""
    outs = [[] for _ in xs]
    for cut in cuts:
        live = [(i, c) for i, c in enumerate(cut) if c is not None]
        batch = batch_of([(slots[i], lo, hi - lo) for i, (lo, hi) in live],
                         None if tables is None else [tables[i] for i, _ in live],
                         1 if tables is None else max(len(t) for t in tables))
        y = forward(torch.cat([xs[i][lo:hi] for i, (lo, hi) in live]), batch)
        at = 0
        for i, (lo, hi) in live:
            outs[i].append(y[at:at + hi - lo].float().cpu())
            at += hi - lo
    return [torch.cat(o) for o in outs]


CUTS = [[(0, 37), (0, 2)], [(37, 38), (2, 19)], [(38, 40), (19, 20)], [(40, 41), (20, 21)], [None, (21, 50)],
        [(41, 64), (50, 51)], [(64, 65), None], [(65, 66), None]]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,taps", [(64, 4), (50, 4), (64, 1), (1100, 2), (96, 3), (64, 6), (30, 7)])
def test_causal_convolution_alone(H, taps, dtype):
    """Portions beside single rows, portions shorter than the convolution, steps of single rows only (the state is then
    brought up to date by the same launch); slots in another order than the requests."""
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    from nano_vllm_cpp_b200.cache import DeviceCache
    W = {"c": rnd(H + taps, H, taps)}
    part = build_part("input_filter", PartSpec("causal_convolution", dict(size=H, taps=taps, name="c")))
    ctx = ctx_for(dtype)
    part.load(Fetch(W, "", torch.float32), ctx)
    view = None
    if taps > 1:
        cache = DeviceCache([part.cache_spec()], 16, 4, DEV, dtype)
        cache.allocate(0)
        view = cache.view(0)
    xs = [rnd(60 + i, n, H).float().double() for i, n in enumerate((66, 51))]
    got = run_cut(lambda x, b: part.forward(dev32(x), b, view), xs, CUTS, [2, 1])
    for i, x in enumerate(xs):
        close(got[i], x + ps.causal_convolution(x, W["c"].float().double()), 1e-6 if dtype == torch.float32 else 2 ** -7, f"request {i}")
    # many rows (a thread then walks several of them), an entry border in the middle of a thread's rows
    xs = [rnd(70 + i, n, H).float().double() for i, n in enumerate((601, 3, 100))]
    if taps > 1:
        cache.allocate(0)
        view = cache.view(0)
    got = run_cut(lambda x, b: part.forward(dev32(x), b, view), xs, [[(0, 600), (0, 3), (0, 77)], [(600, 601), None, (77, 100)]],
                  [0, 3, 1])
    for i, x in enumerate(xs):
        close(got[i], x + ps.causal_convolution(x, W["c"].float().double()), 1e-6 if dtype == torch.float32 else 2 ** -7, f"many rows, request {i}")


def retention_setup(m, width, W, dtype, fast=True):
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    from nano_vllm_cpp_b200.cache import DeviceCache
    rot = m.get("rot")
    position = PartSpec("rotary_neox", dict(rotary_dim=rot["dims"], theta=rot["base"])) if rot else PartSpec("none")
    part = build_part("mixer", PartSpec("retention", dict(hidden_size=width, heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                                          decay=m["decay"], eps=1e-5, position=position)))
    ctx = ctx_for(dtype, fast)
    part.load(Fetch(W, "m.", dtype), ctx)
    cache = DeviceCache([part.cache_spec()], 16, 4, DEV, dtype)
    cache.allocate(0)
    return part, cache, ctx


RETENTIONS = [ps.retention_layer(heads=3, dim=32, vdim=40, rot_dims=20, base=500.0, decay=[0.5, 0.9, 0.995]),
              ps.retention_layer(heads=2, dim=48, vdim=16, rot_dims=0, decay=[0.98, 0.75]),
              ps.retention_layer(heads=2, dim=64, vdim=64, decay=[0.97, 0.999]),
              ps.retention_layer(heads=1, dim=128, vdim=128, rot_dims=64, decay=[0.99]),
              ps.retention_layer(heads=1, dim=16, vdim=200, rot_dims=6, decay=[1.0]),
              ps.retention_layer(heads=2, dim=256, vdim=96, rot_dims=256, decay=[0.9, 0.998]),
              ps.retention_layer(heads=2, dim=7, vdim=13, rot_dims=6, decay=[0.0, 0.95]),
              ps.retention_layer(heads=1, dim=130, vdim=65, rot_dims=2, decay=[0.96]),
              ps.retention_layer(heads=1, dim=300, vdim=300, rot_dims=128, decay=[0.97])]


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", RETENTIONS)
def test_retention_alone(layer, dtype, fast):
    """Two requests in portions beside single rows, in slots that other requests held before: keys and values of many
    sizes, the whole head, part of it and nothing turned, decays of zero and one; the states that are left behind."""
    m, width = layer["mixer"], 80
    W = weights_of(layer, width, 21)
    part, cache, ctx = retention_setup(m, width, W, dtype, fast)
    xs = inputs(width, [66, 51], 22)
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [3, 0])
    state = cache.view(0).state
    for i, x in enumerate(xs):
        last = []
        want = ps.retention(x, W, "m.", m, 1e-5, last)
        close(got[i], want, 1e-4 if dtype == torch.float32 else 2e-2, f"request {i}")
        close(state[[3, 0][i]].reshape(1, -1), last[0].reshape(1, -1), 1e-4 if dtype == torch.float32 else 2e-2, f"state {i}")
    # the slots are zeroed on the device before the step that starts a request in them
    batch = batch_of([(3, 0, 5), (0, 51, 1)])
    cache.reset_fresh(batch)
    assert float(cache.view(0).state[3].abs().max()) == 0.0
    assert float(cache.view(0).state[0].abs().max()) > 0.0


@pytest.mark.parametrize("cut", [[130], [63, 67], [64, 66], [65, 65], [2, 62, 64, 2], [1, 64, 65], [128, 2], [129, 1], [62, 2, 66]])
@pytest.mark.parametrize("layer", [RETENTIONS[2], RETENTIONS[0]])
def test_retention_in_chunks(layer, cut):
    """Portions that end just before, at and just after a chunk of 64 rows, single rows between them."""
    m, width = layer["mixer"], 80
    W = weights_of(layer, width, 23)
    part, cache, _ = retention_setup(m, width, W, torch.bfloat16)
    x = inputs(width, [130], 24)[0]
    at, cuts = 0, []
    for n in cut:
        cuts.append([(at, at + n)])
        at += n
    assert at == 130
    got = run_cut(lambda x, b: part.forward(x.to(torch.bfloat16).to(DEV), b, cache.view(0)), [x], cuts, [1])[0]
    close(got, ps.retention(x, W, "m.", m, 1e-5), 2e-2, f"cut {cut}")


def test_chunked_retention_keeps_sixteen_bits():
    """The operands enter the tensor-core products as two bfloat16 terms each: the states that a long portion leaves
    behind agree with a float64 recurrence over the same float32 projections to far better than bfloat16."""
    from nano_vllm_cpp_b200.csrc import ops
    H, dk, dv, T = 2, 64, 64, 300
    proj = rnd(81, T, 2 * H * (dk + dv)).float()
    decay = torch.tensor([0.96, 0.999], dtype=F64)
    powers = torch.pow(decay[:, None], torch.arange(65, dtype=F64)[None, :]).float().to(DEV)
    cols = {"q": 0, "k": H * dk, "v": 2 * H * dk, "g": 2 * H * dk + H * dv}
    S = torch.zeros(3, H, dk, dv, device=DEV)
    out = torch.empty(T, H * dv, device=DEV)
    ops.retention(proj.to(DEV), cols, batch_of([(1, 0, T)]), S, powers, torch.zeros(1, device=DEV), 0, H, dk, dv, 1e-6, out)
    p = proj.double()
    for h in range(H):
        st, o = torch.zeros(dk, dv, dtype=F64), torch.zeros(T, dv, dtype=F64)
        for t in range(T):
            st = decay[h] * st + torch.outer(p[t, H * dk + h * dk:][:dk] / math.sqrt(dk), p[t, 2 * H * dk + h * dv:][:dv])
            o[t] = st.T @ p[t, h * dk:][:dk]
        y = ps.unit_rms(o, 1e-6) * ps.silu(p[:, cols["g"] + h * dv:][:, :dv])
        close(S[1, h].reshape(1, -1), st.reshape(1, -1), 5e-5, f"state of head {h}")
        close(out[:, h * dv:(h + 1) * dv], y, 2e-4, f"outputs of head {h}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gap,decoded", [(3, False), (64, False), (65, False), (250, False), (250, True), (640, True)])
def test_a_far_token_in_the_state(gap, decoded, dtype):
    """Row i asks for the key of row i - gap, which stands out (its input is row i's, enlarged, plus something that the
    keys do not see, so it has a value of its own): most of row i's output is that value, and without it the output is
    another one.  With a decay close to one through chunks, portions and single rows."""
    i = gap + 5
    T, width = i + 2, 128
    layer = ps.retention_layer(heads=2, dim=32, vdim=32, rot_dims=0, decay=[0.999, 0.9985])
    m = layer["mixer"]
    W = weights_of(layer, width, 31)
    W["m.q"] = W["m.k"].clone()
    x = 0.1 * rnd(32, T, width)
    x[i] = rnd(33, width)
    K, free = W["m.k"], rnd(34, width)
    free = free - K.T @ torch.linalg.solve(K @ K.T, K @ free)          # what the keys do not see
    x[i - gap] = 4.0 * (x[i] + 2.0 * free)
    x = x.to(torch.bfloat16).double()
    part, cache, _ = retention_setup(m, width, W, dtype)
    cuts = [[(0, T)]] if not decoded else [[(0, i - 2)]] + [[(t, t + 1)] for t in range(i - 2, T)]
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), [x], cuts, [2])[0]
    want = ps.retention(x, W, "m.", m, 1e-5)
    close(got, want, 1e-4 if dtype == torch.float32 else 2e-2, "rows")
    without = x.clone()
    without[i - gap] = 0
    other = ps.retention(without, W, "m.", m, 1e-5)
    assert float((other[i] - want[i]).abs().max()) > 0.2 * float(want[i].abs().max())


# ------------------------------------------------------------------------------- attention
def attention_setup(m, width, W, dtype, fast=True, pages=64, own=True, lender=None):
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    from nano_vllm_cpp_b200.cache import DeviceCache
    part = build_part("mixer", PartSpec("paged_attention", dict(
        hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
        bias=False, position=PartSpec("none"), scale=m["scale"], qk_norm_eps=1e-5, qk_norm_whole=True, output_gate=True,
        own_kv=own, round_weights=True,
        names={"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_norm": "q.norm", "k_norm": "k.norm"})))
    ctx = ctx_for(dtype, fast)
    part.load(Fetch(W, "m.", dtype), ctx)
    if lender is not None:
        return part, lender, ctx
    cache = DeviceCache([part.cache_spec()], 16, 4, DEV, dtype)
    cache.allocate(pages, 64)
    return part, cache, ctx


ATTENTIONS = [ps.attention_layer(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.2),
              ps.attention_layer(heads=3, kv_heads=3, dim=40, vdim=24, scale=0.11),
              ps.attention_layer(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.125),
              ps.attention_layer(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.09),
              ps.attention_layer(heads=6, kv_heads=1, dim=96, vdim=96, scale=0.1),
              ps.attention_layer(heads=20, kv_heads=1, dim=64, vdim=32, scale=0.12),
              ps.attention_layer(heads=2, kv_heads=1, dim=256, vdim=256, scale=0.06),
              ps.attention_layer(heads=2, kv_heads=1, dim=192, vdim=80, scale=0.07),
              ps.attention_layer(heads=1, kv_heads=1, dim=8, vdim=16, scale=0.5),
              # between the sizes that the tensor-core forms are made for: the next larger form, its rest filled with zeros
              ps.attention_layer(heads=4, kv_heads=2, dim=80, vdim=80, scale=0.11),
              ps.attention_layer(heads=3, kv_heads=3, dim=112, vdim=104, scale=0.1),
              ps.attention_layer(heads=17, kv_heads=1, dim=144, vdim=136, scale=0.08),
              ps.attention_layer(heads=2, kv_heads=2, dim=208, vdim=208, scale=0.07)]
PAGES = [[7, 3, 11, 0, 9], [5, 2, 8, 10]]


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", ATTENTIONS)
def test_attention_alone(layer, dtype, fast):
    """Two requests on scattered pages, in portions beside single rows: the norms over all heads, grouped heads, values
    of another size than keys, the gates."""
    m, width = layer["mixer"], 80
    W = weights_of(layer, width, 41)
    part, cache, ctx = attention_setup(m, width, W, dtype, fast)
    xs = inputs(width, [66, 51], 42)
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [0, 1], PAGES)
    ctx.err.check("attention")
    for i, x in enumerate(xs):
        want = ps.attention(x, W, "m.", m, 1e-5, ps.keys_and_values(x, W, "m.", m, 1e-5))
        close(got[i], want, 1e-4 if dtype == torch.float32 else 3e-2, f"request {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", [ATTENTIONS[0], ATTENTIONS[2], ATTENTIONS[4]])
def test_keys_and_values_of_another_layer(layer, dtype):
    """A layer without keys and values of its own reads the pages that another layer filled from another input, with its
    own queries, gates, number of heads and scale, in portions and single rows; it writes nothing."""
    m, width = layer["mixer"], 80
    r = dict(m, heads=m["kv_heads"] * 3, scale=m["scale"] * 1.5, kv_from=0)
    W = weights_of(layer, width, 43)
    R = weights_of({"type": "attention", "mixer": r, "mlp": None}, width, 44)
    assert not any(k in R for k in ("m.k", "m.v", "m.k.norm"))
    owner, cache, _ = attention_setup(m, width, W, dtype)
    reader, _, _ = attention_setup(r, width, R, dtype, own=False, lender=cache)
    xs, ys = inputs(width, [66, 51], 45), inputs(width, [66, 51], 46)
    both = [torch.cat([x, y], dim=1) for x, y in zip(xs, ys)]

    def forward(xy, b):
        owner.forward(xy[:, :width].to(dtype).to(DEV), b, cache.view(0))
        before = cache.view(0).k.clone()
        out = reader.forward(xy[:, width:].to(dtype).to(DEV), b, cache.view(0).read_only())
        assert torch.equal(before, cache.view(0).k)
        return out

    got = run_cut(forward, both, CUTS, [0, 1], PAGES)
    for i in range(2):
        want = ps.attention(ys[i], R, "m.", r, 1e-5, ps.keys_and_values(xs[i], W, "m.", m, 1e-5))
        close(got[i], want, 1e-4 if dtype == torch.float32 else 3e-2, f"request {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dim,i,j", [(32, 50, 0), (32, 50, 15), (32, 50, 16), (32, 330, 1), (64, 330, 127), (64, 330, 128),
                                     (64, 700, 0), (128, 300, 63), (96, 500, 64), (96, 333, 2), (80, 400, 65), (176, 290, 17)])
def test_one_key_stands_out(dim, i, j, decoded, dtype):
    """Row i's softmax falls in halves on key j and on itself (row j's input is row i's plus something that the key
    projection does not see, so its key is the same and its value another): the first tokens, page and tile borders,
    hundreds of positions back among scattered pages; in a prompt, and decoded after single rows."""
    T, width = i + 3, 3 * dim
    layer = ps.attention_layer(heads=2, kv_heads=1, dim=dim, vdim=dim, scale=1.0)
    m = layer["mixer"]
    W = weights_of(layer, width, 51)
    W["m.q"] = torch.cat([W["m.k"], W["m.k"]])
    W["m.q.norm"] = torch.cat([W["m.k.norm"], W["m.k.norm"]])
    x = rnd(52, T, width)
    K = W["m.k"]
    free = rnd(53, width)
    free = free - K.T @ torch.linalg.solve(K @ K.T, K @ free)          # what the keys do not see
    x[j] = x[i] + 2.0 * free * (x[i].norm() / free.norm())
    x = x.to(torch.bfloat16).double()
    part, cache, ctx = attention_setup(m, width, W, dtype)
    n_pages = (T + 15) // 16
    table = [(11 * p + 3) % 61 for p in range(n_pages)]
    assert len(set(table)) == n_pages
    cuts = [[(0, T)]] if not decoded else [[(0, i - 2)]] + [[(t, t + 1)] for t in range(i - 2, T)]
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), [x], cuts, [0], [table])[0]
    ctx.err.check("attention")
    k, v = ps.keys_and_values(x, W, "m.", m, 1e-5)
    rows = list(range(i - 2, T))
    q = (ps.unit_rms(x[rows] @ W["m.q"].T, 1e-5) * W["m.q.norm"]).view(len(rows), 2, dim)
    gate = torch.sigmoid(x[rows] @ W["m.g"].T)

    def plain(hide=None):
        out = torch.zeros(len(rows), 2, dim, dtype=F64)
        for a, t in enumerate(rows):
            s = torch.einsum("hd,jd->hj", q[a], k[:t + 1, 0])
            if hide is not None:
                s[:, hide] = -1e30
            out[a] = gate[a][:, None] * (torch.softmax(s, dim=1) @ v[:t + 1, 0])
        return out.reshape(len(rows), -1) @ W["m.o"].T

    want = plain()
    close(got[rows], want, 2e-4 if dtype == torch.float32 else 4e-2, "rows")
    assert float((plain(hide=j)[2] - want[2]).abs().max()) > 0.2 * float(want[2].abs().max())


# ------------------------------------------------------------------------------- feed-forwards
@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff", [(64, 72), (256, 320), (50, 33), (128, 1024)])
def test_gelu_gated_feed_forward_alone(width, ff, dtype, fast):
    """One row, a handful (the weight-streaming product), a prompt (tensor cores), and widths those refuse; gate values
    from deep in gelu's flat part to far in its straight one."""
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    W = weights_of(ps.attention_layer(mlp=ps.dense(ff)), width, 61, "mlp")
    W["m.gate"] = (W["m.gate"] * 2.5).to(torch.bfloat16).double()
    part = build_part("feed_forward", PartSpec("dense_swiglu", dict(
        hidden_size=width, intermediate_size=ff, activation="gelu_tanh", names={"gate": "gate", "up": "up", "down": "down"})))
    part.load(Fetch(W, "m.", dtype), ctx_for(dtype, fast))
    for T in (1, 5, 20, 70, 300):
        x = inputs(width, [T], 62 + T)[0]
        h = x.to(dtype).to(DEV)
        want = ps.glu(x, W, "m.", ps.gelu_tanh)
        close(part.forward(h, h, None), want, 1e-4 if dtype == torch.float32 else 2e-2, f"T={T}")
        assert float((ps.glu(x, W, "m.", ps.silu) - want).abs().max()) > 0.02 * float(want.abs().max())


@pytest.mark.parametrize("E,K", [(6, 2), (8, 3), (5, 5), (1, 1), (70, 4), (8, 1)])
def test_router_with_a_bias(E, K):
    """Biases large enough to change choices: both routing kernels choose by the biased logits and weigh by the softmax
    over the chosen ones."""
    from nano_vllm_cpp_b200.csrc import ops
    for T in (1, 7, 300):
        W = {"m.router": rnd(71 + E, E, 48) / 7, "m.router.b": 1.5 * rnd(72 + E, E)}
        h = rnd(73 + T, T, 48)
        picks, _ = ps.route(h, W, "m.", {"experts": E, "top": K})
        plainly, _ = ps.route(h, {"m.router": W["m.router"], "m.router.b": 0 * W["m.router.b"]}, "m.", {"experts": E, "top": K})
        assert K == E or T == 1 or [[e for e, _ in p] for p in picks] != [[e for e, _ in p] for p in plainly]
        logits = dev32(h @ W["m.router"].T)
        rule = ("softmax", dev32(W["m.router.b"]), 1.0)
        kinds = ["topk"] + (["small"] if ops.moe_route_small_usable(T, E, K, 0, 48) else [])
        for kind in kinds:
            idx = torch.full((T, K), -1, dtype=torch.int32, device=DEV)
            score = torch.empty(T, K, dtype=torch.float32, device=DEV)
            if kind == "topk":
                ops.router_topk(logits, K, True, idx, score, rule=rule)
            else:
                al = ops.MoeAlignment(T * K, E, 16, DEV, 0)
                ops.moe_route_small(logits, K, True, 0, None, idx, score, al, ops.ErrorFlag(DEV), rule=rule)
            gi, gs = idx.cpu(), score.cpu().double()
            for t in range(T):
                assert [int(e) for e in gi[t]] == [e for e, _ in picks[t]], f"{kind} row {t}"
                assert max(abs(float(gs[t, k]) - picks[t][k][1]) for k in range(K)) < 1e-5


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,mlp", [(64, ps.moe(6, 2, 24)), (64, ps.moe(5, 5, 40)), (64, ps.moe(8, 1, 32)), (50, ps.moe(3, 2, 20)),
                                       (256, ps.moe(16, 4, 128)), (128, ps.moe(12, 3, 64)), (64, ps.moe(1, 1, 16))])
def test_mixture_alone(width, mlp, dtype, fast):
    """One row, a handful, and more rows than the one-launch routing takes; widths the tensor-core product refuses."""
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    W = weights_of(ps.attention_layer(mlp=mlp), width, 74, "mlp")
    ff = build_part("feed_forward", PartSpec("sparse_moe_swiglu", dict(
        hidden_size=width, num_experts=mlp["router"]["experts"], top_k=mlp["router"]["top"],
        intermediate_size=mlp["expert"]["ff"], renormalize=True, router_bias=True,
        names={"router": "router", "router_bias": "router.b", "expert_gate": "e{}.gate", "expert_up": "e{}.up",
               "expert_down": "e{}.down"})))
    ff.load(Fetch(W, "m.", dtype), ctx_for(dtype, fast))
    for T in (1, 5, 70, 300):
        x = inputs(width, [T], 75 + T)[0]
        h32 = dev32(x)
        y = ff.forward(h32.to(dtype), h32, None)
        close(y if isinstance(y, torch.Tensor) else y.sum(), ps.mixture(x, W, "m.", mlp), 1e-4 if dtype == torch.float32 else 3e-2, f"T={T}")


def test_an_input_filter_in_a_pre_norm_layer():
    """The convolution is a slot of the pre-norm layer too: ``x + mixer(f(norm(x)))`` and then the feed-forward, its state
    beside the mixer's pages in one composite."""
    from nano_vllm_cpp_b200.parts import LayerSpec, PartSpec, build_layer, StateCacheSpec
    from nano_vllm_cpp_b200.cache import DeviceCache
    width, eps = 64, 1e-5
    layer = ps.attention_layer(heads=2, kv_heads=1, dim=32, vdim=32, scale=0.2, mlp=ps.dense(48))
    cfg = ps.model_config([layer], width=width, vocab=8, taps=3, eps=eps)
    W = ps.make_weights(cfg, 91)
    norm = lambda n: PartSpec("rmsnorm", dict(size=width, eps=eps, weight_offset=1.0, weight_name=n))
    block = build_layer(LayerSpec(
        parts={"norm1": norm("norm1"), "norm2": norm("norm2"),
               "input_filter": PartSpec("causal_convolution", dict(size=width, taps=3, name="canon1")),
               "mixer": PartSpec("paged_attention", dict(
                   hidden_size=width, num_heads=2, num_kv_heads=1, head_dim=32, bias=False, position=PartSpec("none"),
                   scale=0.2, qk_norm_eps=eps, qk_norm_whole=True, output_gate=True,
                   names={"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_norm": "q.norm", "k_norm": "k.norm"})),
               "feed_forward": PartSpec("dense_swiglu", dict(hidden_size=width, intermediate_size=48, activation="gelu_tanh",
                                                             names={"gate": "gate", "up": "up", "down": "down"}))},
        names={"norm1": "", "norm2": "", "input_filter": "", "mixer": "mix.", "feed_forward": "mlp."}))
    ctx = ctx_for(torch.float32)
    for prefix, part in block.parts():
        part.load(Fetch(W, "l0." + prefix, torch.float32), ctx)
    spec = block.cache_spec()
    assert spec.parts[0] == block.mixer.cache_spec() and spec.parts[1] == StateCacheSpec((2, width))
    cache = DeviceCache([spec], 16, 4, DEV, torch.float32)
    cache.allocate(16, 16)
    xs = [rnd(92 + i, n, width).float().double() for i, n in enumerate((66, 51))]

    def forward(x, b):
        x = dev32(x)
        return x + block.forward(x, None, b, cache.view(0))

    got = run_cut(forward, xs, CUTS, [1, 3], PAGES)
    for i, x in enumerate(xs):
        h = ps.norm_one_plus(x, W["l0.norm1"], eps)
        h = h + ps.causal_convolution(h, W["l0.canon1"])
        x = x + ps.attention(h, W, "l0.mix.", layer["mixer"], eps, ps.keys_and_values(h, W, "l0.mix.", layer["mixer"], eps))
        want = x + ps.glu(ps.norm_one_plus(x, W["l0.norm2"], eps), W, "l0.mlp.", ps.gelu_tanh)
        close(got[i], want, 1e-4, f"request {i}")


# ------------------------------------------------------------------------------- whole models through the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_the_stream_layer_by_layer(name, dtype, models):
    """The sum of the copies after every layer."""
    from nano_vllm_cpp_b200.engine.batch import StepEntry
    cfg, W, folder = models[name]
    ids = ids_for(name, 37, salt=3)
    want, margins, got = [], [], []
    ps.forward(cfg, W, ids, layer_sums=want, margins=margins)
    runner = make_runner(folder, dtype, 64)
    n = runner.model.spec.streams

    def look(i, x, pending):
        y = pending.branch if isinstance(pending.branch, torch.Tensor) else pending.branch.sum()
        X = torch.einsum("cd,tcw->tdw", pending.link.carry, x.view(x.shape[0], n, -1)) + pending.link.write[None, :, None] * y[:, None, :]
        got.append(X.sum(dim=1).cpu())

    runner.model.after_call = look
    runner.step([StepEntry("x", ids, [])])
    assert len(got) == len(want)
    half = dtype == "bfloat16"
    edge = torch.stack(margins).min(dim=0).values if margins and half else None
    errors = ps.rounding_errors(cfg, W, ids, NOISE, layer=True) if half else [None] * len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        close(g, w, 3e-2 if half else 2e-5, f"layer {i}", edge, errors[i])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(name, dtype, models):
    runner = make_runner(models[name][2], dtype, 256)
    st = Steps(runner)
    for n in (1, 2, 3, 17, 64, 65, 150):
        ids = ids_for(name, n)
        st.step([(f"w{n}", ids)], end=[f"w{n}"])
        check_rows(st, models, name, f"w{n}", ids, dtype, f"{name} whole n={n}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token(name, dtype, models):
    """A short prompt in one step, then ninety rows one at a time (steps of the same shape are replayed from a captured
    graph), and a sequence that is decoded from its first token on in a slot that was used before."""
    runner = make_runner(models[name][2], dtype, 256)
    st = Steps(runner)
    ids = ids_for(name, 100, salt=1)
    st.step([("d", ids[:10])])
    for t in range(10, 100):
        st.step([("d", ids[t:t + 1])])
    check_rows(st, models, name, "d", ids, dtype, f"{name} decode")
    st.step([], end=["d"])
    ids = ids_for(name, 20, salt=2)
    for t in range(20):
        st.step([("e", ids[t:t + 1])])
    check_rows(st, models, name, "e", ids, dtype, f"{name} decode from the first token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_several_sizes(name, dtype, models):
    runner = make_runner(models[name][2], dtype, 256)
    st = Steps(runner)
    ids = ids_for(name, 131, salt=3)
    sizes = [2, 1, 2, 14, 13, 3, 2, 30, 1, 1, 17, 2, 33, 10]
    assert sum(sizes) == 131
    at = 0
    for s in sizes:
        st.step([("p", ids[at:at + s])])
        at += s
    check_rows(st, models, name, "p", ids, dtype, f"{name} portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_together_with_pages_and_slots_used_again(name, dtype, models):
    """Three slots and 192 tokens of pages for six requests that need more in turn: portions of some beside single rows of
    others; a finished request's pages and slot go to the next one.  Every request's logits equal those of the request
    alone."""
    runner = make_runner(models[name][2], dtype, 192, max_requests=3)
    st = Steps(runner)
    L = {"a": 50, "b": 37, "c": 64, "d": 20, "e": 61, "f": 33}
    ids = {r: ids_for(name, n, salt=ord(r)) for r, n in L.items()}
    at = {r: 0 for r in L}

    def take(r, n):
        toks = ids[r][at[r]:at[r] + n]
        at[r] += len(toks)
        return (r, toks)

    def done(*rs):
        return [r for r in rs if at[r] == L[r]]

    st.step([take("a", 30), take("b", 2)])
    st.step([take("a", 1), take("b", 35), take("c", 3)], end=done("b"))
    st.step([take("a", 19), take("c", 1), take("d", 20)], end=done("a", "d"))
    st.step([take("c", 60), take("e", 2), take("f", 1)], end=done("c"))
    st.step([take("e", 1), take("f", 2)])
    st.step([take("e", 58), take("f", 30)], end=done("e", "f"))
    for r, n in L.items():
        assert at[r] == n
        check_rows(st, models, name, r, ids[r], dtype, f"{name} request {r}")


def drawn_config(seed):
    """A model of drawn sizes: layer order, head counts and sizes, borrowed keys, feed-forwards, copies and taps."""
    rng = random.Random(seed)
    layers, owners = [], []
    for i in range(rng.randint(3, 5)):
        ff = rng.choice([None, ps.dense(rng.choice([24, 40, 64])), ps.moe(rng.choice([3, 4, 8]), rng.choice([1, 2, 3]), rng.choice([16, 24, 32]))])
        if rng.random() < 0.5:
            heads, dim = rng.choice([1, 2, 3, 4]), rng.choice([16, 24, 32, 64, 80])
            rot = rng.choice([0, 2, dim // 2 // 2 * 2, dim])
            layers.append(ps.retention_layer(heads=heads, dim=dim, vdim=rng.choice([dim, 16, 48, 96]), rot_dims=rot,
                                             base=rng.choice([100.0, 1e4]), decay=[rng.uniform(0.8, 1.0) for _ in range(heads)], mlp=ff))
        elif owners and rng.random() < 0.5:
            j = rng.choice(owners)
            m = layers[j]["mixer"]
            layers.append(ps.attention_layer(heads=m["kv_heads"] * rng.choice([1, 2, 3]), kv_heads=m["kv_heads"], dim=m["dim"],
                                             vdim=m["vdim"], scale=rng.uniform(0.1, 0.3), kv_from=j, mlp=ff))
        else:
            kv, dim = rng.choice([1, 2, 3]), rng.choice([16, 24, 40, 64, 96, 128])
            layers.append(ps.attention_layer(heads=kv * rng.choice([1, 2, 4]), kv_heads=kv, dim=dim, vdim=rng.choice([dim, dim, 32]),
                                             scale=rng.uniform(0.1, 0.3), mlp=ff))
            owners.append(i)
    return ps.model_config(layers, width=rng.choice([48, 64, 72, 128]), vocab=rng.choice([97, 160]), streams=rng.choice([1, 2, 3, 4, 5]),
                           taps=rng.choice([1, 2, 3, 4, 5]), eps=rng.choice([1e-6, 1e-4]), embed_scale=rng.uniform(0.5, 6.0))


@pytest.mark.parametrize("seed", range(8))
def test_drawn_models_in_a_mixed_schedule(seed, tmp_path):
    cfg = drawn_config(seed)
    W = ps.make_weights(cfg, 100 + seed)
    folder = ps.write_folder(cfg, W, str(tmp_path))
    g = torch.Generator().manual_seed(seed)
    ids = {r: [int(t) for t in torch.randint(0, cfg["vocab"], (n,), generator=g)] for r, n in (("a", 70), ("b", 1), ("c", 33), ("d", 18))}
    for dtype in ("float32", "bfloat16"):
        st = Steps(make_runner(folder, dtype, 160, max_requests=3))
        st.step([("a", ids["a"][:37]), ("b", ids["b"])], end=["b"])
        st.step([("a", ids["a"][37:38]), ("c", ids["c"][:2])])
        st.step([("a", ids["a"][38:39]), ("c", ids["c"][2:3])])
        st.step([("a", ids["a"][39:68]), ("c", ids["c"][3:4]), ("d", ids["d"][:16])])
        st.step([("a", ids["a"][68:]), ("c", ids["c"][4:]), ("d", ids["d"][16:17])], end=["a"])
        st.step([("d", ids["d"][17:])], end=["c", "d"])
        for r, toks in ids.items():
            margins = []
            want = ps.forward(cfg, W, toks, margins=margins)
            half = dtype == "bfloat16"
            close(st.rows(r, len(toks)), want, TOL[dtype], f"drawn model {seed} {dtype} request {r}",
                  torch.stack(margins).min(dim=0).values if margins and half else None,
                  (lambda: ps.rounding_errors(cfg, W, toks, NOISE)) if half else None)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_cutting_does_not_change_a_row(dtype, models):
    """The same request whole, in portions and beside another request: float32 rows agree to rounding of sums, bfloat16
    rows to bfloat16 rounding."""
    name = "M"
    ids, other = ids_for(name, 70, salt=9), ids_for(name, 40, salt=10)
    _, margins = plain_logits(models, name, ids)
    runs = []
    for cut in ([70], [33, 1, 2, 34], [64, 6]):
        st = Steps(make_runner(models[name][2], dtype, 256))
        at = 0
        for k, s in enumerate(cut):
            st.step([("x", ids[at:at + s])] + ([("o", other[:20] if k == 0 else other[20 + k:21 + k])] if len(cut) == 4 else []))
            at += s
        runs.append(st.rows("x", 70))
    for r in runs[1:]:
        close(r, runs[0], 2e-5 if dtype == "float32" else 3e-2, "the same rows cut another way", margins if dtype == "bfloat16" else None)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(dtype, models):
    """The engine's own entry point, scheduler and sampling: greedy tokens follow the plain implementation's up to the
    first position where its two best logits are closer than the tolerance.  Fewer slots than requests, and prompts cut
    by the token budget."""
    from nano_vllm_cpp_b200 import LLMEngine, SamplingParams
    name = "M"
    cfg, W, folder = models[name]
    prompts = [ids_for(name, 9, salt=20), ids_for(name, 3, salt=21), ids_for(name, 30, salt=22)]
    eng = LLMEngine(folder, max_model_len=96, num_kv_blocks=24, dtype=dtype, max_num_seqs=2, max_num_batched_tokens=16, log_stats=False)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for k, tok in enumerate(o["token_ids"]):
            logits = ps.forward(cfg, W, seq)[-1]
            best = int(torch.argmax(logits))
            if best != tok:
                lead = float(logits[best] - logits[tok])
                bound = 2 * TOL[dtype] * float(logits.abs().max())
                assert lead <= bound, f"token {k} of a prompt of {len(p)}: {tok}, plain takes {best} with a lead of {lead:.3g}"
                break
            seq.append(tok)


def test_command_line_serves_the_design(models, tmp_path, capsys):
    """``nanovllm <folder> --tokens ...`` and ``nanovllm --config <json>`` (random weights) run this design as they run the
    others; the greedy tokens from the folder are the plain implementation's."""
    from nano_vllm_cpp_b200 import cli
    name = "N"
    cfg, W, folder = models[name]
    prompt = ids_for(name, 7, salt=30)
    rc = cli.main([folder, "--tokens", ",".join(map(str, prompt)), "--max-tokens", "6", "--temperature", "0",
                   "--dtype", "float32", "--max-model-len", "64", "--num-kv-blocks", "8", "--ignore-eos"])
    out = capsys.readouterr().out
    assert rc == 0, out
    toks = [int(t) for t in out.strip().splitlines()[-1].split(":")[1].split()]
    assert toks == ps.greedy_generate(cfg, W, prompt, 6)
    path = tmp_path / "config.json"
    path.write_text(json.dumps(CONFIGS["M"]))
    rc = cli.main(["--config", str(path), "--seed", "4", "--tokens", "5,6,7", "--max-tokens", "4", "--temperature", "0",
                   "--max-model-len", "64", "--num-kv-blocks", "8", "--ignore-eos"])
    out = capsys.readouterr().out
    assert rc == 0 and len(out.strip().splitlines()[-1].split(":")[1].split()) == 4
