"""The Dubarax decoder and its mechanisms against the plain implementation (tests/plain_dubarax.py): every part alone, then
whole models through the engine's step function, cache manager and scheduler, for every way of cutting the work into steps.
The configurations are small and of this file's own making; weights are random, and where random weights would hide a fault
(a far key, an edge of a window or a chunk, a far token in a decaying state) they are shaped so that it shows."""
import json
import math
import random

import pytest
import torch

import plain_dubarax as pd

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

CONFIGS = {
    # every mixer with two sets of sizes, values wider and narrower than keys, a loop in the middle, layers without a
    # feed-forward, a mixture without a shared expert, shared experts of a whole number of expert widths and of another width
    "M": pd.model_config(
        [pd.window_layer(heads=4, kv_heads=2, dim=32, vdim=48, size=19, cap=8.0, far=30, rows=10, mlp=pd.moe(8, 2, 24, 4, 2, 40)),
         pd.parallel_layer(pd.chunk_part(6, 3, 16, 24, size=23), pd.lightning_part(3, 24, 40, [0.5, 0.9, 0.995]), mlp=pd.moe(6, 3, 16, 2, 1, 0)),
         pd.mamba_layer(heads=6, vdim=8, state=20, groups=3, conv=3, norm_groups=4, mlp=None),
         pd.window_layer(heads=2, kv_heads=1, dim=40, size=70, cap=30.0, far=50, rows=7, mlp=None, type="attention_2"),
         pd.mamba_layer(heads=4, vdim=24, state=12, groups=1, conv=4, norm_groups=1, mlp=pd.moe(4, 1, 24, 4, 3, 24), type="mamba2_2")],
        width=96, vocab=210, embed_scale=3.0, loop=(1, 3, 3)),
    # sizes of one and values that other models make equal: one head everywhere, chunks and windows of one and two, a
    # convolution of one tap, one expert, every expert and group chosen, a decay of one, no loop, no scale on the embedding
    "N": pd.model_config(
        [pd.parallel_layer(pd.chunk_part(1, 1, 16, size=2), pd.lightning_part(1, 16, 16, [1.0]), 1.0, 1.0, mlp=pd.moe(1, 1, 16, 1, 1, 16)),
         pd.window_layer(heads=1, kv_heads=1, dim=24, vdim=8, size=1, mlp=pd.moe(4, 4, 24, 2, 2, 0)),
         pd.mamba_layer(heads=1, vdim=16, state=8, groups=1, conv=1, norm_groups=1, mlp=None),
         pd.window_layer(heads=5, kv_heads=1, dim=24, vdim=8, size=100, far=64, rows=16, mlp=pd.moe(4, 1, 8, 4, 4, 0)),
         pd.parallel_layer(pd.chunk_part(5, 5, 8, size=1000), pd.lightning_part(1, 8, 24, [0.0]), 0.3, -1.2, mlp=None, type="parallel_2")],
        width=64, vocab=130, embed_scale=1.0),
    # sizes that the tensor-core kernels take: heads of 64 and 128, experts of 64, a width of 128, a loop over everything
    "R": pd.model_config(
        [pd.parallel_layer(pd.chunk_part(8, 2, 64, size=48, scale=0.125), pd.lightning_part(2, 64, 64, [0.97, 0.999]), mlp=pd.moe(8, 3, 64, 4, 3, 128)),
         pd.mamba_layer(heads=8, vdim=32, state=64, groups=2, conv=4, norm_groups=2, mlp=pd.moe(8, 2, 64, 2, 1, 64)),
         pd.window_layer(heads=4, kv_heads=2, dim=128, size=33, scale=0.09, cap=25.0, far=60, rows=16, mlp=pd.moe(8, 2, 64, 4, 2, 64))],
        width=128, vocab=344, embed_scale=8.0, eps=1e-6, loop=(0, 3, 2)),
}
SEEDS = {"M": 3, "N": 5, "R": 7}
NAMES = ["M", "N", "R"]
TOL = {"float32": 1e-4, "bfloat16": 4e-2}
# A bfloat16 row may exceed the tolerance as far as the plain implementation says that roundings move it (NOISE_FACTOR
# times the worst of a few draws of noise of a bfloat16 rounding's size on everything a sublayer reads and gives).  It may
# also rightly choose another expert or group where a router's margin is below EDGE, and then a few of the rows behind it,
# which read what it left in the cache and the states, may be off too.
NOISE, NOISE_FACTOR, EDGE, MAX_BEHIND = 2.0 ** -9, 4.0, 0.02, 0.25


def ids_for(name, n, salt=0):
    g = torch.Generator().manual_seed(1000 * ord(name) + 7 * n + salt)
    return [int(t) for t in torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g)]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        W = pd.make_weights(cfg, SEEDS[name])
        out[name] = (cfg, W, pd.write_folder(cfg, W, str(tmp_path_factory.mktemp("dubarax_" + name))))
    return out


_plain, _errors = {}, {}


def plain_logits(models, name, ids):
    """(logits, per row the smallest router margin of any layer run)"""
    key = (name, tuple(ids))
    if key not in _plain:
        cfg, W, _ = models[name]
        margins = []
        lg = pd.forward(cfg, W, ids, margins=margins)
        _plain[key] = (lg, torch.stack(margins).min(dim=0).values if margins else torch.full((len(ids),), math.inf))
    return _plain[key]


def rounding_errors(models, name, ids):
    key = (name, tuple(ids))
    if key not in _errors:
        _errors[key] = pd.rounding_errors(*models[name][:2], ids, NOISE)
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
    VECTORS = ("rel", "conv", "step")

    def __init__(self, tensors, prefix, dtype):
        self.t, self.p, self.dtype = tensors, prefix, dtype

    def __call__(self, name):
        t = self.t[self.p + name]
        vector = t.dim() <= 1 or name.rpartition(".")[2] in self.VECTORS
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
    cfg = pd.model_config([layer], width=width, vocab=8)
    W = pd.make_weights(cfg, seed)
    return {k.replace(f"l0.{what}.", "m."): v for k, v in W.items() if k.startswith(f"l0.{what}.")}


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
        y = y if isinstance(y, torch.Tensor) else y.sum()
        at = 0
        for i, (lo, hi) in live:
            outs[i].append(y[at:at + hi - lo].float().cpu())
            at += hi - lo
    return [torch.cat(o) for o in outs]


CUTS = [[(0, 37), (0, 2)], [(37, 38), (2, 19)], [(38, 40), (19, 20)], [(40, 41), (20, 21)], [None, (21, 50)],
        [(41, 64), (50, 51)], [(64, 65), None], [(65, 66), None]]
PAGES = [[7, 3, 11, 0, 9], [5, 2, 8, 10]]


def part_on(kind, params, W, dtype, fast=True, pages=64, slots=4):
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    from nano_vllm_cpp_b200.cache import DeviceCache
    part = build_part("mixer", PartSpec(kind, params))
    ctx = ctx_for(dtype, fast)
    part.load(Fetch(W, "m.", dtype), ctx)
    cache = DeviceCache([part.cache_spec()], 16, slots, DEV, dtype)
    cache.allocate(pages, 64)
    return part, cache, ctx


# ------------------------------------------------------------------------------- small pieces
@pytest.mark.parametrize("H,ld,col0,taps", [(64, 64, 0, 4), (50, 61, 7, 4), (64, 96, 16, 1), (1100, 1104, 4, 2), (96, 100, 2, 3),
                                            (64, 64, 0, 6), (30, 30, 0, 7)])
def test_causal_convolution_with_silu(H, ld, col0, taps):
    """Columns of wider rows; portions beside single rows, portions shorter than the convolution, steps of single rows only
    (the state is then brought up to date by the same launch); many rows with an entry border in the middle."""
    from nano_vllm_cpp_b200.csrc import ops
    w, b = rnd(H + taps, H, taps).float().double(), rnd(H, H).float().double()
    state = torch.zeros(4, max(1, taps - 1), H, device=DEV)
    wt, bias = dev32(w.t()), dev32(b)

    def forward(x, batch):
        out = torch.empty(x.shape[0], H, device=DEV)
        ops.causal_conv_silu(dev32(x), col0, wt, bias, batch, state if taps > 1 else None, out)
        return out

    for lengths, cuts, slots in (((66, 51), CUTS, [2, 1]), ((601, 3, 100), [[(0, 600), (0, 3), (0, 77)], [(600, 601), None, (77, 100)]], [0, 3, 1])):
        state.zero_()
        xs = [rnd(60 + i, n, ld).float().double() for i, n in enumerate(lengths)]
        for i, (x, got) in enumerate(zip(xs, run_cut(forward, xs, cuts, slots))):
            close(got, pd.silu(pd.causal_convolution(x[:, col0:col0 + H], w, b)), 2e-6, f"request {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dv,parts", [(4, 32, 1), (6, 8, 4), (3, 7, 1), (3, 7, 3), (64, 64, 4), (9, 600, 1), (1, 16, 2), (2, 96, 2)])
def test_gated_norm(H, dv, parts, dtype):
    """Skip term, gate before the norm over parts of a row, and a gate behind the norm; rows longer than a block's first
    passes; odd sizes and columns."""
    from nano_vllm_cpp_b200.csrc import ops
    T, n, eps = 5, H * dv, 1e-3
    raw, x, gate, w, D = rnd(1, T, n), rnd(2, T, n + 3), rnd(3, T, n + 5), 1 + 0.2 * rnd(4, n), rnd(5, H)
    out = torch.empty(T, n, dtype=dtype, device=DEV)
    tol = 1e-5 if dtype == torch.float32 else 2 ** -7
    ops.gated_norm(dev32(raw), dev32(gate), 5, dev32(w), eps, out, H, dv, parts=parts, gate_first=True, skip=dev32(D), x=dev32(x), x_col=3)
    y = raw + D.repeat_interleave(dv)[None, :] * x[:, 3:]
    want = pd.unit_rms((y * pd.silu(gate[:, 5:])).view(T, parts, n // parts), eps).reshape(T, n) * w
    close(out, want, tol, "gate first")
    ops.gated_norm(dev32(raw), dev32(gate), 0, dev32(w), eps, out, H, dv, parts=parts)
    want = pd.unit_rms(raw.view(T, parts, n // parts), eps).reshape(T, n) * w * torch.sigmoid(gate[:, :n])
    close(out, want, tol, "gate behind")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,N,K,first", [(1, 200, 64, 130), (20, 200, 64, 130), (70, 200, 64, 130), (300, 520, 128, 257), (300, 130, 50, 0), (40, 96, 64, 96)])
def test_silu_on_the_first_columns_of_a_product(M, N, K, first, dtype):
    """The products' epilogue activates the first columns and passes the others: the weight-streaming product, the
    tensor-core product with and without a split sum, the plain one."""
    from nano_vllm_cpp_b200.parts.linear import linear
    a, w, b = rnd(1, M, K).to(torch.bfloat16), (rnd(2, N, K) / 8).to(torch.bfloat16), rnd(3, N)
    want = a.double() @ w.double().T + b
    want[:, :first] = pd.silu(want[:, :first])
    for fast in (True, False):
        got = linear(ctx_for(dtype, fast), a.to(dtype).to(DEV), w.to(dtype).to(DEV), torch.float32, bias=dev32(b), act=("silu_first", first))
        close(got, want, 1e-5, f"fast={fast}")


@pytest.mark.parametrize("H", [64, 50, 1100])
def test_a_norm_takes_two_scaled_branches(H):
    from nano_vllm_cpp_b200.csrc import ops
    T, eps = 7, 1e-4
    x, a, b, w = rnd(1, T, H), rnd(2, T, H), rnd(3, T, H), 1 + 0.1 * rnd(4, H)
    xd, out = dev32(x), torch.empty(T, H, device=DEV)
    ops.add_rmsnorm(xd, dev32(a), dev32(w), eps, out, branch2=dev32(b), branch_scale=0.7, branch2_scale=-1.25)
    want = x + 0.7 * a - 1.25 * b
    close(xd, want, 1e-6, "stream")
    close(out, pd.unit_rms(want, eps) * w, 1e-5, "rows")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [64, 50, 256])
def test_what_stands_before_a_pass(W, dtype):
    """``A x + B x0 + s_t`` with what is pending on the stream taken in first: nothing, a branch, two scaled branches, a sum of
    rows that has not been taken (with a dense term)."""
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    from nano_vllm_cpp_b200.parts.base import BranchSum, RowMix
    T, R = 9, 3
    t = {"loop.in": rnd(1, W, 2 * W) / math.sqrt(2 * W), "loop.step": rnd(2, 3, W)}
    t = {k: v.to(torch.bfloat16).double() for k, v in t.items()}
    part = build_part("pass_input", PartSpec("recall", dict(size=W, passes=3)))
    part.load(Fetch(t, "loop.", dtype), ctx_for(dtype))
    x0, x, a, b = (rnd(3 + i, T, W) for i in range(4))
    rows, dense, weight = rnd(9, T * R, W), rnd(10, T, W), rnd(11, T, R)
    index = torch.randperm(T * R, generator=torch.Generator().manual_seed(1)).view(T, R)
    recalled = part.recall(dev32(x0))
    mixed = dense + torch.einsum("tr,trw->tw", weight, rows[index])
    cases = [(None, 0), (dev32(a), a), (BranchSum(dev32(a), dev32(b), 0.7, 1.3), 0.7 * a + 1.3 * b),
             (RowMix(dev32(rows), index.int().to(DEV), dev32(weight), dev32(dense), None), mixed)]
    for k, (pending, add) in enumerate(cases):
        got, rest = part.forward(dev32(x), pending, recalled, k % 3)
        want = torch.cat([x + add, x0], dim=1) @ t["loop.in"].T + t["loop.step"][k % 3]
        close(got + rest, want, 1e-5 if dtype == torch.float32 else 2e-2, f"case {k}")


@pytest.mark.parametrize("E,K,count,keep", [(8, 2, 4, 2), (6, 3, 2, 1), (12, 4, 3, 3), (64, 6, 8, 3), (70, 4, 35, 4), (1, 1, 1, 1), (9, 2, 9, 2), (160, 8, 2, 1)])
def test_routing_limited_to_groups(E, K, count, keep):
    """Both routing kernels: the best groups by their largest member, the best experts of those, weights as they are; ties go
    to the lower index."""
    from nano_vllm_cpp_b200.csrc import ops
    r = {"experts": E, "top": K, "groups": {"count": count, "keep": keep}}
    for T in (1, 7, 300):
        z = 2.0 * rnd(71 + E + T, T, E).float()
        z[0] = 0.5                                       # a row of ties
        s = torch.softmax(z.double(), dim=1).tolist()
        want = [pd.route(row, r) for row in s]
        free = [pd.route(row, dict(r, groups=None)) for row in s]
        assert keep == count or T == 1 or K <= keep or want != free       # (up to K = keep the limit changes nothing)
        rule = ("softmax", None, 1.0, (count, keep))
        kinds = ["topk"] + (["small"] if ops.moe_route_small_usable(T, E, K, 0, 48, count) else [])
        for kind in kinds:
            idx = torch.full((T, K), -1, dtype=torch.int32, device=DEV)
            score = torch.empty(T, K, dtype=torch.float32, device=DEV)
            if kind == "topk":
                ops.router_topk(z.to(DEV), K, False, idx, score, rule=rule)
            else:
                al = ops.MoeAlignment(T * K, E, 16, DEV, 0)
                ops.moe_route_small(z.to(DEV), K, False, 0, None, idx, score, al, ops.ErrorFlag(DEV), rule=rule)
            gi, gs = idx.cpu(), score.cpu().double()
            for t in range(T):
                assert [int(e) for e in gi[t]] == [e for e, _ in want[t]], f"{kind} row {t}"
                assert max(abs(float(gs[t, k]) - want[t][k][1]) for k in range(K)) < 1e-6


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,mlp", [(64, pd.moe(8, 2, 24, 4, 2, 40)), (64, pd.moe(6, 3, 40, 2, 1, 80)), (50, pd.moe(3, 2, 20, 3, 2, 0)),
                                       (256, pd.moe(16, 4, 128, 4, 2, 256)), (128, pd.moe(10, 3, 128, 5, 3, 192)), (64, pd.moe(1, 1, 16, 1, 1, 16))])
def test_mixture_alone(width, mlp, dtype, fast):
    """One row, a handful, and more rows than the one-launch routing takes; shared experts of a whole number of expert widths
    and of another width, and none."""
    from nano_vllm_cpp_b200.parts import build_part, PartSpec
    W = weights_of(pd.window_layer(mlp=mlp), width, 74, "mlp")
    g = mlp["router"]["groups"]
    ff = build_part("feed_forward", PartSpec("sparse_moe_swiglu", dict(
        hidden_size=width, num_experts=mlp["router"]["experts"], top_k=mlp["router"]["top"], intermediate_size=mlp["expert"]["ff"],
        shared_intermediate_size=mlp.get("shared", {"ff": 0})["ff"], shared_gate=False, groups=(g["count"], g["keep"]),
        names={"router": "router", "expert_gate": "e{}.gate", "expert_up": "e{}.up", "expert_down": "e{}.down",
               "shared_gate_proj": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down"})))
    ff.load(Fetch(W, "m.", dtype), ctx_for(dtype, fast))
    for T in (1, 5, 70, 300):
        x = inputs(width, [T], 75 + T)[0]
        h32 = dev32(x)
        y = ff.forward(h32.to(dtype), h32, None)
        margins = []
        want = pd.mixture(x, W, "m.", mlp, margins)
        got = (y if isinstance(y, torch.Tensor) else y.sum()).double().cpu()
        close(got[margins[0] > 1e-5], want[margins[0] > 1e-5], 1e-4 if dtype == torch.float32 else 3e-2, f"T={T}")


# ------------------------------------------------------------------------------- matrix memories
LIGHTNINGS = [pd.lightning_part(3, 32, 40, [0.5, 0.9, 0.995]), pd.lightning_part(2, 48, 16, [0.98, 0.75]), pd.lightning_part(2, 64, 64, [0.97, 0.999]),
              pd.lightning_part(1, 128, 128, [0.99]), pd.lightning_part(1, 16, 200, [1.0]), pd.lightning_part(2, 256, 96, [0.9, 0.998]),
              pd.lightning_part(2, 7, 13, [0.0, 0.95]), pd.lightning_part(1, 300, 300, [0.97]), pd.lightning_part(5, 8, 8)]


def lightning_on(m, width, W, dtype, fast=True):
    return part_on("lightning_attention", dict(hidden_size=width, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=m["decay"], eps=1e-5),
                   W, dtype, fast, pages=0)


def memory_weights(kind, m, width, seed):
    if kind == "lightning":
        W = weights_of(pd.parallel_layer(right=m), width, seed)
        return {k.replace("m.right.", "m."): v for k, v in W.items() if k.startswith("m.right.")}
    return weights_of(m, width, seed)


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", LIGHTNINGS)
def test_lightning_attention_alone(m, dtype, fast):
    """Two requests in portions beside single rows, in slots that other requests held before: keys and values of many sizes,
    decays of zero and one; the states that are left behind."""
    width = 80
    W = memory_weights("lightning", m, width, 21)
    part, cache, _ = lightning_on(m, width, W, dtype, fast)
    xs = inputs(width, [66, 51], 22)
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [3, 0])
    state = cache.view(0).state
    for i, x in enumerate(xs):
        last = []
        want = pd.lightning(x, W, "m.", m, 1e-5, last)
        close(got[i], want, 1e-4 if dtype == torch.float32 else 2e-2, f"request {i}")
        close(state[[3, 0][i]].reshape(1, -1), last[0].reshape(1, -1), 1e-4 if dtype == torch.float32 else 2e-2, f"state {i}")
    batch = batch_of([(3, 0, 5), (0, 51, 1)])            # a slot is zeroed before the step that starts a request in it
    cache.reset_fresh(batch)
    assert float(cache.view(0).state[3].abs().max()) == 0.0 and float(cache.view(0).state[0].abs().max()) > 0.0


MAMBAS = [pd.mamba_layer(heads=4, vdim=16, state=24, groups=2, conv=4, norm_groups=2), pd.mamba_layer(heads=6, vdim=8, state=20, groups=3, conv=3, norm_groups=4),
          pd.mamba_layer(heads=8, vdim=64, state=64, groups=1, conv=4, norm_groups=8), pd.mamba_layer(heads=4, vdim=64, state=128, groups=4, conv=2, norm_groups=1),
          pd.mamba_layer(heads=1, vdim=16, state=8, groups=1, conv=1, norm_groups=1), pd.mamba_layer(heads=2, vdim=130, state=7, groups=2, conv=6, norm_groups=2),
          pd.mamba_layer(heads=3, vdim=7, state=5, groups=1, conv=4, norm_groups=7), pd.mamba_layer(heads=2, vdim=300, state=300, groups=1, conv=4, norm_groups=3),
          pd.mamba_layer(heads=16, vdim=32, state=200, groups=2, conv=4, norm_groups=2)]


def mamba_on(m, width, W, dtype, fast=True):
    return part_on("state_space_dual", dict(hidden_size=width, heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"],
                                            conv=m["conv"], norm_groups=m["norm_groups"], eps=1e-5), W, dtype, fast, pages=0)


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", MAMBAS)
def test_state_space_mixer_alone(layer, dtype, fast):
    """Two requests in portions beside single rows: shared maps, states and heads of many sizes, one to six taps, norms over
    the row and over parts of it; the states and the convolution's inputs that are left behind."""
    m, width = layer["mixer"], 80
    W = weights_of(layer, width, 23)
    part, cache, _ = mamba_on(m, width, W, dtype, fast)
    xs = inputs(width, [66, 51], 24)
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [3, 0])
    inner, ch = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
    for i, x in enumerate(xs):
        last = []
        want = pd.mamba2(x, W, "m.", m, 1e-5, last)
        tol = 1e-4 if dtype == torch.float32 else 2e-2
        close(got[i], want, tol, f"request {i}")
        close(cache.view(0).parts[0].state[[3, 0][i]].reshape(1, -1), last[0].reshape(1, -1), tol, f"state {i}")
        if m["conv"] > 1:
            u = (x @ W["m.in"].T)[:, inner:inner + ch]
            close(cache.view(0).parts[1].state[[3, 0][i]], u[-(m["conv"] - 1):], 1e-5, f"convolution inputs {i}")


@pytest.mark.parametrize("cut", [[130], [63, 67], [64, 66], [65, 65], [2, 62, 64, 2], [1, 64, 65], [128, 2], [129, 1], [62, 2, 66]])
@pytest.mark.parametrize("kind", ["lightning", "mamba"])
def test_memories_in_chunks(kind, cut):
    """Portions that end just before, at and just after a chunk of 64 rows, single rows between them."""
    width = 80
    m = LIGHTNINGS[2] if kind == "lightning" else MAMBAS[2]
    W = memory_weights(kind, m, width, 25)
    part, cache, _ = lightning_on(m, width, W, torch.bfloat16) if kind == "lightning" else mamba_on(m["mixer"], width, W, torch.bfloat16)
    x = inputs(width, [130], 26)[0]
    at, cuts = 0, []
    for n in cut:
        cuts.append([(at, at + n)])
        at += n
    got = run_cut(lambda x, b: part.forward(x.to(torch.bfloat16).to(DEV), b, cache.view(0)), [x], cuts, [1])[0]
    close(got, pd.lightning(x, W, "m.", m, 1e-5) if kind == "lightning" else pd.mamba2(x, W, "m.", m["mixer"], 1e-5), 2e-2, f"cut {cut}")


@pytest.mark.parametrize("H,G,dk,dv,T", [(4, 4, 64, 64, 300), (8, 2, 64, 64, 300), (16, 2, 32, 24, 130), (8, 1, 24, 96, 70), (16, 1, 128, 64, 700), (8, 8, 20, 136, 65), (6, 3, 11, 9, 200)])
def test_chunked_memory_with_row_decays_keeps_sixteen_bits(H, G, dk, dv, T):
    """Outputs and last states of long portions against a float64 recurrence over the same float32 inputs: heads that share q
    and k in blocks of several, decays from nearly one to nearly zero within a chunk, several requests in one step."""
    from nano_vllm_cpp_b200.csrc import ops
    lengths = [T, 3, max(2, T // 2)]
    total = sum(lengths)
    src, z = rnd(81, total, H * dv + 2 * G * dk + 3).float(), 3.0 * rnd(82, total, H + 1).float()
    A, bias = rnd(83, H).float(), rnd(84, H).float()
    cols = {"v": 1, "k": 1 + H * dv, "q": 1 + H * dv + G * dk}
    S = torch.zeros(4, H, dk, dv, device=DEV)
    raw = torch.empty(total, H, dv, device=DEV)
    S0 = rnd(85, dk, dv).float()
    S[2, 0] = S0.to(DEV)                                 # the second request goes on from a state
    batch = batch_of([(1, 0, lengths[0]), (2, 9, lengths[1]), (0, 0, lengths[2])])
    ops.decayed_memory(src.to(DEV), cols, batch, S, H, dk, dv, raw, q_heads=G, steps=(z.to(DEV), 1, A.to(DEV), bias.to(DEV)))
    at = 0
    for e, n in enumerate(lengths):
        p, dt = src[at:at + n].double(), pd.softplus(z[at:at + n, 1:].double() + bias.double())
        for h in range(H):
            g = h // (H // G)
            st = S0.double().clone() if (e == 1 and h == 0) else torch.zeros(dk, dv, dtype=F64)
            o = torch.zeros(n, dv, dtype=F64)
            rate = math.exp(float(A[h]))
            for t in range(n):
                k, v = p[t, cols["k"] + g * dk:][:dk], p[t, cols["v"] + h * dv:][:dv]
                st = math.exp(-rate * float(dt[t, h])) * st + float(dt[t, h]) * torch.outer(k, v)
                o[t] = st.T @ p[t, cols["q"] + g * dk:][:dk]
            close(raw[at:at + n, h], o, 3e-4, f"request {e} head {h}")
            close(S[[1, 2, 0][e], h].reshape(1, -1), st.reshape(1, -1), 5e-5, f"state of request {e} head {h}")
        at += n


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gap,decoded", [(3, False), (64, False), (65, False), (250, False), (250, True), (640, True)])
def test_a_far_token_in_the_state(gap, decoded, dtype):
    """Row i asks for the key of row i - gap, which stands out (its input is row i's, enlarged, plus something that the keys do
    not see, so it has a value of its own): most of row i's output is that value, and without it the output is another one."""
    i = gap + 5
    T, width = i + 2, 128
    m = pd.lightning_part(2, 32, 32, [0.999, 0.9985])
    W = memory_weights("lightning", m, width, 31)
    W["m.q"] = W["m.k"].clone()
    x = 0.1 * rnd(32, T, width)
    x[i] = rnd(33, width)
    K, free = W["m.k"], rnd(34, width)
    free = free - K.T @ torch.linalg.solve(K @ K.T, K @ free)          # what the keys do not see
    x[i - gap] = 4.0 * (x[i] + 2.0 * free)
    x = x.to(torch.bfloat16).double()
    part, cache, _ = lightning_on(m, width, W, dtype)
    cuts = [[(0, T)]] if not decoded else [[(0, i - 2)]] + [[(t, t + 1)] for t in range(i - 2, T)]
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), [x], cuts, [2])[0]
    want = pd.lightning(x, W, "m.", m, 1e-5)
    close(got, want, 1e-4 if dtype == torch.float32 else 2e-2, "rows")
    without = x.clone()
    without[i - gap] = 0
    other = pd.lightning(without, W, "m.", m, 1e-5)
    assert float((other[i] - want[i]).abs().max()) > 0.2 * float(want[i].abs().max())


# ------------------------------------------------------------------------------- attention
def attention_on(m, width, W, dtype, fast=True, pages=64, page=16):
    from nano_vllm_cpp_b200.parts import PartSpec
    from nano_vllm_cpp_b200.models.dubarax import ATTENTION_NAMES, linear_slopes
    own = dict(window=m["mask"]["size"], score_softcap=m["softcap"], distance_far=m["bias_max"]) if "bias_max" in m else \
        dict(chunk=m["mask"]["size"], distance_slopes=linear_slopes(m["heads"]))
    return part_on("paged_attention", dict(
        hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], bias=True,
        out_bias=True, position=PartSpec("none"), scale=m["scale"], round_weights=True, names=ATTENTION_NAMES, **own), W, dtype, fast, pages)


def plain_attention(x, W, m, only=None):
    return (pd.window_attention if "bias_max" in m else pd.chunk_attention)(x, W, "m.", m, only)


def attention_weights(m, width, seed):
    if "bias_max" in m:
        return weights_of({"type": "attention", "mixer": m, "mlp": None}, width, seed)
    W = weights_of(pd.parallel_layer(left=m), width, seed)
    return {k.replace("m.left.", "m."): v for k, v in W.items() if k.startswith("m.left.")}


SIZES = [(4, 2, 32, 48, 0.2), (3, 3, 40, 24, 0.11), (8, 2, 64, 64, 0.125), (2, 2, 128, 128, 0.09), (6, 1, 96, 96, 0.1), (20, 1, 64, 32, 0.12),
         (2, 1, 256, 256, 0.06), (2, 1, 192, 80, 0.07), (1, 1, 8, 16, 0.5), (12, 2, 48, 40, 0.13), (17, 1, 144, 136, 0.08)]
MASKS = [("chunk", 20), ("chunk", 64), ("chunk", 1000), ("window", 19), ("window", 1), ("window", 400)]


@pytest.mark.parametrize("fast", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("k", range(len(SIZES)))
def test_attention_alone(k, dtype, fast):
    """Two requests on scattered pages, in portions beside single rows: grouped heads, values of another size than keys,
    biases, chunks with slopes, windows with a cap and a learned table."""
    H, G, D, V, scale = SIZES[k]
    width = 80
    for kind, size in (MASKS[k % 3], MASKS[3 + k % 3]):
        if kind == "chunk":
            m = pd.chunk_part(H, G, D, V, size, scale)
        else:
            m = pd.window_layer(H, G, D, V, size, scale * 4, cap=3.0 + k, far=[30, 50, 12][k % 3], rows=[10, 16, 7][k % 3])["mixer"]
        W = attention_weights(m, width, 41 + k)
        part, cache, ctx = attention_on(m, width, W, dtype, fast)
        xs = inputs(width, [66, 51], 42)
        got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [0, 1], PAGES)
        ctx.err.check("attention")
        for i, x in enumerate(xs):
            close(got[i], plain_attention(x, W, m), 1e-4 if dtype == torch.float32 else 3e-2, f"{kind} {size} request {i}")


@pytest.mark.parametrize("page", [16, 32, 128])
@pytest.mark.parametrize("D,H,G", [(16, 4, 2), (32, 8, 1), (48, 4, 4), (64, 17, 1), (112, 6, 2), (128, 4, 2), (256, 2, 1)])
def test_score_options_in_every_kernel(D, H, G, page):
    """Cap, slopes, table, chunk and window in every combination through each kernel that takes them: both prompt kernels, the
    decode kernel (all its forms: with a sink it gives a lane a chunk of a key), the general kernel."""
    from nano_vllm_cpp_b200.csrc import ops
    lengths = [150, 90, 1]
    pos0 = [0, 7, 200]
    T = sum(lengths)
    tables, nxt = [], 0
    for n, p in zip(lengths, pos0):
        need = (n + p + page - 1) // page
        tables.append([(3 * (nxt + i)) % 64 for i in range(need)])
        nxt += need
    assert nxt <= 64 and len({p for t in tables for p in t}) == nxt
    kc, vc = (rnd(s, 64, G, page, D).to(torch.bfloat16).to(DEV) for s in (1, 2))
    q = rnd(3, T, H * D).to(torch.bfloat16)
    batch = batch_of([(i, p, n) for i, (n, p) in enumerate(zip(lengths, pos0))], tables, max(len(t) for t in tables))
    bt = batch.block_tables[0]
    scale = 1.5 / math.sqrt(D)
    slopes, table = dev32(0.05 + 0.2 * rnd(4, H).abs()), dev32(2.0 * rnd(5, H, 41))
    padded = ops.bias_table_of(table)
    rows = [(e, p + t, r) for r, (e, p, t) in enumerate((e, p, t) for e, (n, p) in enumerate(zip(lengths, pos0)) for t in range(n))]
    picked = [x for x in rows if x[2] % 17 == 0 or x[0] == 2 or x[1] in (20, 21, 39, 40)]

    def plain(cap, sl, tb, window, chunk, sink):
        out = torch.zeros(len(picked), H, D, dtype=F64)
        for i, (e, p, r) in enumerate(picked):
            lo = pd.first_visible(p, ("chunk", chunk) if chunk else ("window", window) if window else None)
            at = [(tables[e][j // page], j % page) for j in range(lo, p + 1)]
            k = torch.stack([kc[b, :, s] for b, s in at]).double().cpu()
            v = torch.stack([vc[b, :, s] for b, s in at]).double().cpu()
            dist = torch.arange(p - lo, -1, -1)
            for h in range(H):
                s = (k[:, h // (H // G)] @ q[r, h * D:(h + 1) * D].double()) * scale
                s = cap * torch.tanh(s / cap) if cap else s
                s = s - slopes[h].double().cpu() * dist if sl else s
                s = s + table[h].double().cpu()[torch.clamp(dist, max=40)] if tb else s
                w = torch.exp(s - s.max())
                out[i, h] = (w @ v[:, h // (H // G)]) / (w.sum() + (math.exp(-float(s.max())) if sink else 0))
        return out.reshape(len(picked), -1)

    at = [r for _, _, r in picked]
    single = [i for i, x in enumerate(picked) if x[0] == 2]
    for case, (cap, sl, tb, window, chunk, sink) in enumerate([(4.0, 0, 1, 33, 0, 0), (0, 1, 0, 0, 40, 0), (6.0, 1, 1, 0, 21, 0), (0, 0, 1, 0, 0, 0),
                                                              (3.0, 0, 0, 0, 500, 0), (0, 0, 0, 0, 64, 0), (5.0, 1, 0, 77, 0, 1)]):
        want = plain(cap, sl, tb, window, chunk, sink)
        opts = dict(softcap=cap, chunk=chunk, slopes=slopes if sl else None, bias_table=padded if tb else None, sink_score=0.0 if sink else None)
        err = ops.ErrorFlag(DEV)
        qd = q.to(DEV)
        for kernel, terms in (("auto", 1), ("auto", 3), ("mma", 1), ("mma", 3)):
            out = torch.zeros(T, H * D, dtype=torch.bfloat16, device=DEV)
            ops.attention_prefill(qd, kc, vc, bt, batch.cu_rows, batch.entry_pos0, T // 64 + 3, scale, window, out, H, G, D, err=err,
                                  kernel=kernel, weight_terms=terms, **opts)
            close(out[at], want, 2e-2, f"case {case} prompt {kernel} {terms}")
        for exact in (False, True) if ops.attention_decode_usable(kc, D) else ():
            out = torch.zeros(T, H * D, dtype=torch.bfloat16, device=DEV)
            ops.attention_decode(qd, kc, vc, bt, batch.row_entry, batch.positions, scale, window, out, H, G, D, 201, rows=batch.single_rows,
                                 err=err, float_weights=exact, **opts)
            close(out[at][single], want[single], 2e-2, f"case {case} decode {exact}")
        out = torch.zeros(T, H * D, dtype=torch.float32, device=DEV)
        ops.paged_attention_general(qd, kc, vc, bt, batch.row_entry, batch.positions, scale, window, out, H, G, D, D, **opts)
        close(out[at], want, 1e-5, f"case {case} general")
        err.check("attention")


def standing_out(m, width, T, i, j, seed):
    """(inputs, weights): row i's query meets key j with a score far above all others (row j's input is row i's plus something
    that the key projection does not see, so its key is the same and its value another)."""
    W = attention_weights(m, width, seed)
    G, D = m["kv_heads"], m["dim"]
    W["m.q"] = W["m.k"].view(G, D, width).repeat_interleave(m["heads"] // G, dim=0).reshape(-1, width)
    W["m.q.b"], W["m.k.b"] = torch.zeros_like(W["m.q.b"]), torch.zeros_like(W["m.k.b"])
    x = rnd(seed + 1, T, width)
    K = W["m.k"]
    free = rnd(seed + 2, width)
    free = free - K.T @ torch.linalg.solve(K @ K.T, K @ free)          # what the keys do not see
    x[j] = x[i] + 2.0 * free * (x[i].norm() / free.norm())
    return x.to(torch.bfloat16).double(), W


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dim", [32, 64, 96])
@pytest.mark.parametrize("kind,size,i,j,seen", [
    ("window", 50, 120, 71, True), ("window", 50, 120, 70, False), ("window", 64, 200, 137, True), ("window", 64, 200, 136, False),
    ("window", 33, 330, 298, True), ("window", 33, 330, 297, False), ("window", 600, 600, 1, True), ("window", 600, 600, 0, False),
    ("window", 1000, 330, 0, True), ("window", 1000, 700, 63, True), ("window", 1000, 700, 64, True),
    ("chunk", 50, 149, 100, True), ("chunk", 50, 149, 99, False), ("chunk", 50, 100, 99, False), ("chunk", 64, 191, 128, True),
    ("chunk", 64, 192, 191, False), ("chunk", 37, 300, 296, True), ("chunk", 37, 300, 295, False), ("chunk", 400, 700, 400, True),
    ("chunk", 400, 700, 399, False), ("chunk", 400, 150, 0, True)])
def test_one_key_stands_out(kind, size, i, j, seen, dim, decoded, dtype):
    """A key just inside and just outside a window or a chunk, at the first tokens, at page and tile borders, hundreds of
    positions back among scattered pages; in a prompt, and decoded after single rows.  Hiding a seen key changes the row by
    far more than the tolerance; a key outside changes nothing."""
    T, width = i + 3, 3 * dim
    if kind == "window":
        m = pd.window_layer(2, 1, dim, dim, size, 3.0 / math.sqrt(dim), cap=60.0, far=300, rows=16)["mixer"]
    else:
        m = pd.chunk_part(16, 8, dim, dim, size, 8.0 / math.sqrt(dim))
    x, W = standing_out(m, width, T, i, j, 51)
    rows = list(range(i - 2, T))
    hidden = x.clone()
    hidden[j] = rnd(57, width).to(torch.bfloat16).double()
    want, other = plain_attention(x, W, m, rows), plain_attention(hidden, W, m, rows)
    moved = float((other[2] - want[2]).abs().max()) / float(want[2].abs().max())
    assert moved > 0.2 if seen else moved == 0.0, moved
    if not seen:                                    # ... and is inside by the wrong rule: the row before it, or the same key
        near = plain_attention(x, W, dict(m, mask={"size": size + 1 if kind == "window" else 10 ** 6}), rows)
        assert float((near[2] - want[2]).abs().max()) > 0.1 * float(want[2].abs().max())
    part, cache, ctx = attention_on(m, width, W, dtype)
    n_pages = (T + 15) // 16
    table = [(11 * p + 3) % 61 for p in range(n_pages)]
    assert len(set(table)) == n_pages
    cuts = [[(0, T)]] if not decoded else [[(0, i - 2)]] + [[(t, t + 1)] for t in range(i - 2, T)]
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), [x], cuts, [0], [table])[0]
    ctx.err.check("attention")
    close(got[rows], want, 2e-4 if dtype == torch.float32 else 4e-2, "rows")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decoded", [False, True])
def test_every_row_of_the_distance_table_counts(decoded, dtype):
    """A table with one large entry per head: head h attends to one bucket of distances almost alone; the same cap without
    the bias behind it would hide that."""
    rows, far, T = 8, 60, 130
    m = pd.window_layer(8, 2, 32, 32, 120, 0.05, cap=1.0, far=far, rows=rows)["mixer"]
    W = attention_weights(m, 64, 61)
    W["m.rel"] = 12.0 * torch.eye(rows, dtype=F64)
    x = inputs(64, [T], 62)[0]
    part, cache, ctx = attention_on(m, 64, W, dtype)
    cuts = [[(0, T)]] if not decoded else [[(0, 5)]] + [[(t, t + 1)] for t in range(5, T)]
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), [x], cuts, [0], [list(range(9))])[0]
    close(got, plain_attention(x, W, m), 1e-4 if dtype == torch.float32 else 2e-2, "rows")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_mixers_side_by_side_with_scales(dtype):
    from nano_vllm_cpp_b200.models import dubarax
    from nano_vllm_cpp_b200.config.dubarax_config import DubaraxConfig
    from nano_vllm_cpp_b200.parts import build_part
    from nano_vllm_cpp_b200.cache import DeviceCache
    layer = pd.parallel_layer(pd.chunk_part(4, 2, 32, 16, size=23), pd.lightning_part(2, 24, 40), 0.8, -0.35)
    cfg = DubaraxConfig.from_dict(pd.model_config([layer], width=80, vocab=8))
    part = build_part("mixer", dubarax._mixer(cfg, cfg.layers[0].mixer))
    W = weights_of(layer, 80, 65)
    part.load(Fetch(W, "m.", dtype), ctx_for(dtype))
    cache = DeviceCache([part.cache_spec()], 16, 4, DEV, dtype)
    cache.allocate(16, 16)
    xs = inputs(80, [66, 51], 66)
    got = run_cut(lambda x, b: part.forward(x.to(dtype).to(DEV), b, cache.view(0)), xs, CUTS, [2, 1], PAGES)
    for i, x in enumerate(xs):
        close(got[i], pd.side_by_side(x, W, "m.", layer["mixer"], 1e-5), 1e-4 if dtype == torch.float32 else 2e-2, f"request {i}")


# ------------------------------------------------------------------------------- whole models through the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_the_stream_layer_by_layer(name, dtype, models):
    """The stream after every layer run, the looped ones once per pass."""
    from nano_vllm_cpp_b200.engine.batch import StepEntry
    cfg, W, folder = models[name]
    ids = ids_for(name, 37, salt=3)
    want, margins, got = [], [], []
    pd.forward(cfg, W, ids, layer_sums=want, margins=margins)
    runner = make_runner(folder, dtype, 64)

    def look(i, x, pending):
        y = pending
        if not isinstance(y, torch.Tensor):
            y = type(pending)(pending.first.clone(), *list(vars(pending).values())[1:]).sum() if hasattr(pending, "first") else pending.sum()
        got.append((x + y).cpu())

    runner.model.after_call = look
    runner.step([StepEntry("x", ids, [])])
    assert len(got) == len(want) == len(pd.layer_runs(cfg))
    half = dtype == "bfloat16"
    edge = torch.stack(margins).min(dim=0).values if margins and half else None
    errors = pd.rounding_errors(cfg, W, ids, NOISE, layer=True) if half else [None] * len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        close(g, w, 3e-2 if half else 2e-5, f"layer run {i}", edge, errors[i])


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
    """A model of drawn sizes: layer order, mixers' sizes, masks, feed-forwards and the loop."""
    rng = random.Random(seed)
    layers = []
    for i in range(rng.randint(3, 5)):
        ff = None
        if rng.random() < 0.8:
            count = rng.choice([1, 2, 4])
            n = rng.choice([1, 2, 3])
            keep = rng.randint(1, count)
            ff = pd.moe(count * n, rng.randint(1, keep * n), rng.choice([16, 24, 32, 64]), count, keep, rng.choice([0, 16, 40, 64]))
        kind, suffix = rng.choice(["parallel", "attention", "mamba2"]), rng.choice(["", "_2", "_3"])
        kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 16, 24, 40, 48, 64, 96, 128])
        heads = kv * rng.choice([1, 2, 4])
        if kind == "parallel":
            n = rng.choice([1, 2, 3])
            layers.append(pd.parallel_layer(pd.chunk_part(heads, kv, dim, rng.choice([dim, 32]), rng.choice([5, 16, 31, 48, 180]), rng.uniform(0.1, 0.3)),
                                            pd.lightning_part(n, rng.choice([16, 24, 64, 80]), rng.choice([16, 40, 64, 96]), [rng.uniform(0.5, 1.0) for _ in range(n)]),
                                            rng.uniform(0.3, 1.2), rng.uniform(0.3, 1.2), mlp=ff, type=kind + suffix))
        elif kind == "attention":
            layers.append(pd.window_layer(heads, kv, dim, rng.choice([dim, 32]), rng.choice([1, 7, 16, 40, 100]), rng.uniform(0.1, 0.4), rng.uniform(2.0, 40.0),
                                          rng.choice([20, 64, 100]), rng.choice([4, 7, 16]), mlp=ff, type=kind + suffix))
        else:
            g = rng.choice([1, 2, 3])
            h, v = g * rng.choice([1, 2, 4]), rng.choice([8, 16, 24, 64])
            parts = rng.choice([p for p in (1, 2, 3, 4, 6) if (h * v) % p == 0])
            layers.append(pd.mamba_layer(h, v, rng.choice([8, 20, 64, 128]), g, rng.choice([1, 2, 3, 4, 5]), parts, mlp=ff, type=kind + suffix))
    n = len(layers)
    a = rng.randint(0, n - 1)
    loop = (a, rng.randint(a + 1, n), rng.choice([1, 2, 3])) if rng.random() < 0.8 else None
    return pd.model_config(layers, width=rng.choice([48, 64, 72, 128]), vocab=rng.choice([97, 160]), eps=rng.choice([1e-6, 1e-4]),
                           embed_scale=rng.uniform(0.5, 6.0), loop=loop)


@pytest.mark.parametrize("seed", range(12))
def test_drawn_models_in_a_mixed_schedule(seed, tmp_path):
    cfg = drawn_config(seed)
    W = pd.make_weights(cfg, 100 + seed)
    folder = pd.write_folder(cfg, W, str(tmp_path))
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
            want = pd.forward(cfg, W, toks, margins=margins)
            half = dtype == "bfloat16"
            close(st.rows(r, len(toks)), want, TOL[dtype], f"drawn model {seed} {dtype} request {r}",
                  torch.stack(margins).min(dim=0).values if margins and half else None,
                  (lambda: pd.rounding_errors(cfg, W, toks, NOISE)) if half else None)


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
        close(r, runs[0], 2e-5 if dtype == "float32" else 3e-2, "the same rows cut another way", margins if dtype == "bfloat16" else None,
              (lambda: rounding_errors(models, name, ids)) if dtype == "bfloat16" else None)


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
            logits = pd.forward(cfg, W, seq)[-1]
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
    assert toks == pd.greedy_generate(cfg, W, prompt, 6)
    path = tmp_path / "config.json"
    path.write_text(json.dumps(CONFIGS["M"]))
    rc = cli.main(["--config", str(path), "--seed", "4", "--tokens", "5,6,7", "--max-tokens", "4", "--temperature", "0",
                   "--max-model-len", "64", "--num-kv-blocks", "8", "--ignore-eos"])
    out = capsys.readouterr().out
    assert rc == 0 and len(out.strip().splitlines()[-1].split(":")[1].split()) == 4
