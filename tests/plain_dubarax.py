"""Plain, slow implementation of the Dubarax decoder: whole sequences, no cache, one function per mechanism, float64
arithmetic on bfloat16-rounded weight values.  It shares no code with the package: it reads the configuration as a
dict, makes and writes its own weights, and loops over heads and tokens.

Notation.  ``rms(v) = v / sqrt(mean(v^2) + eps)``; ``h`` is the [tokens, width] matrix a sublayer reads.  A layer is
``x <- x + mixer(rms(x) (1 + g1))`` and, where it has one, ``x <- x + ff(rms(x) (1 + g2))``.  A stretch of layers may run
several times with the same weights; ahead of pass t stands ``x <- A x + B x0 + s_t`` with x0 the embedding rows.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np
import torch

F64 = torch.float64


# ------------------------------------------------------------------------------ small functions
def unit_rms(x, eps):
    """Every row divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_one_plus(x, g, eps):
    return unit_rms(x, eps) * (1.0 + g)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_convolution(u, w, b):
    """y[t, c] = b[c] + sum_j w[c, j] u[t - (taps - 1) + j, c]; nothing before the first token."""
    T, taps = u.shape[0], w.shape[1]
    y = b[None, :].repeat(T, 1)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


# ------------------------------------------------------------------------------ attention
def first_visible(i, mask):
    """The first position that row i sees.  ``mask``: ("window", n), ("chunk", n) or None."""
    if mask is None:
        return 0
    kind, n = mask
    if kind == "window":
        return max(0, i - n + 1)
    return (i // n) * n


def linear_bias(heads):
    """Per head, what a distance of one takes off the score."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def bucket_of(n, rows, far):
    """Distances below half of the rows have a row each; the others share the rest on a logarithmic scale that ends at
    ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def attention(h, W, p, m, mask, cap=0.0, slopes=None, table=None, far=0, only=None):
    """Grouped-query softmax attention with biased projections: a score is ``scale q.k``, then capped, then changed by what
    the distance gives (``slopes`` per head, or a learned ``table`` [rows, heads] read through ``bucket_of``).  ``only``: just
    these rows are worked out and returned."""
    T, H, G, D = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    V = int(m.get("vdim", D))
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, V)
    out = torch.zeros(T, H, V, dtype=F64)
    rows = [bucket_of(n, table.shape[0], far) for n in range(T)] if table is not None else None
    for i in range(T) if only is None else only:
        lo = first_visible(i, mask)
        dist = [i - j for j in range(lo, i + 1)]
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * float(m["scale"])
            if cap:
                s = cap * torch.tanh(s / cap)
            if slopes is not None:
                s = s - slopes[hd] * torch.tensor(dist, dtype=F64)
            if table is not None:
                s = s + table[[rows[n] for n in dist], hd]
            out[i, hd] = torch.softmax(s, dim=0) @ v[lo:i + 1, g]
    out = out.reshape(T, H * V) if only is None else out.reshape(T, H * V)[only]
    return out @ W[p + "o"].T + W[p + "o.b"]


def chunk_attention(h, W, p, m, only=None):
    return attention(h, W, p, m, ("chunk", int(m["mask"]["size"])), slopes=linear_bias(int(m["heads"])), only=only)


def window_attention(h, W, p, m, only=None):
    return attention(h, W, p, m, ("window", int(m["mask"]["size"])), cap=float(m["softcap"]), table=W[p + "rel"],
                     far=int(m["bias_max"]), only=only)


# ------------------------------------------------------------------------------ matrix memories
def lightning(h, W, p, m, eps, final_state=None):
    """Per head S <- d S + k v^T, o = S^T q with silu on q, k and v; the row of all heads over its root mean square, times a
    weight and a sigmoid gate.  ``final_state``: a list that receives the last S [heads, dim, vdim]."""
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = silu(h @ W[p + "q"].T).view(T, H, D), silu(h @ W[p + "k"].T).view(T, H, D)
    v = silu(h @ W[p + "v"].T).view(T, H, V)
    out, last = torch.zeros(T, H, V, dtype=F64), torch.zeros(H, D, V, dtype=F64)
    for hd in range(H):
        S = torch.zeros(D, V, dtype=F64)
        for t in range(T):
            S = float(m["decay"][hd]) * S + torch.outer(k[t, hd], v[t, hd])
            out[t, hd] = S.T @ q[t, hd]
        last[hd] = S
    if final_state is not None:
        final_state.append(last)
    y = unit_rms(out.reshape(T, H * V), eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def mamba2(h, W, p, m, eps, final_state=None):
    """Per head S <- exp(-exp(a) dt) S + dt b x^T, y = S^T c + D x, with x, b and c behind a short convolution and silu; the
    gate silu(z) comes before the norm, which is taken over equal parts of the row."""
    T, H, V, N, G = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner, bc = H * V, G * N
    u = h @ W[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * bc], u[:, 2 * inner + 2 * bc:]
    xbc = silu(causal_convolution(xbc, W[p + "conv"], W[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, V)
    b = xbc[:, inner:inner + bc].reshape(T, G, N)
    c = xbc[:, inner + bc:].reshape(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"])
    y, last = torch.zeros(T, H, V, dtype=F64), torch.zeros(H, N, V, dtype=F64)
    for hd in range(H):
        g, rate = hd // (H // G), math.exp(float(W[p + "A_log"][hd]))
        S = torch.zeros(N, V, dtype=F64)
        for t in range(T):
            S = math.exp(-rate * float(dt[t, hd])) * S + float(dt[t, hd]) * torch.outer(b[t, g], x[t, hd])
            y[t, hd] = S.T @ c[t, g] + W[p + "D"][hd] * x[t, hd]
        last[hd] = S
    if final_state is not None:
        final_state.append(last)
    y = y.reshape(T, inner) * silu(z)
    parts = int(m["norm_groups"])
    y = unit_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * W[p + "norm"]
    return y @ W[p + "o"].T


def side_by_side(h, W, p, m, eps):
    return (float(m["left_scale"]) * chunk_attention(h, W, p + "left.", m["left"])
            + float(m["right_scale"]) * lightning(h, W, p + "right.", m["right"], eps))


def mixer(h, W, p, L, eps):
    kind = L["type"]
    if kind.startswith("parallel"):
        return side_by_side(h, W, p, L["mixer"], eps)
    if kind.startswith("mamba2"):
        return mamba2(h, W, p, L["mixer"], eps)
    return window_attention(h, W, p, L["mixer"])


# ------------------------------------------------------------------------------ the feed-forward
def glu(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(s, r):
    """One row's scores -> [(expert, weight)]: of the groups of neighbouring experts those ``keep`` with the largest
    member, then the ``top`` largest of their experts (the lower index on a tie), each with its score."""
    E, K = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    n = E // int(groups["count"])
    best = [max(s[g * n:(g + 1) * n]) for g in range(int(groups["count"]))]
    kept = sorted(range(len(best)), key=lambda g: (-best[g], g))[:int(groups["keep"])]
    allowed = [e for e in range(E) if e // n in kept]
    return [(e, s[e]) for e in sorted(allowed, key=lambda e: (-s[e], e))[:K]]


def route_margin(z, r):
    """How far a row's routing is from another one, in units of the logits' spread: the gap between the last group kept
    and the first left out, and between the last expert chosen and the best one left out of the kept groups."""
    E, K = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    n, keep = E // int(groups["count"]), int(groups["keep"])
    spread = max(z) - min(z) if E > 1 else 1.0
    best = sorted((max(z[g * n:(g + 1) * n]) for g in range(int(groups["count"]))), reverse=True)
    gaps = [best[keep - 1] - best[keep]] if keep < len(best) else []
    order = sorted(range(len(best)), key=lambda g: (-max(z[g * n:(g + 1) * n]), g))[:keep]
    allowed = sorted((z[e] for e in range(E) if e // n in order), reverse=True)
    if K < len(allowed):
        gaps.append(allowed[K - 1] - allowed[K])
    return min(gaps) / max(spread, 1e-9) if gaps else math.inf


def mixture(h, W, p, mlp, margins=None):
    z = h @ W[p + "router"].T
    scores = torch.softmax(z, dim=1).tolist()
    out = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=F64)
    for t in range(h.shape[0]):
        for e, w in route(scores[t], mlp["router"]):
            out[t] += w * glu(h[t:t + 1], W, f"{p}e{e}.")[0]
    if margins is not None:
        margins.append(torch.tensor([route_margin(r, mlp["router"]) for r in z.tolist()], dtype=F64))
    if mlp.get("shared"):
        out = out + glu(h, W, p + "shared.")
    return out


# ------------------------------------------------------------------------------ the whole model
def layer_runs(cfg):
    """[(layer, pass index or None)] in running order; the pass index stands at the first layer of every pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    runs = [(i, None) for i in range(a)]
    for t in range(int(loop["times"])):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, W, tokens, layer_sums=None, margins=None, noise=None):
    """Logits [T, vocab] of a whole sequence.  ``layer_sums``: a list that receives the stream after every layer run;
    ``margins``: a list that receives every router's margins; ``noise`` = (generator, size): what every sublayer reads
    and gives is multiplied by 1 + size * N(0, 1), element by element, as roundings would change it."""

    def noisy(t):
        return t if noise is None else t * (1.0 + noise[1] * torch.randn(t.shape, generator=noise[0], dtype=F64))

    eps = float(cfg["norm"]["eps"])
    x0 = W["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    x = x0
    for i, t in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = torch.cat([noisy(x), noisy(x0)], dim=1) @ W["loop.in"].T + W["loop.step"][t]
        x = x + noisy(mixer(noisy(norm_one_plus(x, W[p + "norm1"], eps)), W, p + "mix.", L, eps))
        if L.get("mlp"):
            x = x + noisy(mixture(noisy(norm_one_plus(x, W[p + "norm2"], eps)), W, p + "mlp.", L["mlp"], margins))
        if layer_sums is not None:
            layer_sums.append(x)
    return noisy(norm_one_plus(x, W["final.norm"], eps)) @ W["head"].T


def rounding_errors(cfg, W, tokens, size, draws=4, layer=None):
    """Per row, the largest change of the logits (or of the stream after every layer run) that roundings of the relative
    size ``size`` cause."""
    def run(noise):
        sums = []
        lg = forward(cfg, W, tokens, layer_sums=sums, noise=noise)
        return sums if layer else [lg]

    want = run(None)
    worst = [torch.zeros(len(tokens), dtype=F64) for _ in want]
    for d in range(draws):
        for i, got in enumerate(run((torch.Generator().manual_seed(d), size))):
            worst[i] = torch.maximum(worst[i], (got - want[i]).abs().max(dim=1).values)
    return worst if layer else worst[0]


def greedy_generate(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(torch.argmax(forward(cfg, W, seq)[-1])))
    return seq[len(prompt):]


# ------------------------------------------------------------------------------ weights

def tensor_table(cfg):
    """name -> (shape, kind) of every tensor the model has; kinds: embed, matrix, vector (a bias), shift (around zero), gain
    (around one), taps, table, rate, step, router."""
    Wd, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": ((V, Wd), "embed"), "head": ((V, Wd), "matrix"), "final.norm": ((Wd,), "shift")}
    if cfg.get("loop"):
        out["loop.in"], out["loop.step"] = ((Wd, 2 * Wd), "matrix"), ((int(cfg["loop"]["times"]), Wd), "step")

    def attn(x, m):
        H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
            out[x + n], out[x + n + ".b"] = ((rows, Wd), "matrix"), ((rows,), "vector")
        out[x + "o"], out[x + "o.b"] = ((Wd, H * Dv), "matrix"), ((Wd,), "vector")
        if "bias_max" in m:
            out[x + "rel"] = ((int(m.get("_rows", 12)), H), "table")

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        out[p + "norm1"] = ((Wd,), "shift")
        if L["type"].startswith("parallel"):
            attn(x + "left.", m["left"])
            r = m["right"]
            H, D, Dv = int(r["heads"]), int(r["dim"]), int(r["vdim"])
            x += "right."
            out[x + "q"], out[x + "k"] = ((H * D, Wd), "matrix"), ((H * D, Wd), "matrix")
            out[x + "v"], out[x + "g"] = ((H * Dv, Wd), "matrix"), ((H * Dv, Wd), "matrix")
            out[x + "o"], out[x + "norm"] = ((Wd, H * Dv), "matrix"), ((H * Dv,), "gain")
        elif L["type"].startswith("mamba2"):
            H, Dv, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
            inner, ch = H * Dv, H * Dv + 2 * G * N
            out[x + "in"] = ((inner + ch + H, Wd), "matrix")
            out[x + "conv"], out[x + "conv.b"] = ((ch, int(m["conv"])), "taps"), ((ch,), "vector")
            out[x + "dt_bias"], out[x + "A_log"], out[x + "D"] = ((H,), "rate"), ((H,), "rate"), ((H,), "gain")
            out[x + "norm"], out[x + "o"] = ((inner,), "gain"), ((Wd, inner), "matrix")
        else:
            attn(x, m)
        f = L.get("mlp")
        if f:
            out[p + "norm2"] = ((Wd,), "shift")
            y, ff = p + "mlp.", int(f["expert"]["ff"])
            names = [(f"{y}e{e}.", ff) for e in range(int(f["router"]["experts"]))]
            if f.get("shared"):
                names.append((y + "shared.", int(f["shared"]["ff"])))
            out[y + "router"] = ((int(f["router"]["experts"]), Wd), "router")
            for z, n in names:
                out[z + "gate"], out[z + "up"], out[z + "down"] = ((n, Wd), "matrix"), ((n, Wd), "matrix"), ((Wd, n), "matrix")
    return out


def make_weights(cfg, seed, scale=1.0):
    """bfloat16-rounded values as float64: matrices N(0, scale / sqrt(columns))."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, (shape, kind) in sorted(tensor_table(cfg).items()):
        z = torch.randn(shape, generator=g, dtype=F64)
        if kind == "matrix":
            t = z * scale / math.sqrt(shape[-1])
        elif kind == "embed":
            t = z * 0.5
        elif kind == "gain":
            t = 1.0 + 0.2 * z
        elif kind in ("shift", "vector"):
            t = 0.2 * z
        elif kind == "rate":
            t = 0.5 * z - 1.0
        elif kind == "table":
            t = 1.0 * z
        elif kind == "router":
            t = z * 1.5 / math.sqrt(shape[-1])
        elif kind == "step":
            t = 0.7 * z
        else:
            t = 0.4 * z
        W[name] = t.to(torch.bfloat16).double()
    return W


def write_folder(cfg, W, path):
    """config.json and model.safetensors (bfloat16) in ``path``, written here byte by byte."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    head, blobs, at = {}, [], 0
    for name in sorted(W):
        t = W[name].to(torch.bfloat16).contiguous()
        raw = t.view(torch.int16).numpy().astype("<i2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for b in blobs:
            f.write(b)
    return path


def read_folder(path):
    """(cfg, float64 weights) of a folder in the bfloat16 safetensors format."""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    W = {}
    for name, info in head.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        raw = np.frombuffer(data[a:b], dtype="<i2").copy()
        W[name] = torch.from_numpy(raw).view(torch.bfloat16).reshape(info["shape"]).double()
    return cfg, W


# ------------------------------------------------------------------------------ configurations
def chunk_part(heads=4, kv_heads=2, dim=32, vdim=None, size=20, scale=0.2):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim,
            "mask": {"size": size}, "scale": scale}


def lightning_part(heads=2, dim=32, vdim=None, decay=None):
    return {"heads": heads, "dim": dim, "vdim": dim if vdim is None else vdim,
            "decay": [1.0 - 2.0 ** (-2 - i) for i in range(heads)] if decay is None else list(decay)}


def parallel_layer(left=None, right=None, left_scale=0.7, right_scale=1.1, mlp=None, type="parallel"):
    return {"type": type, "mlp": mlp, "mixer": {"left": left or chunk_part(), "right": right or lightning_part(),
                                                "left_scale": left_scale, "right_scale": right_scale}}


def window_layer(heads=4, kv_heads=2, dim=32, vdim=None, size=24, scale=0.2, cap=20.0, far=40, rows=12, mlp=None,
                 type="attention"):
    """``rows``: of the learned table.  A configuration file does not have that number (it is the tensor's first size); it
    travels here under a key that no reader looks at."""
    return {"type": type, "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim,
                      "mask": {"size": size}, "scale": scale, "softcap": cap, "bias_max": far, "_rows": rows}}


def mamba_layer(heads=4, vdim=16, state=24, groups=2, conv=4, norm_groups=2, mlp=None, type="mamba2"):
    return {"type": type, "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                "conv": conv, "norm_groups": norm_groups}}


def moe(experts=8, top=2, ff=24, count=4, keep=2, shared=40):
    f = {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
         "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def model_config(layers, width=64, vocab=150, eps=1e-5, embed_scale=2.5, loop=None):
    cfg = {"architecture": "Dubarax", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": embed_scale}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg
