"""Plain, slow implementation of the Sevelorn decoder: whole sequences, no cache, one function per mechanism, float64
arithmetic on bfloat16-rounded weight values.  It shares no code with the package: it reads the configuration as a
dict, makes and writes its own weights, and loops over heads and tokens.

Notation.  The model keeps ``n`` copies of the residual stream, ``X[t, c]`` (token t, copy c), all equal to the
token's embedding row times a constant at the start.  A sublayer F with its three small tensors ``r`` (read, [n]),
``M`` (carry, [n, n], indexed [from, to]) and ``w`` (write, [n]) does

    u = sum_c r[c] X[:, c];   y = F(rms(u) (1 + g));   X'[:, d] = sum_c M[c, d] X[:, c] + w[d] y

and what a mixer reads is ``h + conv(h)``, conv a causal convolution over time on every channel.  After the last layer
the copies are summed, normed once more and projected by ``head``.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_convolution(h, w):
    """y[t, c] = sum_j w[c, j] h[t - (taps - 1) + j, c]; nothing before the first token."""
    T, taps = h.shape[0], w.shape[1]
    y = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * h[s]
    return y


def rotate_halves(x, positions, rot):
    """x [T, heads, dim]: element i < dims / 2 is paired with element i + dims / 2; the pair at position p is turned by
    p * base^(-2i / dims).  Elements from ``dims`` on pass unchanged."""
    if not rot or int(rot["dims"]) == 0:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = torch.tensor(positions, dtype=F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    a, b = x[..., :half], x[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


# ------------------------------------------------------------------------------ the mixers
def retention(h, W, p, m, eps, final_state=None):
    """Per head: S <- d S + k v^T, o = S^T q, a fixed decay d; q and k turned, k divided by sqrt(dim); o divided by its
    root mean square; the heads side by side times silu(g h), then projected.  ``final_state``: a list that receives
    the last S [heads, dim, vdim]."""
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"]))
    pos = list(range(T))
    q = rotate_halves((h @ W[p + "q"].T).view(T, H, D), pos, m.get("rot"))
    k = rotate_halves((h @ W[p + "k"].T).view(T, H, D), pos, m.get("rot")) / math.sqrt(D)
    v = (h @ W[p + "v"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=F64)
    last = torch.zeros(H, D, V, dtype=F64)
    for hd in range(H):
        S = torch.zeros(D, V, dtype=F64)
        for t in range(T):
            S = float(m["decay"][hd]) * S + torch.outer(k[t, hd], v[t, hd])
            out[t, hd] = S.T @ q[t, hd]
        last[hd] = S
    if final_state is not None:
        final_state.append(last)
    y = unit_rms(out, eps).reshape(T, H * V) * silu(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def keys_and_values(h, W, p, m, eps):
    """What a layer that makes its own keys and values keeps: the keys normed over all kv heads' rows at once."""
    T, G, D, V = h.shape[0], int(m["kv_heads"]), int(m["dim"]), int(m.get("vdim", m["dim"]))
    k = (unit_rms(h @ W[p + "k"].T, eps) * W[p + "k.norm"]).view(T, G, D)
    return k, (h @ W[p + "v"].T).view(T, G, V)


def attention(h, W, p, m, eps, kv):
    """Causal softmax attention without positions over ``kv`` = (k, v); the queries normed over all heads' rows at once;
    every head's output times one sigmoid of the row."""
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (unit_rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]).view(T, H, D)
    k, v = kv
    gate = torch.sigmoid(h @ W[p + "g"].T)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        for t in range(T):
            w = torch.softmax((k[:t + 1, g] @ q[t, hd]) * float(m["scale"]), dim=0)
            out[t, hd] = gate[t, hd] * (w @ v[:t + 1, g])
    return out.reshape(T, -1) @ W[p + "o"].T


# ------------------------------------------------------------------------------ the feed-forwards
def glu(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, r):
    """Per token: z = router h + bias; the ``top`` largest (the lower index on a tie), weighed by their own softmax."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    E, K = int(r["experts"]), int(r["top"])
    picks = []
    for t in range(h.shape[0]):
        order = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:K]
        w = torch.softmax(z[t, order], dim=0)
        picks.append([(e, float(w[i])) for i, e in enumerate(order)])
    return picks, z


def choice_margins(z, K):
    """Per token: how far the last chosen expert's logit lies above the first one left out (inf if none is)."""
    if K >= z.shape[1]:
        return torch.full((z.shape[0],), float("inf"), dtype=F64)
    top = torch.sort(z, dim=1, descending=True).values
    return top[:, K - 1] - top[:, K]


def mixture(h, W, p, mlp, margins=None):
    picks, z = route(h, W, p, mlp["router"])
    if margins is not None:
        margins.append(choice_margins(z, int(mlp["router"]["top"])))
    out = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=F64)
    for t, chosen in enumerate(picks):
        for e, w in chosen:
            out[t] += w * glu(h[t:t + 1], W, f"{p}e{e}.", silu)[0]
    return out


def feed_forward(h, W, p, mlp, margins=None):
    return glu(h, W, p, gelu_tanh) if mlp["kind"] == "dense" else mixture(h, W, p, mlp, margins)


# ------------------------------------------------------------------------------ the copies of the stream
def connected(X, W, p, g, eps, F):
    """One sublayer around the copies X [T, n, width]; ``p`` names its read / carry / write tensors, ``g`` its norm's."""
    r, M, w = W[p + "in"], W[p + "mix"], W[p + "out"]
    u = torch.einsum("c,tcw->tw", r, X)
    y = F(norm_one_plus(u, W[g], eps))
    return torch.einsum("cd,tcw->tdw", M, X) + w[None, :, None] * y[:, None, :]


# ------------------------------------------------------------------------------ the whole model
def forward(cfg, W, tokens, layer_sums=None, margins=None, noise=None):
    """Logits [T, vocab] of a whole sequence.  ``layer_sums``: a list that receives the sum of the copies after every
    layer; ``margins``: a list that receives every router's ``choice_margins``; ``noise`` = (generator, size): what every
    sublayer reads and gives is multiplied by 1 + size * N(0, 1), element by element, as roundings would change it."""

    def noisy(t):
        return t if noise is None else t * (1.0 + noise[1] * torch.randn(t.shape, generator=noise[0], dtype=F64))

    n, eps = int(cfg.get("streams", 1)), float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    X = x[:, None, :].repeat(1, n, 1)
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]

        def mixer(h):
            h = noisy(h + causal_convolution(h, W[p + "canon1"]))
            if L["type"].startswith("retention"):
                return retention(h, W, p + "mix.", m, eps)
            j = m.get("kv_from")
            if j is None:
                kept[i] = keys_and_values(h, W, p + "mix.", m, eps)
            return attention(h, W, p + "mix.", m, eps, kept[i if j is None else int(j)])

        X = connected(X, W, p + "hc1.", p + "norm1", eps, lambda h: noisy(mixer(h)))
        if L.get("mlp"):
            X = connected(X, W, p + "hc2.", p + "norm2", eps,
                          lambda h: noisy(feed_forward(noisy(h), W, p + "mlp.", L["mlp"], margins)))
        if layer_sums is not None:
            layer_sums.append(X.sum(dim=1))
    return norm_one_plus(X.sum(dim=1), W["final.norm"], eps) @ W["head"].T


def rounding_errors(cfg, W, tokens, size, draws=4, layer=None):
    """Per row, the largest change of the logits (or of the stream's sum after layer ``layer``) that roundings of the
    relative size ``size`` cause: some rows carry small differences of large terms (a retention head that is divided by
    its root mean square) and move further than others."""
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
    """name -> (shape, kind) of every tensor the model has; kinds: embed, matrix, shift (around zero), gain (around one),
    read / carry / write (the copies' small tensors), taps, router, bias."""
    Wd, V, n = int(cfg["width"]), int(cfg["vocab"]), int(cfg.get("streams", 1))
    out = {"embed": ((V, Wd), "embed"), "head": ((V, Wd), "matrix"), "final.norm": ((Wd,), "shift")}

    def sublayer(p, q):
        out[f"{p}norm{q}"] = ((Wd,), "shift")
        out[f"{p}hc{q}.in"] = ((n,), "read")
        out[f"{p}hc{q}.out"] = ((n,), "write")
        out[f"{p}hc{q}.mix"] = ((n, n), "carry")

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        sublayer(p, 1)
        out[p + "canon1"] = ((Wd, int(cfg["canon"]["taps"])), "taps")
        H, D, Dv = int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"]))
        x = p + "mix."
        out[x + "q"], out[x + "o"] = ((H * D, Wd), "matrix"), ((Wd, H * Dv), "matrix")
        if L["type"].startswith("retention"):
            out[x + "k"], out[x + "v"], out[x + "g"] = ((H * D, Wd), "matrix"), ((H * Dv, Wd), "matrix"), ((H * Dv, Wd), "matrix")
        else:
            out[x + "q.norm"], out[x + "g"] = ((H * D,), "gain"), ((H, Wd), "matrix")
            if m.get("kv_from") is None:
                G = int(m["kv_heads"])
                out[x + "k"], out[x + "v"] = ((G * D, Wd), "matrix"), ((G * Dv, Wd), "matrix")
                out[x + "k.norm"] = ((G * D,), "gain")
        f = L.get("mlp")
        if f:
            sublayer(p, 2)
            y = p + "mlp."
            if f["kind"] == "dense":
                names, ff = [y], int(f["ff"])
            else:
                E = int(f["router"]["experts"])
                names, ff = [f"{y}e{e}." for e in range(E)], int(f["expert"]["ff"])
                out[y + "router"], out[y + "router.b"] = ((E, Wd), "router"), ((E,), "bias")
            for z in names:
                out[z + "gate"], out[z + "up"], out[z + "down"] = ((ff, Wd), "matrix"), ((ff, Wd), "matrix"), ((Wd, ff), "matrix")
    return out


def make_weights(cfg, seed, scale=1.0):
    """bfloat16-rounded values as float64: matrices N(0, scale / sqrt(columns)); the carry matrices lie around the unit
    matrix with a clear part off the diagonal, so that swapping [from, to] shows."""
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
        elif kind == "shift":
            t = 0.2 * z
        elif kind == "router":      # (choices that hang on the bias as much as on the row: few of them are close)
            t = z * 0.5 / math.sqrt(shape[-1])
        elif kind == "bias":
            t = 1.2 * z
        elif kind == "taps":
            t = 0.4 * z
        elif kind == "read":
            t = 1.0 / shape[0] + 0.2 * z
        elif kind == "write":
            t = 1.0 + 0.3 * z
        else:
            t = 0.9 * torch.eye(shape[0], dtype=F64) + 0.15 * z
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
def retention_layer(heads=3, dim=32, vdim=None, rot_dims=None, base=10000.0, decay=None, mlp=None, type="retention"):
    decay = [1.0 - 2.0 ** (-2 - i) for i in range(heads)] if decay is None else list(decay)
    rot_dims = dim if rot_dims is None else rot_dims
    return {"type": type, "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": dim if vdim is None else vdim, "decay": decay,
                      "rot": {"dims": rot_dims, "base": base} if rot_dims else None}}


def attention_layer(heads=4, kv_heads=2, dim=32, vdim=None, scale=0.2, kv_from=None, mlp=None, type="attention"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": type, "mixer": m, "mlp": mlp}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def model_config(layers, width=64, vocab=150, streams=2, taps=3, eps=1e-5, embed_scale=2.5):
    return {"architecture": "Sevelorn", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps},
            "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}
