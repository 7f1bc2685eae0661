"""Plain, slow restatement of the Zetunex layer types in torch (CPU, float64): one function per mechanism, token by token where the
mechanism is a recurrence, row by row where it is a mask.  Test infrastructure only: nothing here is imported by the package, and nothing
of the package is imported here.

Notation: T tokens of ONE sequence, W model width, weights as a dict name -> tensor with the checkpoint's names.

The design in short.  Parallel layers: one RMS norm per layer, its output h goes to the mixer and to the feed-forward, and
x <- x + residual_mult * (mixer(h) + ff(h)).  Mixers: a linear attention with one fixed decay per head (silu on q, k and v, one RMS norm
over all heads, a sigmoid gate), or a windowed attention without positions beside a selective scan (each result normed over the model
width, half their sum).  Feed-forward: dense silu-gated, or silu-gated experts chosen inside the best groups by soft-max scores that are
also the weights.  A span of layers may run several times with a learned row added in front of each pass.  The output projection is the
embedding table.
"""
from __future__ import annotations

import json
import os
import struct
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, eps: float, w: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension, times w when given"""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def project(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str, bias: bool = False) -> torch.Tensor:
    y = h @ w[name].T
    return y + w[name + ".b"] if bias else y


# ---- linear attention with fixed decays ------------------------------------------------------------------------------------------------
def decayed_linear_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: List[float]) -> torch.Tensor:
    """q, k [T, H, D], v [T, H, V]: S <- decay_h S + k v^T, o = S^T q, token by token -> [T, H, V]"""
    T, H, D = q.shape
    d = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = d * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append((S * q[t].unsqueeze(2)).sum(1))
    return torch.stack(out)


def lightning(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q, k = silu(project(h, w, p + "q")).view(T, H, D), silu(project(h, w, p + "k")).view(T, H, D)
    v = silu(project(h, w, p + "v")).view(T, H, V)
    o = decayed_linear_attention(q, k, v, m["decay"]).reshape(T, H * V)
    return project(rms_norm(o, eps, w[p + "norm"]) * torch.sigmoid(project(h, w, p + "g")), w, p + "o")


# ---- windowed attention ----------------------------------------------------------------------------------------------------------------
def windowed_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V]; row i sees rows max(0, i - window + 1) .. i (window <= 0: 0 .. i) -> [T, H, V]"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        lo = max(0, i - window + 1) if window > 0 else 0
        for h in range(H):
            g = h // (H // G)
            out[i, h] = torch.softmax((k[lo:i + 1, g] @ q[i, h]) * scale, 0) @ v[lo:i + 1, g]
    return out


def attention_branch(h, w, p, m):
    T = h.shape[0]
    q = project(h, w, p + "q", True).view(T, m["heads"], m["dim"])
    k = project(h, w, p + "k", True).view(T, m["kv_heads"], m["dim"])
    v = project(h, w, p + "v", True).view(T, m["kv_heads"], m["vdim"])
    o = windowed_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size", 0))
    return project(o.reshape(T, -1), w, p + "o")


# ---- selective scan --------------------------------------------------------------------------------------------------------------------
def causal_conv(x: torch.Tensor, cw: torch.Tensor, cb: torch.Tensor) -> torch.Tensor:
    """x [T, C], cw [C, taps] whose last column meets the current token; zeros before the start"""
    T, taps = x.shape[0], cw.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = cb.clone()
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + cw[:, j] * x[s]
        out[t] = acc
    return out


def selective_scan(x, dt, A, B, C, D) -> torch.Tensor:
    """x, dt [T, channels], A [channels, N], B, C [T, N], D [channels]: S <- exp(dt A) S + dt x B, y = S C + D x, token by token"""
    S = torch.zeros_like(A)
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t].unsqueeze(1) * A) * S + (dt[t] * x[t]).unsqueeze(1) * B[t].unsqueeze(0)
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out)


def scan_branch(h, w, p, m):
    inner, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = project(h, w, p + "in")
    x = silu(causal_conv(xz[:, :inner], w[p + "conv"], w[p + "conv.b"]))
    dbc = project(x, w, p + "x")
    dt = torch.nn.functional.softplus(project(dbc[:, :R], w, p + "dt") + w[p + "dt.b"])
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), dbc[:, R:R + N], dbc[:, R + N:], w[p + "D"])
    return project(y * silu(xz[:, inner:]), w, p + "o")


def parallel_mixer(h, w, p, m, eps):
    left = rms_norm(attention_branch(h, w, p + "left.", m["left"]), eps, w[p + "left.out"])
    right = rms_norm(scan_branch(h, w, p + "right.", m["right"]), eps, w[p + "right.out"])
    return 0.5 * (left + right)


# ---- feed-forward ----------------------------------------------------------------------------------------------------------------------
def gated(h, w, p):
    return project(silu(project(h, w, p + "gate")) * project(h, w, p + "up"), w, p + "down")


def route(z: torch.Tensor, r: dict):
    """router logits of one token -> (expert indices, weights)"""
    E, top = r["experts"], r["top"]
    s = torch.softmax(z, 0)
    allowed = list(range(E))
    g = r.get("groups")
    if g:
        size = E // g["count"]
        best = sorted(range(g["count"]), key=lambda i: (-float(s[i * size:(i + 1) * size].max()), i))[:g["keep"]]
        allowed = [e for e in range(E) if e // size in best]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    return chosen, [float(s[e]) * r["scale"] for e in chosen]


def experts(h, w, p, mlp):
    z = project(h, w, p + "router")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(*route(z[t], mlp["router"])):
            out[t] += wt * gated(h[t:t + 1], w, p + f"e{e}.")[0]
    return out


def feed_forward(h, w, p, mlp):
    if mlp is None:
        return torch.zeros_like(h)
    return gated(h, w, p) if mlp["kind"] == "dense" else experts(h, w, p, mlp)


# ---- the model -------------------------------------------------------------------------------------------------------------------------
def layer_order(cfg: dict):
    """(layer, pass to enter in front of it or None)"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab] of one sequence; layers_out: receives the residual after every layer run"""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens)]
    for i, enter in layer_order(cfg):
        lay, p = cfg["layers"][i], f"l{i}."
        if enter is not None:
            x = x + w["loop.step"][enter]
        h = rms_norm(x, eps, w[p + "norm1"])
        mix = lightning(h, w, p + "mix.", lay["mixer"], eps) if lay["type"] == "lightning" else parallel_mixer(h, w, p + "mix.", lay["mixer"], eps)
        x = x + m * (mix + feed_forward(h, w, p + "mlp.", lay["mlp"]))
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, eps, w["final.norm"]) @ w["embed"].T


# ---- checkpoints for tests -------------------------------------------------------------------------------------------------------------
def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bfloat16 weights of the configuration's shapes, scaled so that every mechanism has an effect"""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, scale=1.0, shift=0.0):
        return (torch.randn(shape, generator=g) * scale + shift).to(torch.bfloat16)

    t = {"embed": rnd(V, W), "final.norm": rnd(W, scale=0.1, shift=1.0)}
    if cfg.get("loop"):
        t["loop.step"] = rnd(cfg["loop"]["times"], W, scale=0.5)

    def lin(name, o, i, s=1.0):
        t[name] = rnd(o, i, scale=s * i ** -0.5)

    for n, lay in enumerate(cfg["layers"]):
        p, m, f = f"l{n}.", lay["mixer"], lay["mlp"]
        t[p + "norm1"] = rnd(W, scale=0.2, shift=1.0)
        if lay["type"] == "lightning":
            H, D, Vd = m["heads"], m["dim"], m["vdim"]
            lin(p + "mix.q", H * D, W), lin(p + "mix.k", H * D, W), lin(p + "mix.v", H * Vd, W), lin(p + "mix.g", H * Vd, W), lin(p + "mix.o", W, H * Vd)
            t[p + "mix.norm"] = rnd(H * Vd, scale=0.2, shift=1.0)
        else:
            a, r = m["left"], m["right"]
            H, G, D, Vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for nm, o in (("q", H * D), ("k", G * D), ("v", G * Vd)):
                lin(p + "mix.left." + nm, o, W)
                t[p + "mix.left." + nm + ".b"] = rnd(o, scale=0.3)
            lin(p + "mix.left.o", W, H * Vd)
            C, N, R, taps = r["inner"], r["state"], r["dt_rank"], r["conv"]
            q = p + "mix.right."
            lin(q + "in", 2 * C, W), lin(q + "x", R + 2 * N, C, 2.0), lin(q + "dt", C, R), lin(q + "o", W, C)
            t[q + "conv"], t[q + "conv.b"] = rnd(C, taps, scale=taps ** -0.5), rnd(C, scale=0.1)
            t[q + "dt.b"] = rnd(C, scale=1.0, shift=-2.0)
            t[q + "A_log"] = (torch.log(torch.arange(1, N + 1).float())[None, :] + 0.2 * torch.randn(C, N, generator=g)).to(torch.bfloat16)
            t[q + "D"] = rnd(C)
            t[p + "mix.left.out"], t[p + "mix.right.out"] = rnd(W, scale=0.2, shift=1.0), rnd(W, scale=0.2, shift=1.0)
        if f is None:
            continue
        if f["kind"] == "dense":
            lin(p + "mlp.gate", f["ff"], W), lin(p + "mlp.up", f["ff"], W), lin(p + "mlp.down", W, f["ff"], 2.0)
        else:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            lin(p + "mlp.router", E, W, 3.0)
            for e in range(E):
                q = p + f"mlp.e{e}."
                lin(q + "gate", ff, W), lin(q + "up", ff, W), lin(q + "down", W, ff, 3.0)
    return t


def write_checkpoint(folder: str, cfg: dict, weights: Dict[str, torch.Tensor]) -> None:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, v in weights.items():
        raw = v.contiguous().view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": {torch.bfloat16: "BF16", torch.int32: "I32", torch.float32: "F32"}[v.dtype], "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
