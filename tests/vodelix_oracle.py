"""Plain, slow restatement of the Vodelix design in torch (CPU, float64): one function per mechanism, position by position where the
mechanism is a mask or a recurrence.  Test infrastructure only: nothing here is imported by the package, and nothing of the package is
imported here.

Notation: T tokens of ONE sequence, W model width, weights as a dict name -> tensor with the checkpoint's names.

The design in short.  Each sublayer is normed on both sides, x <- x + nb(f(na(x))), with RMS norms whose weights are stored around zero.
Mixers: soft-max attention without positions (one RMS norm over the whole q and k projections, a constant one in the denominator), or a
delta-rule recurrence with a decay per key channel.  Feed-forward: dense with squared relu, or experts (exact gelu) weighted by the soft-max
over the chosen router logits, plus a shared expert.  Every layer ends with an addition that depends on the token id.  A span of layers may
run several times.  Positions enter once, as a sinusoid added to the embedding.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ---- norms and activations ---------------------------------------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + w)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


# ---- embedding ---------------------------------------------------------------------------------------------------------------------
def sinusoid(pos: int, width: int) -> torch.Tensor:
    out = torch.zeros(width, dtype=F64)
    for j in range(width):
        angle = pos * 10000.0 ** (-2.0 * (j // 2) / width)
        out[j] = math.sin(angle) if j % 2 == 0 else math.cos(angle)
    return out


def embed(tokens: List[int], table: torch.Tensor, pos0: int = 0) -> torch.Tensor:
    return torch.stack([table[t] + sinusoid(pos0 + i, table.shape[1]) for i, t in enumerate(tokens)])


# ---- mixers ------------------------------------------------------------------------------------------------------------------------
def attend_with_unit_sink(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V]: row i over keys 0..i; weights exp(s) / (1 + sum exp(s))"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            s = (k[:i + 1, g] @ q[i, h]) * scale
            m = torch.clamp(s.max(), min=0.0)
            e = torch.exp(s - m)
            out[i, h] = (e / (torch.exp(-m) + e.sum())) @ v[:i + 1, g]
    return out


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    q = rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T
    o = attend_with_unit_sink(q.reshape(T, m["heads"], m["dim"]), k.reshape(T, m["kv_heads"], m["dim"]), v.reshape(T, m["kv_heads"], m["vdim"]), m["scale"])
    return o.reshape(T, -1) @ w[p + "o"].T


def delta_scan(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, w: torch.Tensor, a: torch.Tensor, S: Optional[torch.Tensor] = None, unit_eps: float = 1e-6):
    """one head, all [T, D] (v [T, V]): S <- diag(w) S - (a u)(u^T S) + k v^T with u = k / sqrt(sum k^2 + unit_eps), o = S^T r;
    returns (o [T, V], last S [D, V])"""
    T, D = k.shape
    V = v.shape[1]
    S = torch.zeros(D, V, dtype=k.dtype) if S is None else S.clone()
    out = torch.zeros(T, V, dtype=k.dtype)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + unit_eps)
        S = w[t][:, None] * S - torch.outer(a[t] * u, u @ S) + torch.outer(k[t], v[t])
        out[t] = r[t] @ S
    return out, S


def delta_decay(z: torch.Tensor, w0: torch.Tensor) -> torch.Tensor:
    """decay from the low-rank branch's output z"""
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(z + w0))


def delta_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, D = h.shape[0], m["heads"], m["dim"]
    heads = lambda x: x.reshape(T, H, D)
    r, k, v = heads(h @ w[p + "r"].T), heads(h @ w[p + "k"].T), heads(h @ w[p + "v"].T)
    dec = heads(delta_decay(torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T, w[p + "w0"]))
    rem = heads(torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]))
    o = torch.stack([delta_scan(r[:, i], k[:, i], v[:, i], dec[:, i], rem[:, i])[0] for i in range(H)], 1)
    o = rms(o, eps).reshape(T, H * D) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------------------
def route(z: torch.Tensor, top: int):
    """(chosen experts, weights) of one token: the largest logits, soft-max over them alone"""
    best = torch.topk(z, top)
    return best.indices.tolist(), torch.softmax(best.values, 0)


def experts(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, f: dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    one = lambda x, q: gelu_erf(x @ w[q + "up"].T) @ w[q + "down"].T
    for t in range(h.shape[0]):
        ids, wts = route(h[t] @ w[p + "router"].T, f["router"]["top"])
        for e, c in zip(ids, wts):
            out[t] += c * one(h[t], p + f"e{e}.")
    if f.get("shared"):
        out = out + one(h, p + "shared.")
    return out


def dense(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


# ---- the addition that depends on the token id ---------------------------------------------------------------------------------------
def token_side(x: torch.Tensor, tokens: List[int], w: Dict[str, torch.Tensor], layer: int, dim: int, eps: float) -> torch.Tensor:
    p = f"l{layer}.side."
    e = w["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return x + rms(y, eps) * w[p + "norm"]


# ---- the model ---------------------------------------------------------------------------------------------------------------------
def layer_runs(cfg: dict) -> List[tuple]:
    """(layer, pass) in the order they run; pass is None outside the loop"""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    return [(i, None) for i in range(lp["start"])] + [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])] + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg: dict, P: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """float64 logits [T, vocab] of a whole sequence"""
    w = {k: v.to(F64) for k, v in P.items()}
    eps = cfg["norm"]["eps"]
    tokens = list(tokens)
    x0 = x = embed(tokens, w["embed"])
    for i, t in layer_runs(cfg):
        lay, p = cfg["layers"][i], f"l{i}."
        if t is not None and i == cfg["loop"]["start"]:
            if t > 0:
                x = x + x0
            x = x + w["loop.step"][t]
        h = norm_around_one(x, w[p + "norm1"], eps)
        mixer = attention_mixer if lay["type"] == "attention" else delta_mixer
        x = x + norm_around_one(mixer(h, w, p + "mix.", lay["mixer"], eps), w[p + "norm1b"], eps)
        f = lay.get("mlp")
        if f is not None:
            h = norm_around_one(x, w[p + "norm2"], eps)
            y = dense(h, w, p + "mlp.") if f["kind"] == "dense" else experts(h, w, p + "mlp.", f)
            x = x + norm_around_one(y, w[p + "norm2b"], eps)
        if cfg.get("token_side"):
            x = token_side(x, tokens, w, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_around_one(x, w["final.norm"], eps) @ w["embed"].T


# ---- random checkpoints ------------------------------------------------------------------------------------------------------------
def random_model(cfg: dict, seed: int = 0, rank: int = 7) -> Dict[str, torch.Tensor]:
    """random weights that are exact in bfloat16 (so that float32 runs of the framework see the same numbers); rank: size of the low-rank decay branch"""
    gen = torch.Generator().manual_seed(seed)
    W, Vc, n = cfg["width"], cfg["vocab"], len(cfg["layers"])
    P: Dict[str, torch.Tensor] = {}

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=gen) * std + mean).to(torch.bfloat16).to(torch.float32)

    def lin(name, o, i, gain=1.0):
        P[name] = rnd(o, i, std=gain / math.sqrt(i))

    P["embed"] = rnd(Vc, W)
    P["final.norm"] = rnd(W, std=0.2)
    if cfg.get("loop"):
        P["loop.step"] = rnd(cfg["loop"]["times"], W, std=0.5)
    sd = (cfg.get("token_side") or {}).get("dim")
    if sd:
        P["side.embed"] = rnd(Vc, n * sd)
    for i, lay in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", lay["mixer"], lay.get("mlp")
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            P[p + nm] = rnd(W, std=0.2, mean=-0.1)
        q = p + "mix."
        H, D = m["heads"], m["dim"]
        if lay["type"] == "attention":
            G, V = m["kv_heads"], m["vdim"]
            lin(q + "q", H * D, W), lin(q + "k", G * D, W), lin(q + "v", G * V, W), lin(q + "o", W, H * V)
            P[q + "q.norm"], P[q + "k.norm"] = rnd(H * D, std=0.3, mean=1.0), rnd(G * D, std=0.3, mean=1.0)
        else:
            for nm in "rkvga":
                lin(q + nm, H * D, W, gain=1.5 if nm == "k" else 1.0)
            P[q + "a.b"], P[q + "w0"], P[q + "norm"] = rnd(H * D, std=0.5), rnd(H * D, std=1.0, mean=-1.5), rnd(H * D, std=0.3, mean=1.0)
            lin(q + "w1", rank, W), lin(q + "w2", H * D, rank), lin(q + "o", W, H * D)
        if f and f["kind"] == "dense":
            lin(p + "mlp.up", f["ff"], W), lin(p + "mlp.down", W, f["ff"])
        elif f:
            lin(p + "mlp.router", f["router"]["experts"], W, gain=2.0)
            for e in range(f["router"]["experts"]):
                lin(p + f"mlp.e{e}.up", f["expert"]["ff"], W, gain=2.0), lin(p + f"mlp.e{e}.down", W, f["expert"]["ff"])
            if f.get("shared"):
                lin(p + "mlp.shared.up", f["shared"]["ff"], W, gain=2.0), lin(p + "mlp.shared.down", W, f["shared"]["ff"])
        if sd:
            lin(p + "side.gate", sd, W, gain=0.3), lin(p + "side.proj", W, sd)      # (logits far below zero everywhere would leave the norm behind it nothing but rounding)
            P[p + "side.norm"] = rnd(W, std=0.2, mean=0.6)
    return P


def write_checkpoint(folder: str, cfg: dict, P: Dict[str, torch.Tensor]) -> None:
    """config.json + model.safetensors (bfloat16 tensors; header = 8-byte length + JSON, then the data)"""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, t in P.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(head).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
