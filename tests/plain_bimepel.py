"""Bimepel restated plainly: float64 torch on the CPU, whole sequences at once, one function per
mechanism, written from the design's equations and sharing no code with the engine.

A model is (cfg, tensors): ``cfg`` the parsed config.json, ``tensors`` name -> float64 tensor.
``forward(cfg, tensors, tokens)`` returns the logits of every position; ``trace`` additionally the
residual stream after every layer run.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_div(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def token_shift(h: torch.Tensor, s: torch.Tensor) -> torch.Tensor:
    """Row t becomes h_t + (h_(t-1) - h_t) * s, with zeros ahead of the first row."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * s


def rotary_frequencies(rot: dict):
    """(frequencies [dims/2], the factor of cosines and sines), with the stretched frequencies of ``scaling`` if given."""
    dims, base = rot["dims"], rot["base"]
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim(sc["fast"])), 0)
    hi = min(math.ceil(dim(sc["slow"])), dims - 1)
    out = f.clone()
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / sc["factor"] * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, n]: pairs (i, i + dims/2) of the first ``dims`` elements turn by pos * f_i; the rest pass."""
    out = x.clone()
    if not rot:
        return out
    f, m = rotary_frequencies(rot)
    half = rot["dims"] // 2
    a = pos.to(F)[:, None] * f[None, :]
    c, s = (m * torch.cos(a))[:, None, :], (m * torch.sin(a))[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def visible(T: int, chunk: int = 0) -> torch.Tensor:
    """[T, T] bool: row i sees column j when j <= i and both lie in the same chunk (0: one chunk)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if chunk > 0:
        ok = ok & (i // chunk == j // chunk)
    return ok


def mixer_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rms_div((h @ w["q"].T).view(T, H, dk), eps) * w["q.norm"]
    k = rms_div((h @ w["k"].T).view(T, G, dk), eps) * w["k.norm"]
    v = rms_div((h @ w["v"].T).view(T, G, dv), eps)
    q, k = rotate_halves(q, pos, m.get("rot")), rotate_halves(k, pos, m.get("rot"))
    ok = visible(T, (m.get("mask") or {}).get("size", 0))
    o = torch.empty(T, H, dv, dtype=F)
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * m["scale"]
        o[:, n] = torch.softmax(s.masked_fill(~ok, float("-inf")), dim=-1) @ v[:, g]
    o = o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def mixer_lightning(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(T, H, dk)
    k = silu(h @ w["k"].T).view(T, H, dk)
    v = silu(h @ w["v"].T).view(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=F)[:, None, None]
    S = torch.zeros(H, dk, dv, dtype=F)
    o = torch.empty(T, H, dv, dtype=F)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    o = rms_div(o.reshape(T, H * dv), eps) * w["norm"]
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def clamped_ff(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    lim = mlp["limit"]
    g = torch.clamp(h @ w["gate"].T, max=lim)
    u = torch.clamp(h @ w["up"].T, min=-lim, max=lim)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def route(h: torch.Tensor, router: torch.Tensor, r: dict):
    """(chosen experts [T, top], their weights [T, top])."""
    s = torch.sigmoid(h @ router.T)
    val, idx = s.topk(r["top"], dim=-1)
    return idx, val / (val.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def expert_ff(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    idx, wt = route(h, w["router"], mlp["router"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            e = f"e{int(idx[t, k])}."
            x = h[t]
            y[t] += wt[t, k] * (w[e + "down"] @ (silu(w[e + "gate"] @ x) * (w[e + "up"] @ x)))
    return y


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x: torch.Tensor, spec: dict, tensors: Dict[str, torch.Tensor], i: int, eps: float) -> torch.Tensor:
    p = f"l{i}."
    h = token_shift(rms_div(x, eps) * tensors[p + "norm1"], tensors[p + "shift"])
    mix = {"attention": mixer_attention, "lightning": mixer_lightning}[spec["type"]]
    y = mix(h, spec["mixer"], sub(tensors, p + "mix."), eps)
    mlp = spec.get("mlp")
    if mlp is None:
        return x + y
    h2 = rms_div(x, eps) * tensors[p + "norm2"]
    ff = {"dense": clamped_ff, "moe": expert_ff}[mlp["kind"]]
    return x + (y + ff(h2, mlp, sub(tensors, p + "mlp.")))


def run_order(cfg: dict) -> List[int]:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def trace(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]):
    eps = cfg["norm"]["eps"]
    x = tensors["embed"][torch.tensor(tokens)]
    after = []
    for i in run_order(cfg):
        x = layer(x, cfg["layers"][i], tensors, i, eps)
        after.append(x)
    return (rms_div(x, eps) * tensors["final.norm"]) @ tensors["embed"].T, after


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    return trace(cfg, tensors, tokens)[0]
