"""Pemorax restated plainly: float64 torch on the CPU, whole sequences at once, one function per
mechanism, written from the design's equations and sharing no code with the engine.

A model is (cfg, tensors): ``cfg`` the parsed config.json, ``tensors`` name -> float64 tensor.
``forward(cfg, tensors, tokens)`` returns the logits of every position; ``trace`` additionally the
residual stream after every layer.
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


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def short_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: the last tap weighs the row itself, the first the row taps - 1 earlier (zeros ahead of row 0)."""
    taps, y = w.shape[1], torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            back = taps - 1 - j
            if t >= back:
                y[t] += w[:, j] * u[t - back]
    return y


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


def rotate(x: torch.Tensor, rot: Optional[dict], interleaved: bool) -> torch.Tensor:
    """x [T, heads, n], row t at position t: the pairs of the first ``dims`` elements turn by t * f_i; the rest pass."""
    out = x.clone()
    if not rot:
        return out
    f, m = rotary_frequencies(rot)
    for i in range(rot["dims"] // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + rot["dims"] // 2)
        angle = torch.arange(x.shape[0], dtype=F) * f[i]
        c, s = (m * torch.cos(angle))[:, None], (m * torch.sin(angle))[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a] = u * c - v * s
        out[..., b] = v * c + u * s
    return out


def visible(T: int, mask: Optional[dict]) -> torch.Tensor:
    """[T, T] bool: row i sees column j when j <= i and the column is near enough or one of the first."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask:
        ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return ok


def softmax_with_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s) / (1 + sum exp(s)) along the last dimension."""
    m = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def windowed_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[n].T for n in ("q", "k", "v"))
    if m.get("conv"):
        q, k, v = (short_conv(u, w[n + ".conv"]) for u, n in ((q, "q"), (k, "k"), (v, "v")))
    q, k = rotate(q.view(T, H, dk), m.get("rot"), True), rotate(k.view(T, G, dk), m.get("rot"), True)
    v = v.view(T, G, dv)
    ok = visible(T, m.get("mask"))
    o = torch.empty(T, H, dv, dtype=F)
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * m["scale"]
        if m.get("softcap"):
            s = m["softcap"] * torch.tanh(s / m["softcap"])
        o[:, n] = softmax_with_one(s.masked_fill(~ok, float("-inf"))) @ v[:, g]
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def retention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w["q"].T).view(T, H, dk), m.get("rot"), False)
    k = rotate((h @ w["k"].T).view(T, H, dk), m.get("rot"), False) / math.sqrt(dk)
    v = (h @ w["v"].T).view(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=F)[:, None, None]
    S = torch.zeros(H, dk, dv, dtype=F)
    o = torch.empty(T, H, dv, dtype=F)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return (rms_div(o, eps).reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def joined(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    a = windowed_attention(h, m["left"], sub(w, "left."))
    b = retention(h, m["right"], sub(w, "right."), eps)
    return 0.5 * (rms_div(a, eps) * w["left.out"] + rms_div(b, eps) * w["right.out"])


def dense_ff(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return gelu_tanh(h @ w["up"].T) @ w["down"].T


def route(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int):
    """(chosen experts [T, top], their weights [T, top])."""
    val, idx = (h @ router.T + bias).topk(top, dim=-1)
    return idx, torch.softmax(val, dim=-1)


def expert_ff(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    idx, wt = route(h, w["router"], w["router.b"], mlp["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            e = f"e{int(idx[t, k])}."
            y[t] += wt[t, k] * (w[e + "down"] @ (silu(w[e + "gate"] @ h[t]) * (w[e + "up"] @ h[t])))
    return y


def layer(x: torch.Tensor, spec: dict, tensors: Dict[str, torch.Tensor], i: int, eps: float) -> torch.Tensor:
    w = sub(tensors, f"l{i}.")
    y = joined(rms_div(x, eps) * w["norm1"], spec["mixer"], sub(w, "mix."), eps)
    x = x + rms_div(y, eps) * w["norm1b"]
    mlp = spec.get("mlp")
    if mlp is None:
        return x
    y = {"dense": dense_ff, "moe": expert_ff}[mlp["kind"]](rms_div(x, eps) * w["norm2"], mlp, sub(w, "mlp."))
    return x + rms_div(y, eps) * w["norm2b"]


def trace(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]):
    eps = cfg["norm"]["eps"]
    x = tensors["embed"][torch.tensor(tokens)]
    after = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, spec, tensors, i, eps)
        after.append(x)
    return (rms_div(x, eps) * tensors["final.norm"]) @ tensors["head"].T, after


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    return trace(cfg, tensors, tokens)[0]
