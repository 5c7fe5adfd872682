"""Small Pemorax configurations for the tests, their model folders and the plain implementation's logits.
The configurations differ from each other in every size and constant and avoid values that would hide a mix-up: as many KV
heads as heads, a value size equal to the key size, the same sizes left and right, a rotation over a whole head, windows
that are a multiple of the page, one decay for all heads, all experts chosen.

pem-a: convolutions of four, two and three taps; windows of 37 with three kept tokens and of 21 with none on pages of 16; a
       layer without window, cap and rotations; no feed-forward, experts, dense.
pem-b: sizes that the tensor-core kernels take (heads of 64 with 64 values, of 48 with 128; experts of 64) on pages of 32;
       windows of 70 with 5 kept tokens and of 50 with 40.
pem-c: an odd width, odd head sizes and channels, a window of 9 with 20 kept tokens on pages of 8, one expert of four per
       token, a layer without convolution.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List

import torch

import plain_pemorax as P


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _rot(rot):
    """(base, dims) or (base, dims, scaling)."""
    d = {"base": rot[0], "dims": rot[1]}
    if len(rot) > 2:
        d["scaling"] = rot[2]
    return d


def left(heads, kv, dim, vdim, scale, conv=3, rot=None, window=None, keep=None, cap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if conv:
        m["conv"] = conv
    if rot:
        m["rot"] = _rot(rot)
    if window:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if cap:
        m["softcap"] = cap
    return m


def right(dim, vdim, decay, rot=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        m["rot"] = _rot(rot)
    return m


def layer(l, r, mlp=None):
    return {"type": "parallel", "mixer": {"left": l, "right": r}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, eps, layers):
    return {"architecture": "Pemorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    "pem-a": dict(seed=71, block_size=16, cfg=model(203, 72, 2e-5, [
        layer(left(4, 2, 20, 12, 0.4, 4, (1000.0, 12, yarn(3.0, 64, 8.0, 0.5)), 37, 3, 5.0), right(10, 14, [0.9, 0.37, 0.995], (50.0, 6))),
        layer(left(3, 1, 12, 28, 0.25, 2, (500.0, 12), 21, None, 30.0), right(24, 40, [0.8, 0.999], (9000.0, 24)), moe(8, 3, 24)),
        layer(left(6, 3, 8, 16, 0.5, 3), right(16, 6, [0.7]), dense(100)),
    ])),
    "pem-b": dict(seed=72, block_size=32, cfg=model(150, 128, 1e-6, [
        layer(left(4, 1, 64, 64, 0.14, 3, (50000.0, 32, yarn(8.0, 128, 32.0, 1.0)), 70, 5, 20.0),
              right(64, 32, [0.6, 0.97, 0.9, 0.999], (10000.0, 64)), moe(16, 4, 64)),
        layer(left(4, 2, 48, 128, 0.2, 4, (777.0, 48), 50, 40, 8.0), right(32, 128, [0.95, 0.5], (777.0, 8)), dense(160)),
    ])),
    "pem-c": dict(seed=73, block_size=8, cfg=model(97, 41, 1e-4, [
        layer(left(3, 1, 7, 9, 0.5, 3, (50.0, 2), 9, 20, 3.0), right(5, 7, [0.5], (20.0, 4)), dense(13)),
        layer(left(2, 2, 10, 6, 0.6, 0, (50.0, 10, yarn(2.0, 32, 4.0, 0.5)), 12, 1, 2.0), right(6, 5, [0.9, 0.99], (3.0, 6)), moe(4, 1, 10)),
    ])),
}

TORCH_DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def decisive_routers(cfg: dict, w: Dict[str, torch.Tensor], seed: int) -> None:
    """Makes every router's choice a clear one, so that a rounding of the 16-bit path cannot turn it (two experts of
    nearly equal logits are no fault of the engine, but they move a position's logits by much).  Every routed layer
    gets residual coordinates of its own, one per expert.  On them the token table holds a permutation of evenly
    spaced codes per token, and no sublayer writes there (the rows of every output matrix are zero), so through all
    layers the stream holds the code; the router reads exactly these coordinates of the normed stream.  A row's router
    logits are then a scaled permutation that depends on its token, moved a little by the router's bias."""
    g = torch.Generator().manual_seed(seed)
    at = 0
    for i, spec in enumerate(cfg["layers"]):
        mlp = spec.get("mlp")
        if not mlp or mlp["kind"] != "moe":
            continue
        E = mlp["router"]["experts"]
        cols = slice(at, at + E)
        at += E
        assert at <= cfg["width"]
        codes = torch.stack([torch.randperm(E, generator=g) for _ in range(cfg["vocab"])]).float()
        w["embed"][:, cols] = ((codes - (E - 1) / 2) * (3.0 / E)).to(w["embed"].dtype)
        for name in w:
            if name.endswith((".o", ".down")):
                w[name][cols] = 0
        router = torch.zeros_like(w[f"l{i}.mlp.router"])
        router[:, cols] = 2.0 * torch.eye(E, dtype=router.dtype)
        w[f"l{i}.mlp.router"] = router
        w[f"l{i}.mlp.router.b"] = w[f"l{i}.mlp.router.b"] * 0.1
        w[f"l{i}.norm2"][cols] = 1.0


def write_model_from(cfg_dict: dict, seed: int, dtype: str, folder: str, decisive: bool = True) -> str:
    """Random weights through the package's own writer; the token table and the output head are scaled up so that the
    embedding counts beside the normalised sublayers and the logits spread over several units."""
    import kvcm
    cfg = kvcm.config.config_from_dict(cfg_dict)
    kvcm.write_random_model(folder, cfg, seed, TORCH_DT[dtype])
    _, w = read_model(folder)
    w["embed"], w["head"] = w["embed"] * 50.0, w["head"] * 25.0
    for name in w:
        if name.endswith("router.b"):
            w[name] = w[name] * 10.0
    if decisive:
        decisive_routers(cfg_dict, w, seed)
    save_weights(folder, w, dtype)
    return folder


def write_model(name: str, dtype: str, folder: str) -> str:
    c = CONFIGS[name]
    return write_model_from(c["cfg"], c["seed"], dtype, folder)


def read_model(folder: str):
    """(config dict, weights as float64)."""
    from safetensors import safe_open
    cfg = json.load(open(os.path.join(folder, "config.json")))
    w: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for k in f.keys():
            w[k] = f.get_tensor(k).double()
    return cfg, w


def save_weights(folder: str, w: Dict[str, torch.Tensor], dtype: str) -> None:
    from safetensors.torch import save_file
    save_file({n: t.to(TORCH_DT[dtype]).contiguous() for n, t in w.items()}, os.path.join(folder, "model.safetensors"),
              metadata={"format": "pt"})


def plain_logits(folder: str, tokens: List[int]) -> torch.Tensor:
    cfg, w = read_model(folder)
    return P.forward(cfg, w, list(tokens))
