"""Small Bimepel configurations for the tests, their model folders and the plain implementation's logits.
The configurations differ from each other in every size and constant, put the layer kinds in different orders,
and avoid values that would hide a mix-up: as many KV heads as heads, a value size equal to the key size, a rotation
over a whole head, chunks that are a multiple of the page, one decay for all heads, a router scale of 1, a loop
over everything.

bim-a: attention with a chunk of 37 on pages of 16 (partial YaRN rotation), lightning with wide values, both inside a
       loop that runs three times; a lightning layer without a feed-forward ahead of it; attention without chunks behind.
bim-b: sizes that the tensor-core kernels take (heads of 64 with 64 values, of 48 with 128; experts of 64) on pages of
       32; chunks of 70 and 50: two page groups; no loop.
bim-c: an odd width, odd head sizes, a chunk of 9 on pages of 8, one expert of four per token, an unrotated
       attention layer, a looped single layer.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List

import torch

import plain_bimepel as P


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attn(heads, kv, dim, vdim, scale, rot, chunk=None):
    """``rot``: (base, dims) or (base, dims, scaling), or None."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = rot[2]
    if chunk:
        m["mask"] = {"size": chunk}
    return m


def lightning(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


CONFIGS = {
    "bim-a": dict(seed=61, block_size=16, cfg={
        "architecture": "Bimepel", "vocab": 203, "width": 72, "norm": {"eps": 2e-5}, "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [
            {"type": "lightning", "mixer": lightning(10, 14, [0.9, 0.37, 0.995]), "mlp": None},
            {"type": "attention", "mixer": attn(4, 2, 20, 12, 0.4, (1000.0, 12, yarn(3.0, 64, 8.0, 0.5)), 37), "mlp": moe(8, 3, 24, 1.7)},
            {"type": "lightning", "mixer": lightning(24, 40, [0.8, 0.999]), "mlp": dense(100, 0.8)},
            {"type": "attention", "mixer": attn(3, 1, 12, 28, 0.25, (500.0, 12)), "mlp": dense(60, 2.5)}]}),
    "bim-b": dict(seed=62, block_size=32, cfg={
        "architecture": "Bimepel", "vocab": 150, "width": 128, "norm": {"eps": 1e-6},
        "layers": [
            {"type": "attention", "mixer": attn(4, 1, 64, 64, 0.14, (50000.0, 32, yarn(8.0, 128, 32.0, 1.0)), 70), "mlp": moe(16, 4, 64, 2.5)},
            {"type": "lightning", "mixer": lightning(64, 32, [0.6, 0.97, 0.9, 0.999]), "mlp": moe(5, 2, 20, 0.7)},
            {"type": "attention", "mixer": attn(4, 2, 48, 128, 0.2, (777.0, 48), 50), "mlp": dense(160, 1.2)}]}),
    "bim-c": dict(seed=63, block_size=8, cfg={
        "architecture": "Bimepel", "vocab": 97, "width": 41, "norm": {"eps": 1e-4}, "loop": {"start": 1, "stop": 2, "times": 2},
        "layers": [
            {"type": "attention", "mixer": attn(3, 1, 7, 9, 0.5, None), "mlp": None},
            {"type": "attention", "mixer": attn(2, 2, 10, 6, 0.6, (50.0, 2), 9), "mlp": moe(4, 1, 10, 1.3)},
            {"type": "lightning", "mixer": lightning(5, 7, [0.5]), "mlp": dense(13, 0.4)}]}),
}

TORCH_DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def decisive_routers(cfg: dict, w: Dict[str, torch.Tensor], seed: int) -> None:
    """Makes every router's choice a clear one, so that a rounding of the 16-bit path cannot turn it (two experts of
    nearly equal score are no fault of the engine, but they move a position's logits by much).  Every routed layer
    gets residual coordinates of its own, one per expert.  On them the token table holds a permutation of evenly
    spaced codes per token, and no sublayer writes there (the rows of every output matrix are zero), so through all
    layers the stream holds a multiple of the code; the router reads exactly these coordinates of the normed stream.  A
    row's router logits are then a scaled permutation that depends on its token."""
    g = torch.Generator().manual_seed(seed)
    at = 0
    for i, layer in enumerate(cfg["layers"]):
        mlp = layer.get("mlp")
        if not mlp or mlp["kind"] != "moe":
            continue
        E = mlp["router"]["experts"]
        cols = slice(at, at + E)
        at += E
        assert at <= cfg["width"]
        codes = torch.stack([torch.randperm(E, generator=g) for _ in range(cfg["vocab"])]).float()
        w["embed"][:, cols] = ((codes - (E - 1) / 2) * (3.0 / E)).to(w["embed"].dtype)
        for name in w:
            if name.endswith((".mix.o", ".down")):
                w[name][cols] = 0
        router = torch.zeros_like(w[f"l{i}.mlp.router"])
        router[:, cols] = 2.0 * torch.eye(E, dtype=router.dtype)
        w[f"l{i}.mlp.router"] = router
        w[f"l{i}.norm2"][cols] = 1.0


def write_model_from(cfg_dict: dict, seed: int, dtype: str, folder: str, decisive: bool = True) -> str:
    """Random weights through the package's own writer; the token table, which is the output head too, is scaled up so
    that the logits spread over several units, and the shifts reach from below zero to above one."""
    import kvcm
    cfg = kvcm.config.config_from_dict(cfg_dict)
    kvcm.write_random_model(folder, cfg, seed, TORCH_DT[dtype])
    _, w = read_model(folder)
    w["embed"] = w["embed"] * 25.0
    for name in w:
        if name.endswith(".shift"):
            w[name] = w[name] + 0.4
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
