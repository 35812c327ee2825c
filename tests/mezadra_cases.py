"""Tiny Mezadra configurations for the tests, and how their random model folders are made and read back."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _attn(heads, kv_heads, dim, vdim, scale, conv=0, rot=None, softcap=0.0, v_mix=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if conv:
        m["conv"] = conv
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if softcap:
        m["softcap"] = softcap
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _light(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


# M: odd sizes everywhere (no tensor-core attention shape, no tensor-core experts); an attention layer that does not mix in front of the first
# one that keeps its values; two layers that mix with them; taps of several lengths; a layer without a feed-forward; experts without a shared one.
MEZADRA_M = {
    "architecture": "Mezadra", "vocab": 211, "width": 92, "norm": {"eps": 3e-5}, "embedding": {"scale": 2.5},
    "layers": [_attn(4, 2, 22, 27, 0.6, 3, (10, 500.0), 2.0, False, _moe(5, 2, 37, 26)),
               _light(3, 20, 37, [0.5, 0.9, 0.97], _dense(51, 0.7)),
               _attn(6, 3, 18, 10, 0.9, 2, (18, 10000.0), 5.0, True, _dense(33, 2.5)),
               _attn(3, 3, 24, 10, 0.5, 5, (4, 100.0), 0.0, True),
               _light(1, 9, 12, [0.99], _moe(3, 3, 20)),
               _attn(5, 1, 16, 30, 0.7, 4, None, 3.0, True, _dense(20, 1.0))],
}
# N: shapes that the tensor-core kernels take: heads of 64 and of 128, a pair of sizes of its own (48 / 80), 16 query heads on one key head;
# experts' rows in several tiles; a shared expert larger than the others.
MEZADRA_N = {
    "architecture": "Mezadra", "vocab": 320, "width": 160, "norm": {"eps": 1e-5}, "embedding": {"scale": 6.0},
    "layers": [_attn(8, 2, 64, 64, 0.15, 4, (24, 20000.0), 25.0, True, _moe(6, 2, 72, 40)),
               _light(4, 48, 32, [0.7, 0.9, 0.98, 0.999], _dense(200, 1.5)),
               _attn(2, 1, 128, 128, 0.1, 3, (128, 10000.0), 4.0, True, _moe(40, 3, 24, 136)),
               _attn(4, 4, 48, 80, 0.2, 4, (48, 1000.0), 12.0, False, _dense(136, 0.8)),
               _attn(16, 1, 64, 64, 0.15, 6, (64, 5000.0), 0.0, None, _moe(4, 1, 48))],
}
# O: a width that no tensor-core product takes, no convolution or one of a single tap, no rotation, no cap, nothing mixed, a single expert,
# an embedding without a scale.
MEZADRA_O = {
    "architecture": "Mezadra", "vocab": 150, "width": 100, "norm": {"eps": 1e-6},
    "layers": [_attn(4, 4, 20, 12, 0.9, 0, mlp=_moe(1, 1, 33, 12)),
               _attn(2, 1, 16, 24, 0.8, 1, (16, 77.0), mlp=_dense(30, 3.0)),
               _light(2, 24, 8, [0.2, 0.95])],
}
# Q: recurrences alone between two layers that mix; the longest convolution; keys longer than values.
MEZADRA_Q = {
    "architecture": "Mezadra", "vocab": 130, "width": 64, "norm": {"eps": 1e-4}, "embedding": {"scale": 0.5},
    "layers": [_light(2, 40, 70, [0.6, 0.9995], _moe(9, 4, 16, 24)), _attn(2, 2, 32, 16, 0.4, 9, (8, 300.0), 6.0, True),
               _light(4, 8, 8, [0.5, 0.6, 0.7, 0.8]), _attn(4, 2, 64, 16, 0.3, 2, (2, 9.0), 1.5, True, _dense(64, 0.5))],
}
MEZADRA = {"M": (MEZADRA_M, 71, 16), "N": (MEZADRA_N, 72, 32), "O": (MEZADRA_O, 73, 8), "Q": (MEZADRA_Q, 74, 24)}   # config, weight seed, page size

STD, GAIN_STD = 0.2, 0.2


def _visible(tensors):
    """Numbers that random weights leave too small to matter: mixing weights around 0.6, convolutions with weight on every tap, sinks that
    weigh as much as a few keys."""
    for n in list(tensors):
        if n.endswith("vmix"):
            tensors[n] = (tensors[n].float() + 0.6).to(tensors[n].dtype)
        elif n.endswith(".conv"):
            tensors[n] = (tensors[n].float() * 2.0 + 0.3).to(tensors[n].dtype)
        elif n.endswith("mix.sink"):
            tensors[n] = (tensors[n].float() * 2.0 + 1.0).to(tensors[n].dtype)


def write_model(folder, name, transform=None, config=None, seed=None) -> Path:
    """A model folder with random weights for configuration `name`; `transform(tensors)` edits them first."""
    from stride_b200.weights.random_init import random_tensors
    from stride_b200.weights.safetensors_io import write_safetensors
    cfg, own_seed, _ = MEZADRA.get(name, (config, seed, 0))
    cfg = config or cfg
    tensors = random_tensors(cfg, seed or own_seed, std=STD, gain_std=GAIN_STD)
    _visible(tensors)
    if transform is not None:
        transform(tensors)
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", tensors)
    return folder


def load_plain(folder):
    """(config dict, name -> tensor) for the plain implementation."""
    from stride_b200.weights.safetensors_io import SafetensorsFile
    cfg = json.loads((Path(folder) / "config.json").read_text())
    f = SafetensorsFile(Path(folder) / "model.safetensors")
    try:
        return cfg, {n: f.get(n).clone() for n in f.names()}
    finally:
        f.close()


def near_uniform(cfg) -> dict:
    """The configuration with small score scales: every attention is close to uniform, so that EVERY visible key carries weight and a key
    too many or too few moves the logits."""
    cfg = json.loads(json.dumps(cfg))
    for l in cfg["layers"]:
        if l["type"] == "attention":
            l["mixer"]["scale"] *= 0.05
    return cfg


def drawn(seed):
    """A configuration drawn at random: any sizes, order of layers, with and without convolution, rotation, cap and mixing, feed-forwards of
    every kind and none."""
    import random
    r = random.Random(seed)
    eight = r.random() < 0.5                     # half of them in multiples that the tensor-core kernels take
    size = (lambda lo, hi: 8 * r.randint((lo + 7) // 8, hi // 8)) if eight else r.randint
    kv_mix, v_mix = r.choice([1, 2]), size(8, 48)
    layers = []
    for _ in range(r.randint(2, 6)):
        mlp = r.choice(["dense", "moe", "moe", None])
        if mlp == "dense":
            mlp = _dense(size(8, 90), r.choice([0.3, 1.0, 4.0]))
        elif mlp == "moe":
            experts = r.randint(1, 12)
            mlp = _moe(experts, r.randint(1, min(experts, 4)), size(8, 60), r.choice([0, size(8, 60)]))
        if r.random() < 0.4:
            heads = r.randint(1, 5)
            layers.append(_light(heads, size(8, 60), size(8, 60), [r.choice([0.3, 0.8, 0.95, 0.999]) for _ in range(heads)], mlp))
            continue
        mixes = r.random() < 0.5
        kv, vdim = (kv_mix, v_mix) if mixes else (r.randint(1, 3), size(8, 48))
        dim = size(8, 48)
        if eight and not mixes and r.random() < 0.4:
            dim = vdim = r.choice([64, 128])
        elif eight:
            dim = 16 * ((dim + 15) // 16)
        dims = 2 * r.randint(0, dim // 2)
        layers.append(_attn(kv * r.choice([1, 2, 4, 8] if eight else [1, 2, 3, 5]), kv, dim, vdim, r.choice([0.1, 0.3, 0.8]), r.choice([0, 1, 2, 3, 4, 7]),
                            (dims, r.choice([10.0, 10000.0])) if dims else None, r.choice([0.0, 2.0, 20.0]), mixes, mlp))
    cfg = {"architecture": "Mezadra", "vocab": r.randint(30, 300), "width": size(24, 140), "norm": {"eps": r.choice([1e-6, 1e-4])}, "layers": layers}
    if r.random() < 0.7:
        cfg["embedding"] = {"scale": r.choice([0.5, 1.0, 9.0])}
    return cfg
