"""Tiny Viperax configurations for the tests, and how their random model folders are made and read back."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _layer(heads, dim, vdim, kv_rank, scale, window=0, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


# X: odd sizes everywhere (no tensor-core attention shape, no tensor-core experts); windows that are no multiple of a page; a reader of
# another layer's latents whose window is longer than its owner's; a layer without a feed-forward; experts without a shared one; all
# experts chosen.
VIPERAX_X = {
    "architecture": "Viperax", "vocab": 211, "width": 92, "streams": 3, "norm": {"eps": 3e-5}, "embedding": {"scale": 2.5},
    "logit_scale": 0.7, "logit_softcap": 9.0,
    "layers": [_layer(3, 22, 27, 44, 0.21, 13, mlp=_moe(5, 2, 37)),
               _layer(5, 18, 31, 44, 0.25, 29, kv_from=0, mlp=_dense(51)),
               _layer(2, 30, 12, 35, 0.2, 40),
               _layer(1, 9, 40, 44, 0.3, 7, kv_from=0, mlp=_moe(3, 3, 20, 26))],
}
# Y: shapes that the tensor-core kernels take; a layer that sees everything and a windowed reader of it, and the other way round; the
# experts' rows in several tiles; two streams.
VIPERAX_Y = {
    "architecture": "Viperax", "vocab": 320, "width": 160, "streams": 2, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
    "logit_scale": 1.0, "logit_softcap": 30.0,
    "layers": [_layer(8, 32, 48, 64, 0.18, 0, mlp=_moe(4, 1, 72, 40)),
               _layer(4, 48, 64, 96, 0.14, 50, mlp=_dense(200)),
               _layer(16, 16, 32, 64, 0.25, 100, kv_from=0, mlp=_moe(6, 3, 48, 136)),
               _layer(2, 64, 96, 96, 0.12, 0, kv_from=1, mlp=_moe(40, 2, 24))],
}
# Z: one stream; a width that no tensor-core product takes; a window of one token; one head; a single expert; no cap, no scale; a
# sequence of layers that all read the first one's latents.
VIPERAX_Z = {
    "architecture": "Viperax", "vocab": 150, "width": 100, "streams": 1, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
    "layers": [_layer(4, 20, 12, 24, 0.25, 1, mlp=_moe(1, 1, 33)),
               _layer(1, 16, 8, 24, 0.3, 64, kv_from=0, mlp=_dense(30)),
               _layer(6, 8, 20, 24, 0.35, 9, kv_from=0)],
}
# S: more streams than the kernels' widest unrolled form.
VIPERAX_S = {
    "architecture": "Viperax", "vocab": 130, "width": 64, "streams": 6, "norm": {"eps": 1e-4}, "embedding": {"scale": 3.0}, "logit_softcap": 5.0,
    "layers": [_layer(2, 16, 16, 32, 0.25, 20, mlp=_moe(9, 4, 16, 24)), _layer(2, 24, 32, 32, 0.2, 33, kv_from=0, mlp=_dense(64))],
}
VIPERAX = {"X": (VIPERAX_X, 61, 16), "Y": (VIPERAX_Y, 62, 32), "Z": (VIPERAX_Z, 63, 8), "S": (VIPERAX_S, 64, 16)}   # config, weight seed, page size

STD, GAIN_STD = 0.2, 0.2


def write_model(folder, name, transform=None, config=None, seed=None) -> Path:
    """A model folder with random weights for configuration `name`; `transform(tensors)` edits them first."""
    from stride_b200.weights.random_init import random_tensors
    from stride_b200.weights.safetensors_io import write_safetensors
    cfg, own_seed, _ = VIPERAX.get(name, (config, seed, 0))
    cfg = config or cfg
    tensors = random_tensors(cfg, seed or own_seed, std=STD, gain_std=GAIN_STD)
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


def near_uniform(tensors):
    """Queries scaled down: every attention is close to uniform, so that EVERY visible key carries weight and one key too many or too few
    (a window one token off, a sink left out) moves the logits; the sinks are raised so that they weigh as much as a few keys."""
    for n in list(tensors):
        if n.endswith("mix.q"):
            tensors[n] = (tensors[n].float() * 0.05).to(tensors[n].dtype)
        elif n.endswith("mix.sink"):
            tensors[n] = (tensors[n].float() + 2.0).to(tensors[n].dtype)


def drawn(seed):
    """A configuration drawn at random: any sizes, streams, order of layers, sharing of latents, windows of one token and windows longer
    than the request, feed-forwards of every kind and none."""
    import random
    r = random.Random(seed)
    eight = r.random() < 0.5                     # half of them in multiples that the tensor-core kernels take
    size = (lambda lo, hi: 8 * r.randint((lo + 7) // 8, hi // 8)) if eight else r.randint
    layers, own = [], []
    for i in range(r.randint(2, 6)):
        mlp = r.choice(["dense", "moe", "moe", None])
        if mlp == "dense":
            mlp = _dense(size(8, 90))
        elif mlp == "moe":
            experts = r.randint(1, 12)
            mlp = _moe(experts, r.randint(1, min(experts, 4)), size(8, 60), r.choice([0, size(8, 60)]))
        kv_from = r.choice(own) if own and r.random() < 0.5 else None
        rank = layers[kv_from]["mixer"]["kv_rank"] if kv_from is not None else (16 * r.randint(1, 5) if eight else r.randint(3, 70))
        heads = r.choice([1, 2, 4, 8, 16]) if eight else r.randint(1, 7)
        layers.append(_layer(heads, size(8, 40), size(8, 40), rank, r.choice([0.1, 0.2, 0.35]), r.choice([0, 1, 2, 5, 16, 33, 64, 500]), kv_from, mlp))
        if kv_from is None:
            own.append(i)
    cfg = {"architecture": "Viperax", "vocab": r.randint(30, 300), "width": size(24, 140), "streams": r.choice([1, 2, 3, 4, 5]),
           "norm": {"eps": r.choice([1e-6, 1e-4])}, "embedding": {"scale": r.choice([0.5, 1.0, 6.0])}, "layers": layers}
    if r.random() < 0.7:
        cfg["logit_scale"] = r.choice([0.25, 1.5])
    if r.random() < 0.7:
        cfg["logit_softcap"] = r.choice([4.0, 20.0])
    return cfg
