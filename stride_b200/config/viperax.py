"""Viperax: a decoder whose layers are listed one by one in config.json. In place of one residual there are several streams that every
sublayer reads a weighted sum of and that all take a weighted sum of each other and of its result (hyper-connections); in front of a sublayer
stands a layer norm with a gain and no bias. The mixer is latent attention without positions: queries straight from the input, keys and values
out of one normed latent per token (all that is cached), a sliding window, a learned sink per head in the softmax's denominator, an
elementwise sigmoid gate on the heads' results. A layer may store no latent and read an earlier layer's, with its own projections and its own
window. The feed-forward is a gated silu one, or experts that a stored table gives each token id (no router), beside a shared expert. The
embedding is scaled; the logits are scaled and softly capped.

config.json keys read here:
  architecture "Viperax"; vocab, width, streams; norm.eps; embedding.scale (absent: 1); logit_scale (absent: 1); logit_softcap (absent: none);
  layers[i]: type "latent_attention", mixer {heads, dim, vdim, kv_rank, scale, mask.size (absent: every earlier key), kv_from (absent: a latent
    of its own)}, mlp ({kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top}, shared {ff} (absent: none)} | null).
Tensor names: embed, head, final.norm, l<i>.{norm1,norm2}, l<i>.hc{1,2}.{in,out,mix}, l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,g,o},
  l<i>.mlp.{gate,up,down} or l<i>.mlp.{table,e<j>.gate,e<j>.up,e<j>.down,shared.gate,shared.up,shared.down}.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .keralorn import _get
from .llama import ConfigError
from .registry import Architecture, register_architecture

DEFAULT_MAX_POSITIONS = 32768      # config.json names no longest sequence; `max_context` of the engine overrides this


@dataclass(frozen=True)
class ViperaxLayer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int = 0                    # 0: every earlier key
    kv_from: Optional[int] = None      # the layer whose latents this one reads; None: its own
    ff: int = 0                        # the dense feed-forward's size, or one expert's; 0: no feed-forward
    experts: int = 0                   # 0: a dense feed-forward
    top: int = 0
    shared: int = 0                    # the shared expert's size; 0: none


@dataclass(frozen=True)
class ViperaxConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float               # 0: no cap
    layers: tuple
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()

    @staticmethod
    def from_dict(j: dict) -> "ViperaxConfig":
        vocab, width, streams = (_get(j, k, "", int, True) for k in ("vocab", "width", "streams"))
        eps = _get(j.get("norm"), "eps", "norm.", float, True)
        optional = lambda d, key, where, default, positive=False: _get(d, key, where, float, positive) if d and d.get(key) is not None else default
        embedding_scale = optional(j.get("embedding"), "scale", "embedding.", 1.0)
        logit_scale, softcap = optional(j, "logit_scale", "", 1.0), optional(j, "logit_softcap", "", 0.0, True)
        raw_layers = j.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, l in enumerate(raw_layers):
            w = f"layers[{i}]."
            kind = _get(l, "type", w)
            if kind != "latent_attention":
                raise ConfigError(f"config.json: '{w}type' {kind!r} is not supported (latent_attention)")
            m, mw = _get(l, "mixer", w), w + "mixer."
            heads, dim, vdim, kv_rank = (_get(m, k, mw, int, True) for k in ("heads", "dim", "vdim", "kv_rank"))
            mask, kv_from = m.get("mask"), m.get("kv_from")
            if kv_from is not None:
                kv_from = _get(m, "kv_from", mw, int)
                if not 0 <= kv_from < i or layers[kv_from].kv_from is not None or layers[kv_from].kv_rank != kv_rank:
                    raise ConfigError(f"config.json: '{mw}kv_from' {kv_from} is no earlier layer with latents of its own of kv_rank {kv_rank}")
            fields = {}
            mlp = l.get("mlp")
            if mlp is not None:
                ml = w + "mlp."
                mk = _get(mlp, "kind", ml)
                if mk == "dense":
                    fields.update(ff=_get(mlp, "ff", ml, int, True))
                elif mk == "moe":
                    r = _get(mlp, "router", ml)
                    experts, top = (_get(r, k, ml + "router.", int, True) for k in ("experts", "top"))
                    if top > experts:
                        raise ConfigError(f"config.json: '{ml}router' chooses {top} of {experts} experts")
                    fields.update(ff=_get(_get(mlp, "expert", ml), "ff", ml + "expert.", int, True), experts=experts, top=top)
                    if mlp.get("shared"):
                        fields.update(shared=_get(mlp["shared"], "ff", ml + "shared.", int, True))
                else:
                    raise ConfigError(f"config.json: '{ml}kind' {mk!r} is not supported (dense, moe)")
            layers.append(ViperaxLayer(heads, dim, vdim, kv_rank, _get(m, "scale", mw, float), kv_from=kv_from,
                                       window=_get(mask, "size", mw + "mask.", int, True) if mask else 0, **fields))
        eos = j.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, list) else (int(eos),)
        return ViperaxConfig(vocab, width, streams, eps, embedding_scale, logit_scale, softcap, tuple(layers), eos_token_ids=eos)


def viperax_model_spec(cfg: ViperaxConfig) -> ModelSpec:
    W = cfg.width

    def norm(name):
        return PartSpec("layernorm", {"size": W, "eps": cfg.eps}, {"weight": name})

    def connection(p):
        return PartSpec("hyper_connection", {"hidden_size": W, "streams": cfg.streams}, {r: p + r for r in ("in", "out", "mix")})

    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        own = l.kv_from is None
        tensors = {r: p + "mix." + r for r in ("q", "uk", "uv", "sink", "g", "o")}
        if own:
            tensors.update(dkv=p + "mix.dkv", dkv_norm=p + "mix.dkv.norm")
        mixer = PartSpec("latent_attention",
                         {"hidden_size": W, "num_heads": l.heads, "key_dim": l.dim, "value_dim": l.vdim, "q_rank": 0, "kv_rank": l.kv_rank,
                          "scale": l.scale, "norm_eps": cfg.eps, "window": l.window, "sink": True, "gate": True, "own_latent": own}, tensors)
        parts = {"mixer_norm": norm(p + "norm1"), "mixer": mixer, "mixer_streams": connection(p + "hc1.")}
        if not l.ff:
            layers.append(LayerSpec("hyper_mixer", parts))
            continue
        f = p + "mlp."
        if l.experts:
            names = {r: tuple(f"{f}e{e}.{r}" for e in range(l.experts)) for r in ("gate", "up", "down")}
            shared = {"shared_" + r: f"{f}shared.{r}" for r in ("gate", "up", "down")} if l.shared else {}
            ff = PartSpec("table_experts", {"hidden_size": W, "vocab_size": cfg.vocab, "intermediate_size": l.ff, "experts": l.experts, "top": l.top,
                                            "shared": l.shared}, {"table": f + "table", **names, **shared})
        else:
            ff = PartSpec("gated", {"hidden_size": W, "intermediate_size": l.ff}, {r: f + r for r in ("gate", "up", "down")})
        parts.update(feed_forward_norm=norm(p + "norm2"), feed_forward=ff, feed_forward_streams=connection(p + "hc2."))
        layers.append(LayerSpec("hyper", parts))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec("lookup", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i, cache_of=l.kv_from) for i, l in enumerate(cfg.layers)),
        final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False, "scale": cfg.logit_scale, "cap": cfg.logit_softcap},
                      {"weight": "head", "tied_to": "embed"}),
        max_positions=cfg.max_positions, eos_token_ids=cfg.eos_token_ids)


register_architecture(Architecture("Viperax", ViperaxConfig.from_dict, viperax_model_spec), "viperax")
