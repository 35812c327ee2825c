"""Mezadra: a decoder whose layers are listed one by one in config.json, each with its own mixer (softmax attention behind a short convolution,
with capped scores, a sink and values mixed with those of an earlier layer; or linear attention with a decay per head) and an optional
feed-forward (gated with clamps, or experts behind a sigmoid router beside a gated shared one). Sublayers read the residual itself; the only
norms around them are RMS norms on their results. The embedding is scaled.

config.json keys read here:
  architecture "Mezadra"; vocab, width; norm.eps; embedding.scale (absent: 1);
  layers[i]: type ("attention" | "lightning"), mixer {...},
    attention mixer: heads, kv_heads, dim, vdim, scale, conv (taps; absent or 0: no convolution), rot {dims, base} (absent: no
                     rotation), softcap (absent or 0: none), v_mix (absent: false);
    lightning mixer: heads, dim, vdim, decay [one per head];
    mlp ({kind "dense", ff, limit} | {kind "moe", expert {ff}, router {experts, top}, shared {ff} (absent: none)} | null).
Tensor names: embed, head, final.norm, l<i>.{norm1,norm2}, l<i>.mix.{q,k,v,o,sink,q.conv,k.conv,v.conv,vmix} or
  l<i>.mix.{q,k,v,g,o,norm}, l<i>.mlp.{gate,up,down} or
  l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down,shared.gate,shared.up,shared.down,shared.sg}.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .keralorn import _get
from .llama import ConfigError
from .registry import Architecture, register_architecture

DEFAULT_MAX_POSITIONS = 32768      # config.json names no longest sequence; `max_context` of the engine overrides this
GATE_SLOPE = 1.702                 # of the dense feed-forward's gate, g sigmoid(1.702 g)


@dataclass(frozen=True)
class MezadraLayer:
    kind: str                      # "attention" | "lightning"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float = 0.0
    conv: int = 0                  # taps; 0: no convolution
    rot_dims: int = 0
    rot_base: float = 10000.0
    softcap: float = 0.0           # 0: none
    v_mix: bool = False
    decay: tuple = ()
    ff: int = 0                    # the dense feed-forward's size, or one expert's; 0: no feed-forward
    limit: float = 0.0
    experts: int = 0               # 0: a dense feed-forward
    top: int = 0
    shared: int = 0                # the shared expert's size; 0: none


@dataclass(frozen=True)
class MezadraConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()

    @staticmethod
    def from_dict(j: dict) -> "MezadraConfig":
        vocab, width = (_get(j, k, "", int, True) for k in ("vocab", "width"))
        eps = _get(j.get("norm"), "eps", "norm.", float, True)
        embedding = j.get("embedding")
        scale = _get(embedding, "scale", "embedding.", float) if embedding and embedding.get("scale") is not None else 1.0
        raw_layers = j.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, l in enumerate(raw_layers):
            w = f"layers[{i}]."
            kind = _get(l, "type", w)
            m, mw = _get(l, "mixer", w), w + "mixer."
            fields = {}
            if kind == "attention":
                heads, kv, dim, vdim = (_get(m, k, mw, int, True) for k in ("heads", "kv_heads", "dim", "vdim"))
                if heads % kv:
                    raise ConfigError(f"config.json: '{mw}heads' {heads} is no multiple of kv_heads {kv}")
                fields.update(scale=_get(m, "scale", mw, float), v_mix=bool(m.get("v_mix", False)))
                if m.get("conv"):
                    fields.update(conv=_get(m, "conv", mw, int, True))
                if m.get("softcap"):
                    fields.update(softcap=_get(m, "softcap", mw, float, True))
                if m.get("rot"):
                    dims = _get(m["rot"], "dims", mw + "rot.", int)
                    if dims < 0 or dims % 2 or dims > dim:
                        raise ConfigError(f"config.json: '{mw}rot.dims' {dims} must be even and at most dim {dim}")
                    fields.update(rot_dims=dims, rot_base=_get(m["rot"], "base", mw + "rot.", float, True))
                first = next((k for k in layers if k.v_mix), None)
                if fields["v_mix"] and first is not None and first.kv_heads * first.vdim != kv * vdim:
                    raise ConfigError(f"config.json: '{mw}v_mix': values of {kv} x {vdim} cannot be mixed with the first such layer's "
                                      f"{first.kv_heads} x {first.vdim}")
            elif kind == "lightning":
                heads, dim, vdim = (_get(m, k, mw, int, True) for k in ("heads", "dim", "vdim"))
                kv, decay = heads, m.get("decay")
                if not isinstance(decay, list) or len(decay) != heads:
                    raise ConfigError(f"config.json: '{mw}decay' must list one factor for each of the {heads} heads")
                fields.update(decay=tuple(float(d) for d in decay))
            else:
                raise ConfigError(f"config.json: '{w}type' {kind!r} is not supported (attention, lightning)")
            mlp = l.get("mlp")
            if mlp is not None:
                ml = w + "mlp."
                mk = _get(mlp, "kind", ml)
                if mk == "dense":
                    fields.update(ff=_get(mlp, "ff", ml, int, True), limit=_get(mlp, "limit", ml, float, True))
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
            layers.append(MezadraLayer(kind, heads, kv, dim, vdim, **fields))
        eos = j.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, list) else (int(eos),)
        return MezadraConfig(vocab, width, eps, scale, tuple(layers), eos_token_ids=eos)


def mezadra_model_spec(cfg: MezadraConfig) -> ModelSpec:
    W = cfg.width

    def norm(name):
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.eps}, {"weight": name})

    layers, keeps = [], True       # keeps: the next layer that mixes values is the first one
    for i, l in enumerate(cfg.layers):
        p, f = f"l{i}.mix.", f"l{i}.mlp."
        if l.kind == "attention":
            position = PartSpec("rope", {"head_dim": l.dim, "rotary_dim": l.rot_dims, "theta": l.rot_base, "exact_angles": True}) if l.rot_dims else None
            tensors = {r: p + r for r in ("q", "k", "v", "o", "sink")}
            if l.conv:
                tensors.update({f"{r}_conv": f"{p}{r}.conv" for r in "qkv"})
            if l.v_mix:
                tensors["lambda"] = p + "vmix"
            mixer = PartSpec("conv_attention",
                             {"hidden_size": W, "num_heads": l.heads, "num_kv_heads": l.kv_heads, "key_dim": l.dim, "value_dim": l.vdim, "scale": l.scale,
                              "norm_eps": cfg.eps, "taps": l.conv, "qk_unit": True, "position": position, "cap": l.softcap, "sink": True,
                              "value_mix": None if not l.v_mix else "keep" if keeps else "mix"}, tensors)
            keeps = keeps and not l.v_mix
        else:
            mixer = PartSpec("lightning", {"hidden_size": W, "num_heads": l.heads, "key_dim": l.dim, "value_dim": l.vdim, "decay": l.decay,
                                           "norm_eps": cfg.eps}, {r: p + r for r in ("q", "k", "v", "g", "o", "norm")})
        parts = {"mixer": mixer, "mixer_scale": norm(f"l{i}.norm1")}
        if not l.ff:
            layers.append(LayerSpec("postnorm_mixer", parts))
            continue
        if l.experts:
            tensors = {r: tuple(f"{f}e{e}.{r}" for e in range(l.experts)) for r in ("gate", "up", "down")}
            tensors["router"] = f + "router"
            if l.shared:
                tensors.update({"shared_" + r: f"{f}shared.{r}" for r in ("gate", "up", "down", "sg")})
            ff = PartSpec("sigmoid_experts", {"hidden_size": W, "intermediate_size": l.ff, "experts": l.experts, "top": l.top, "shared": l.shared,
                                              "shared_gate": bool(l.shared)}, tensors)
        else:
            ff = PartSpec("gated", {"hidden_size": W, "intermediate_size": l.ff, "activation": "clamped", "limit": l.limit, "slope": GATE_SLOPE},
                          {r: f + r for r in ("gate", "up", "down")})
        parts.update(feed_forward=ff, feed_forward_scale=norm(f"l{i}.norm2"))
        layers.append(LayerSpec("postnorm", parts))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec("lookup", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False}, {"weight": "head", "tied_to": "embed"}),
        max_positions=cfg.max_positions, eos_token_ids=cfg.eos_token_ids)


register_architecture(Architecture("Mezadra", MezadraConfig.from_dict, mezadra_model_spec), "mezadra")
