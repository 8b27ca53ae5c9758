"""Architecture builder for ``Folavik``: a decoder that mixes, layer by layer, latent attention without positions, attention
inside chunks and differential attention over a sliding window, all listed one by one in ``config.json``.

The configuration names its architecture as a string (``"architecture": "Folavik"``) and gives ``vocab``, ``width``,
``norm.eps``, ``logit_scale``, ``logit_softcap`` and ``layers``: per layer its ``type`` (the kind of mixer), the mixer's sizes
and constants under ``mixer``, and its feed-forward under ``mlp`` (null: the layer has none).  In this file's notation, with
the float32 stream x and every norm N a layer norm with a weight and no bias:

* x = N(embed[token]); logits = c tanh(s head N(x) / c) with s = ``logit_scale`` and c = ``logit_softcap``;
* a layer: x <- x + mixer(N(x)); x <- x + ff(N(x));
* mixer ``latent_attention``: :class:`~..parts.latent_attention.LatentAttention` with q = W_q h, nothing rotated, every
  earlier position seen, and an output gate per element;
* mixer ``attention``: :class:`~..parts.attention.ValueAttention`: halves rotated over ``rot.dims`` dimensions with the
  frequencies smoothed by wavelength (``rot.scaling`` {factor, low, high, original}), keys of the token's own chunk of
  ``mask.size`` positions;
* mixer ``attention_2``: :class:`~..parts.attention.DifferentialAttention` with biases, halves rotated under the YaRN ramp
  (``rot.scaling`` {factor, original, fast, slow}), a capped score, the last ``mask.size`` keys, and the constant ``diff``;
* feed-forward ``dense``: W_down (gelu_tanh(W_gate h) * W_up h).

This file is the only place that knows the configuration's keys and the checkpoint's tensor names (``embed``,
``embed.norm``, ``final.norm``, ``head``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Tuple

from ..config.model_config import ConfigError
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..registry import register_architecture
from .layered import need, opt_count, opt_number, read_eos, read_layers

# The design sets no limit on positions; the engine's tables need one.  EngineConfig.max_context overrides it.
DEFAULT_MAX_POSITION = 131072


@dataclass(frozen=True)
class FolavikConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    logit_scale: float
    logit_softcap: float
    layers: Tuple[Mapping[str, Any], ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITION
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


def _positive(obj: Any, key: str, where: str) -> float:
    v = need(obj, key, where, float)
    if not v > 0.0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _heads(mixer: Mapping[str, Any], where: str):
    heads = need(mixer, "heads", where, int)
    kv = need(mixer, "kv_heads", where, int) if mixer.get("kv_heads") is not None else heads    # no groups named: one key/value head a query head
    if heads % kv:
        raise ConfigError(f"config.json: {where}.heads {heads} must be a multiple of {where}.kv_heads {kv}")
    return heads, kv


def _rotary(mixer: Mapping[str, Any], where: str, dim: int, yarn: bool) -> PartSpec:
    rot = mixer.get("rot")
    if not rot:
        return PartSpec("none", {})
    w = where + ".rot"
    dims = need(rot, "dims", w, int)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}.dims {dims} must be even and at most {where}.dim {dim}")
    params = {"head_dim": dim, "theta": _positive(rot, "base", w), "rotary_dim": dims, "pairing": "halves", "theta_as_float32": False}
    scaling = rot.get("scaling")
    if scaling:
        sw = w + ".scaling"
        if yarn:
            params["yarn"] = {k: _positive(scaling, k, sw) for k in ("factor", "original", "fast", "slow")}
        else:
            params["scaling"] = {"factor": _positive(scaling, "factor", sw), "low_freq_factor": _positive(scaling, "low", sw),
                                 "high_freq_factor": _positive(scaling, "high", sw),
                                 "original_max_position_embeddings": _positive(scaling, "original", sw)}
    return PartSpec("rotary", params)


def _grouped(mixer: Mapping[str, Any], where: str, width: int, yarn: bool):
    heads, kv = _heads(mixer, where)
    dim = need(mixer, "dim", where, int)
    params = {"hidden_size": width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": opt_count(mixer, "vdim", dim, where) or dim,
              "scale": need(mixer, "scale", where, float)}
    names = {f"mixer.{n}_proj": f"mix.{n}" for n in ("q", "k", "v", "o")}
    return _rotary(mixer, where, dim, yarn), params, names, opt_count(mixer.get("mask") or {}, "size", 0, where + ".mask")


def _attention(i: int, mixer: Mapping[str, Any], width: int, eps: float):
    position, params, names, size = _grouped(mixer, f"layers[{i}].mixer", width, yarn=False)
    return position, PartSpec("value_attention", {**params, "chunk": size}), names


def _differential(i: int, mixer: Mapping[str, Any], width: int, eps: float):
    where = f"layers[{i}].mixer"
    position, params, names, size = _grouped(mixer, where, width, yarn=True)
    params.update({"window": size, "softcap": opt_number(mixer, "softcap", 0.0, where), "bias": True, "diff": need(mixer, "diff", where, float),
                   "norm_eps": eps})
    names.update({f"mixer.{n}_bias": f"mix.{n}.b" for n in ("q", "k", "v")})
    names.update({f"mixer.{n}": f"mix.{n}" for n in ("lq1", "lk1", "lq2", "lk2")})
    return position, PartSpec("differential_attention", params), names


def _latent(i: int, mixer: Mapping[str, Any], width: int, eps: float):
    where = f"layers[{i}].mixer"
    dim = need(mixer, "dim", where, int)
    params = {"hidden_size": width, "num_heads": need(mixer, "heads", where, int), "head_dim": dim, "rot_dim": 0,
              "value_dim": opt_count(mixer, "vdim", dim, where) or dim, "kv_rank": need(mixer, "kv_rank", where, int), "q_rank": 0,
              "scale": need(mixer, "scale", where, float), "norm_eps": eps, "out_gate": True}
    names = {"mixer.q_proj": "mix.q", "mixer.dkv_proj": "mix.dkv", "mixer.dkv_norm": "mix.dkv.norm", "mixer.uk_proj": "mix.uk",
             "mixer.uv_proj": "mix.uv", "mixer.g_proj": "mix.g", "mixer.o_proj": "mix.o"}
    return PartSpec("none", {}), PartSpec("latent_attention", params), names


_MIXERS = {"latent_attention": _latent, "attention": _attention, "attention_2": _differential}


def spec_from_config(cfg: FolavikConfig) -> ModelSpec:
    norm = PartSpec("layernorm", {"eps": cfg.norm_eps})
    layers = []
    for i, layer in enumerate(cfg.layers):
        kind = layer.get("type") if isinstance(layer, Mapping) else None
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: layers[{i}].type {kind!r}: this design has the mixers {sorted(_MIXERS)}")
        position, mixer, names = _MIXERS[kind](i, need(layer, "mixer", f"layers[{i}]"), cfg.hidden_size, cfg.norm_eps)
        names = {**names, "norm_in.weight": "norm1"}
        mlp = layer.get("mlp")
        ff = None
        if mlp:
            where = f"layers[{i}].mlp"
            if mlp.get("kind", "dense") != "dense":
                raise ConfigError(f"config.json: {where}.kind {mlp.get('kind')!r}: this design has the feed-forward 'dense'")
            ff = PartSpec("swiglu", {"hidden_size": cfg.hidden_size, "intermediate_size": need(mlp, "ff", where, int), "act": "gelu_tanh"})
            names.update({"norm_post.weight": "norm2", "feed_forward.gate_proj": "mlp.gate", "feed_forward.up_proj": "mlp.up",
                          "feed_forward.down_proj": "mlp.down"})
        layers.append(LayerSpec(block="prenorm" if ff is not None else "prenorm_mixer", mixer=mixer, feed_forward=ff, norm=norm,
                                position=position, prefix=f"l{i}.", names=names))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size, layers=tuple(layers),
        run_list=tuple(RunEntry(layer=i, cache=i, writes_cache=True) for i in range(len(layers))),
        embedding=PartSpec("table_normed", {"name": "embed", "norm": {"kind": "layernorm", "eps": cfg.norm_eps},
                                            "names": {"norm.weight": "embed.norm"}}),
        final_norm=PartSpec("layernorm", {"eps": cfg.norm_eps, "name": "final.norm"}),
        head=PartSpec("linear", {"tied": False, "name": "head", "softcap": cfg.logit_softcap, "scale": cfg.logit_scale}),
        max_position=cfg.max_position_embeddings, stop_token_ids=tuple(cfg.eos_token_ids),
    )


def config_from_dict(raw: Mapping[str, Any], generation_config=None) -> FolavikConfig:
    return FolavikConfig(
        architecture="Folavik", vocab_size=need(raw, "vocab", "config", int), hidden_size=need(raw, "width", "config", int),
        norm_eps=need(need(raw, "norm", "config"), "eps", "config.norm", float), logit_scale=opt_number(raw, "logit_scale", 1.0),
        logit_softcap=opt_number(raw, "logit_softcap", 0.0), layers=tuple(read_layers(raw)),
        eos_token_ids=read_eos(generation_config, raw),
    )


@register_architecture("Folavik")
def _build(raw, generation_config=None, strict=False):
    cfg = config_from_dict(raw, generation_config)
    return cfg, spec_from_config(cfg)
