"""Architecture builder for ``Kuvidra``: a decoder whose sublayers read one norm's output side by side and that mixes, layer
by layer, attention over a cached latent without positions and a matrix memory with exponential gates; a stretch of its
layers may run several times in a row; its layers are listed one by one in ``config.json``.

The configuration names its architecture as a string (``"architecture": "Kuvidra"``) and gives ``vocab``, ``width``,
``norm.eps``, ``loop`` and ``layers``: per layer its ``type`` (the kind of mixer), the mixer's sizes and constants under
``mixer``, and its feed-forward under ``mlp`` (null: the layer has none).  In this file's notation, with the float32 stream
x, e = embed[token] and N(y, w) = y / sqrt(mean y^2 + eps) * w:

* x = e; logits = embed N(x, w_final) (the head is the embedding's table);
* a layer: h = N(x, norm1); x <- x + mixer(h) + ff(h);
* ``loop`` {start, stop, times}: the stretch start .. stop - 1 is gone through ``times`` times on one set of tensors, each
  pass keeping its own cache and states; ahead of pass t, the first one included, x <- loop.in [x; e] + loop.step[t];
* mixer ``latent_attention``: :class:`~..parts.latent_attention.LatentAttention` without a rotated part, with a gate per head;
* mixer ``mlstm``: :class:`~..parts.recurrent.MatrixMemory`;
* feed-forward ``dense``: W_down gelu(W_up h), the erf form; ``moe``: :class:`~..parts.moe.RoutedExperts` with sigmoid scores
  that are not renormalised and multiply the chosen expert's input, gated experts W_down (silu(W_gate h) * (W_up h)), and a
  shared expert of the same form times sigmoid(w_sg . h).

This file is the only place that knows the configuration's keys and the checkpoint's tensor names (``embed``, ``loop.in``,
``loop.step``, ``final.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..config.model_config import ConfigError
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..registry import register_architecture
from .layered import need, opt_count, read_eos, read_layers, read_loop, run_order

# The design sets no limit on positions; the engine's tables need one.  EngineConfig.max_context overrides it.
DEFAULT_MAX_POSITION = 131072
MEMORY_DENOMINATOR_EPS = 1e-6      # added to the matrix memory's denominator


@dataclass(frozen=True)
class KuvidraConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]           # (start, stop, times) or None
    layers: Tuple[Mapping[str, Any], ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITION
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


def _latent_attention(i: int, mixer: Mapping[str, Any], width: int, eps: float):
    where = f"layers[{i}].mixer"
    if mixer.get("rot_dim") or mixer.get("rot"):
        raise ConfigError(f"config.json: {where}: this design's latent attention has no rotated part")
    dim = need(mixer, "dim", where, int)
    params = {"hidden_size": width, "num_heads": need(mixer, "heads", where, int), "head_dim": dim, "rot_dim": 0,
              "value_dim": opt_count(mixer, "vdim", dim, where) or dim, "kv_rank": need(mixer, "kv_rank", where, int),
              "q_rank": need(mixer, "q_rank", where, int), "scale": need(mixer, "scale", where, float), "norm_eps": eps, "head_gate": True}
    names = {"mixer.dq_proj": "mix.dq", "mixer.dq_norm": "mix.dq.norm", "mixer.uq_proj": "mix.uq", "mixer.dkv_proj": "mix.dkv",
             "mixer.dkv_norm": "mix.dkv.norm", "mixer.uk_proj": "mix.uk", "mixer.uv_proj": "mix.uv", "mixer.g_proj": "mix.g",
             "mixer.o_proj": "mix.o"}
    return PartSpec("latent_attention", params), names


def _mlstm(i: int, mixer: Mapping[str, Any], width: int, eps: float):
    where = f"layers[{i}].mixer"
    dim = need(mixer, "dim", where, int)
    cap = need(mixer, "gate_cap", where, float)
    if not cap > 0.0:
        raise ConfigError(f"config.json: {where}.gate_cap must be positive, got {cap!r}")
    params = {"hidden_size": width, "num_heads": need(mixer, "heads", where, int), "head_dim": dim,
              "value_dim": opt_count(mixer, "vdim", dim, where) or dim, "gate_cap": cap, "norm_eps": eps,
              "denominator_eps": MEMORY_DENOMINATOR_EPS}
    names = {f"mixer.{k}_proj": f"mix.{k}" for k in ("q", "k", "v", "g", "o", "i", "f")}
    names.update({"mixer.norm": "mix.norm", "mixer.i_bias": "mix.i.b", "mixer.f_bias": "mix.f.b"})
    return PartSpec("matrix_memory", params), names


_MIXERS = {"latent_attention": _latent_attention, "mlstm": _mlstm}


def _feed_forward(i: int, mlp: Mapping[str, Any], width: int):
    where = f"layers[{i}].mlp"
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        ff = PartSpec("mlp_act", {"hidden_size": width, "intermediate_size": need(mlp, "ff", where, int), "act": "gelu"})
        return ff, {"feed_forward.up": "mlp.up", "feed_forward.down": "mlp.down"}
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r}: this design has the feed-forwards 'dense' and 'moe'")
    router = need(mlp, "router", where)
    experts, top = need(router, "experts", where + ".router", int), need(router, "top", where + ".router", int)
    if top > experts:
        raise ConfigError(f"config.json: {where}.router.top {top} exceeds the {experts} experts")
    shared = mlp.get("shared")
    params = {"hidden_size": width, "expert_ff": need(need(mlp, "expert", where), "ff", where + ".expert", int), "num_experts": experts,
              "top": top, "act": "swiglu", "score": "sigmoid", "weight_on_input": True,
              "shared_ff": need(shared, "ff", where + ".shared", int) if shared else 0, "shared_gate": bool(shared)}
    names = {"feed_forward.router": "mlp.router", "feed_forward.shared.gate_proj": "mlp.shared.gate", "feed_forward.shared.up": "mlp.shared.up",
             "feed_forward.shared.down": "mlp.shared.down", "feed_forward.shared.gate": "mlp.shared.sg"}
    for e in range(experts):
        for m in ("gate", "up", "down"):
            names[f"feed_forward.experts.{e}.{m}"] = f"mlp.e{e}.{m}"
    return PartSpec("routed_experts", params), names


def spec_from_config(cfg: KuvidraConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"eps": cfg.norm_eps})
    layers = []
    for i, layer in enumerate(cfg.layers):
        kind = layer.get("type")
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: layers[{i}].type {kind!r}: this design has the mixers {sorted(_MIXERS)}")
        mixer, names = _MIXERS[kind](i, need(layer, "mixer", f"layers[{i}]"), cfg.hidden_size, cfg.norm_eps)
        names = dict(names, **{"norm_in.weight": "norm1"})
        mlp, ff = layer.get("mlp"), None
        if mlp:
            ff, ff_names = _feed_forward(i, mlp, cfg.hidden_size)
            names.update(ff_names)
        layers.append(LayerSpec(block="parallel", mixer=mixer, feed_forward=ff, norm=norm, position=PartSpec("none", {}), prefix=f"l{i}.",
                                names=names))
    # every run keeps a cache or state of its own, also the later passes over a layer
    runs = tuple(RunEntry(layer=i, cache=n, writes_cache=True, enter=t) for n, (i, t) in enumerate(run_order(len(layers), cfg.loop)))
    pass_input = None
    if cfg.loop is not None:
        pass_input = PartSpec("step_projection", {"times": cfg.loop[2], "names": {"in_proj": "loop.in", "steps": "loop.step"}})
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size,
        layers=tuple(layers), run_list=runs, embedding=PartSpec("table", {"name": "embed"}),
        final_norm=PartSpec("rmsnorm", {"eps": cfg.norm_eps, "name": "final.norm"}), head=PartSpec("linear", {"tied": True}),
        max_position=cfg.max_position_embeddings, stop_token_ids=tuple(cfg.eos_token_ids), pass_input=pass_input,
    )


def config_from_dict(raw: Mapping[str, Any], generation_config: Optional[Mapping[str, Any]] = None) -> KuvidraConfig:
    layers = read_layers(raw)
    return KuvidraConfig(
        architecture="Kuvidra", vocab_size=need(raw, "vocab", "config", int), hidden_size=need(raw, "width", "config", int),
        norm_eps=need(need(raw, "norm", "config"), "eps", "config.norm", float), loop=read_loop(raw, len(layers)), layers=tuple(layers),
        eos_token_ids=read_eos(generation_config, raw),
    )


@register_architecture("Kuvidra")
def _build(raw, generation_config=None, strict=False):
    cfg = config_from_dict(raw, generation_config)
    return cfg, spec_from_config(cfg)
