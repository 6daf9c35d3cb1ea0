"""Typed configuration of the Kesitar design and its model spec.

A Kesitar model is a decoder whose layers norm each sublayer's input and its output, x <- x + N(mixer(N(x))), then
x <- x + N(ff(N(x))), with layer norms that have a weight and no bias (``norm1``, ``norm1b``, ``norm2``, ``norm2b``).  The
embedding is scaled (``embedding.scale``) and its table, unscaled, is the output head, whose logits are multiplied by
``logit_scale``.  The mixers: ``attention`` (grouped queries; biases on q, k and v; an RMS norm per query and key head; a
rotation of the head's first ``rot.dims`` dimensions; an explicit ``scale``; a window of ``mask.size`` tokens beside which
each block of ``mask.pool`` tokens, once its last token has left the window, stands in as the mean key and value; a softmax
whose denominator counts one more than its keys; with ``v_mix`` the values are mixed with those of the first such layer)
and ``hgrn2`` (a matrix-valued state per head whose forget gate decides what is written).  The feed-forward is dense
and gated with silu, or absent.  config.json gives every size and every constant that may differ between models; the
tensor names (``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``) are fixed.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Optional

from .luvavik import _positive
from .qwen3 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Kesitar"
DEFAULT_MAX_POSITIONS = 1 << 17       # the design has no position limit; the engine needs one for its tables
SINK = 1.0                            # what the softmax's denominator counts beside its keys: fixed by the design

_ATTENTION_KEYS = ("heads", "kv_heads", "dim", "scale")
_HGRN2_KEYS = ("heads", "dim", "vdim")


@dataclass(frozen=True)
class KesitarConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[dict, ...]               # as in config.json: type, mixer, mlp
    norm_eps: float
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: tuple[int, ...] = field(default_factory=tuple)
    model_type: str = "kesitar"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: dict) -> "KesitarConfig":
        for k in ("vocab", "width", "layers", "norm"):
            if k not in d:
                raise ConfigError(f"config.json lacks required key {k!r}")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: `layers` must be a list with at least one layer")
        if "eps" not in d["norm"]:
            raise ConfigError("config.json: norm lacks 'eps'")
        eos = d.get("eos_token_id", ())
        if isinstance(eos, int):
            eos = (eos,)
        cfg = cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                  layers=tuple(copy.deepcopy(layer) for layer in d["layers"]), norm_eps=float(d["norm"]["eps"]),
                  embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)),
                  max_position_embeddings=int(d.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)),
                  eos_token_id=tuple(int(t) for t in (eos or ())))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0:
            raise ConfigError("vocab and width must be positive")
        if not self.norm_eps >= 0.0:
            raise ConfigError(f"norm.eps must be >= 0, got {self.norm_eps}")
        mixed = None                       # (layer, elements of its values) of the first layer that mixes values
        for i, layer in enumerate(self.layers):
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in ("attention", "hgrn2"):
                raise ConfigError(f"config.json: layer {i} has the unknown mixer type {kind!r}; known: attention, hgrn2")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: layer {i} lacks its mixer's sizes")
            where = f"layers[{i}].mixer"
            if kind == "hgrn2":
                _positive(where, m, _HGRN2_KEYS)
            else:
                _positive(where, m, _ATTENTION_KEYS)
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"config.json: {where}: {m['heads']} heads do not divide into {m['kv_heads']} kv heads")
                vdim = int(m.get("vdim", m["dim"]))
                if vdim <= 0:
                    raise ConfigError(f"config.json: {where}.vdim must be positive")
                rot = m.get("rot")
                if rot is not None:
                    _positive(f"{where}.rot", rot, ("base", "dims"))
                    if rot["dims"] % 2 or rot["dims"] > m["dim"]:
                        raise ConfigError(f"config.json: {where}.rot.dims {rot['dims']} must be even and at most dim")
                mask = m.get("mask")
                if mask is not None:
                    _positive(f"{where}.mask", mask, ("size",))
                    if mask.get("pool") is not None:
                        _positive(f"{where}.mask", mask, ("pool",))
                if m.get("v_mix"):
                    shape = (int(m["kv_heads"]), vdim)
                    if mixed is None:
                        mixed = (i, shape)
                    elif mixed[1] != shape:
                        raise ConfigError(f"config.json: {where}.v_mix: the values of layer {mixed[0]}, which these are mixed with, "
                                          f"are {mixed[1][0]} heads of {mixed[1][1]}, not {shape[0]} of {shape[1]}")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind", "dense") != "dense":
                raise ConfigError(f"config.json: layer {i} has the unknown feed-forward kind {mlp.get('kind')!r}; known: dense")
            _positive(f"layers[{i}].mlp", mlp, ("ff",))

    def describe(self) -> list[str]:
        """Lines for the command line's model inspection."""
        lines = [f"hidden_size: {self.hidden_size}", f"vocab_size: {self.vocab_size}", f"num_layers: {len(self.layers)}",
                 f"norm_eps: {self.norm_eps:e}", f"embedding_scale: {self.embedding_scale}", f"logit_scale: {self.logit_scale}"]
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] == "hgrn2":
                mixer = f"heads={m['heads']} dim={m['dim']} vdim={m['vdim']}"
            else:
                mask, rot = m.get("mask"), m.get("rot")
                mixer = (f"heads={m['heads']} kv_heads={m['kv_heads']} dim={m['dim']} vdim={m.get('vdim', m['dim'])} scale={m['scale']}"
                         + (f" rot dims={rot['dims']} base={rot['base']}" if rot else " no rotation")
                         + (f" window={mask['size']}" + (f" pooled blocks of {mask['pool']}" if mask.get("pool") else "") if mask else " no window")
                         + (" mixed values" if m.get("v_mix") else ""))
            mlp = layer.get("mlp")
            lines.append(f"layer {i}: {layer['type']} ({mixer}); feed-forward: " + (f"dense ff={mlp['ff']}" if mlp is not None else "none"))
        return lines

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                             "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
                             "layers": [copy.deepcopy(layer) for layer in self.layers], "norm": {"eps": self.norm_eps}}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d


# ---------------------------------------------------------------------- the family
def _attention_spec(cfg: KesitarConfig, m: dict, first_mix: bool) -> PartSpec:
    rot, mask = m.get("rot"), m.get("mask") or {}
    position = None
    if rot is not None:
        position = PartSpec("rope", {"head_dim": int(rot["dims"]), "theta": float(rot["base"]),
                                     "max_positions": cfg.max_position_embeddings})
    return PartSpec("gqa_attention", {
        "hidden_size": cfg.hidden_size, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
        "head_dim": int(m["dim"]), "value_dim": int(m.get("vdim", m["dim"])), "qk_norm_eps": cfg.norm_eps, "bias": "qkv",
        "window": int(mask["size"]) if mask else None, "pool": int(mask.get("pool") or 0), "position": position,
        "scale": float(m["scale"]), "sink": SINK,
        "value_mix": {"tensor": "vmix", "first": first_mix} if m.get("v_mix") else None,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}})


def _hgrn2_spec(cfg: KesitarConfig, m: dict) -> PartSpec:
    return PartSpec("hgrn2", {"hidden_size": cfg.hidden_size, "num_heads": int(m["heads"]), "dim": int(m["dim"]),
                              "vdim": int(m["vdim"]), "norm_eps": cfg.norm_eps})


def _ffn_spec(cfg: KesitarConfig, layer: dict) -> Optional[PartSpec]:
    mlp = layer.get("mlp")
    if mlp is None:
        return None
    return PartSpec("swiglu_mlp", {"hidden_size": cfg.hidden_size, "intermediate_size": int(mlp["ff"]), "activation": "silu",
                                   "names": ("gate", "up", "down")})


def kesitar_model_spec(cfg: KesitarConfig) -> ModelSpec:
    H = cfg.hidden_size
    norm = lambda tensor: PartSpec("layernorm", {"size": H, "eps": cfg.norm_eps, "tensor": tensor})
    layers, seen_mix = [], False
    for i, layer in enumerate(cfg.layers):
        m = layer["mixer"]
        if layer["type"] == "hgrn2":
            mixer = _hgrn2_spec(cfg, m)
        else:
            mixer = _attention_spec(cfg, m, first_mix=not seen_mix)
            seen_mix = seen_mix or bool(m.get("v_mix"))
        ffn = _ffn_spec(cfg, layer)
        block = PartSpec("sandwich_block", {
            "mixer": mixer, "mixer_norm": norm("norm1"), "mixer_post_norm": norm("norm1b"), "mixer_name": "mix.",
            "feed_forward": ffn, "ffn_norm": norm("norm2") if ffn is not None else None,
            "ffn_post_norm": norm("norm2b") if ffn is not None else None, "ffn_name": "mlp.", "mixer_norm_name": "",
            "mixer_post_norm_name": "", "ffn_norm_name": "", "ffn_post_norm_name": "", "verbatim_names": True})
        layers.append(LayerSpec(block=block, prefix=f"l{i}."))
    embedding = {"vocab_size": cfg.vocab_size, "hidden_size": H, "name": "embed", "suffix": "", "scale": cfg.embedding_scale}
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=cfg.vocab_size, hidden_size=H, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", embedding), layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=PartSpec("layernorm", {"size": H, "eps": cfg.norm_eps, "tensor": "norm", "prefix": "final."}),
        # the embedding's table (without its scale) is the output head; a file holds no table of its own for it
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab_size, "hidden_size": H, "name": "head", "suffix": "", "tied_to": "embed",
                                  "scale": cfg.logit_scale}),
        eos_token_ids=cfg.eos_token_id)
