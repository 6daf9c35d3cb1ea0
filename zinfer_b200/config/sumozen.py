"""Typed configuration of the Sumozen design and its model spec.

A Sumozen model is a pre-norm decoder, x <- x + mixer(norm1(x)), then x <- x + ff(norm2(x)); the norms' stored weights
lie around zero (the multiplier is 1 + w).  A layer's ``type`` names its mixer:

* ``parallel``: two mixers side by side on the same input, left_scale * left + right_scale * right.  ``left`` is
  grouped-query attention with biases on all four projections, a causal convolution of ``conv`` taps on every channel of
  q, k and v before the rotation, a rotation of the first ``rot.dims`` dimensions of a head in neighbouring pairs with
  ramped frequency scaling (``rot.scaling``: factor, original, fast, slow), an explicit ``scale``, a capped score
  (``softcap``) and an ordinary softmax over every earlier key.  ``right`` is a gated delta rule behind convolutions of
  ``conv`` taps with one decay per head and a full silu gate.
* ``mamba2``: a state-space mixer (``heads`` of ``vdim`` channels, a state of ``state`` per channel, ``groups`` of B and C, a
  convolution with a bias, ``norm_groups`` parts of the gated norm).

The feed-forward is a mixture of silu-gated experts with sigmoid scores, not renormalised, whose weights multiply the
experts' inputs, beside a shared expert with a sigmoid gate per token; or absent.  config.json gives every size and every
constant that may differ between models; the tensor names (``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``, ``head``) are fixed.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Optional

from .luvavik import _positive
from .qwen3 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Sumozen"
DEFAULT_MAX_POSITIONS = 1 << 17       # the design has no position limit; the engine needs one for its tables
MAX_TAPS = 17                         # of a short convolution

_LEFT_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "conv")
_RIGHT_KEYS = ("heads", "kv_heads", "dim", "vdim", "conv")
_MAMBA2_KEYS = ("heads", "vdim", "state", "groups", "norm_groups", "conv")


def _taps_ok(where: str, m: dict) -> None:
    if m["conv"] > MAX_TAPS:
        raise ConfigError(f"config.json: {where}.conv: a short convolution has at most {MAX_TAPS} taps, got {m['conv']}")


@dataclass(frozen=True)
class SumozenConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[dict, ...]               # as in config.json: type, mixer, mlp
    norm_eps: float
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: tuple[int, ...] = field(default_factory=tuple)
    model_type: str = "sumozen"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: dict) -> "SumozenConfig":
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
                  max_position_embeddings=int(d.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)),
                  eos_token_id=tuple(int(t) for t in (eos or ())))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0:
            raise ConfigError("vocab and width must be positive")
        if not self.norm_eps >= 0.0:
            raise ConfigError(f"norm.eps must be >= 0, got {self.norm_eps}")
        for i, layer in enumerate(self.layers):
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in ("parallel", "mamba2"):
                raise ConfigError(f"config.json: layer {i} has the unknown mixer type {kind!r}; known: parallel, mamba2")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: layer {i} lacks its mixer's sizes")
            where = f"layers[{i}].mixer"
            if kind == "mamba2":
                _positive(where, m, _MAMBA2_KEYS)
                _taps_ok(where, m)
                if m["heads"] % m["groups"]:
                    raise ConfigError(f"config.json: {where}: {m['heads']} heads do not divide into {m['groups']} groups")
                if m["heads"] * m["vdim"] % m["norm_groups"]:
                    raise ConfigError(f"config.json: {where}: {m['heads'] * m['vdim']} channels do not divide into {m['norm_groups']} norm groups")
            else:
                self._parallel_ok(where, m)
            self._mlp_ok(i, layer.get("mlp"))

    @staticmethod
    def _parallel_ok(where: str, m: dict) -> None:
        for side, keys in (("left", _LEFT_KEYS), ("right", _RIGHT_KEYS)):
            if not isinstance(m.get(side), dict):
                raise ConfigError(f"config.json: {where} lacks {side!r}")
            _positive(f"{where}.{side}", m[side], keys)
            _taps_ok(f"{where}.{side}", m[side])
            if m[side]["heads"] % m[side]["kv_heads"]:
                raise ConfigError(f"config.json: {where}.{side}: {m[side]['heads']} heads do not divide into {m[side]['kv_heads']} kv heads")
        for k in ("left_scale", "right_scale"):
            if k not in m:
                raise ConfigError(f"config.json: {where} lacks {k!r}")
        left = m["left"]
        if left.get("softcap") is not None:
            _positive(f"{where}.left", left, ("softcap",))
        rot = left.get("rot")
        if rot is not None:
            _positive(f"{where}.left.rot", rot, ("base", "dims"))
            if rot["dims"] % 2 or rot["dims"] > left["dim"]:
                raise ConfigError(f"config.json: {where}.left.rot.dims {rot['dims']} must be even and at most dim")
            if rot.get("scaling") is not None:
                _positive(f"{where}.left.rot.scaling", rot["scaling"], ("factor", "original", "fast", "slow"))

    @staticmethod
    def _mlp_ok(i: int, mlp: Optional[dict]) -> None:
        if mlp is None:
            return
        if mlp.get("kind", "moe") != "moe":
            raise ConfigError(f"config.json: layer {i} has the unknown feed-forward kind {mlp.get('kind')!r}; known: moe")
        _positive(f"layers[{i}].mlp.expert", mlp.get("expert") or {}, ("ff",))
        router = mlp.get("router") or {}
        _positive(f"layers[{i}].mlp.router", router, ("experts", "top"))
        if router["top"] > router["experts"]:
            raise ConfigError(f"config.json: layer {i}: {router['top']} of {router['experts']} experts cannot be chosen")
        if mlp.get("shared") is not None:
            _positive(f"layers[{i}].mlp.shared", mlp["shared"], ("ff",))

    def describe(self) -> list[str]:
        """Lines for the command line's model inspection."""
        lines = [f"hidden_size: {self.hidden_size}", f"vocab_size: {self.vocab_size}", f"num_layers: {len(self.layers)}",
                 f"norm_eps: {self.norm_eps:e}"]
        flat = lambda m: ", ".join(f"{k}={v}" for k, v in sorted(m.items()) if not isinstance(v, dict))
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] == "mamba2":
                mixer = flat(m)
            else:
                rot = m["left"].get("rot")
                mixer = (f"left {m['left_scale']} x attention ({flat(m['left'])}" + (f", rot {flat(rot)}" if rot else "")
                         + f"); right {m['right_scale']} x delta rule ({flat(m['right'])})")
            mlp = layer.get("mlp")
            if mlp is None:
                ff = "none"
            else:
                r = mlp["router"]
                ff = (f"moe experts={r['experts']} top={r['top']} ff={mlp['expert']['ff']}"
                      + (f" shared ff={mlp['shared']['ff']}" if mlp.get("shared") else ""))
            lines.append(f"layer {i}: {layer['type']} ({mixer}); feed-forward: {ff}")
        return lines

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                             "layers": [copy.deepcopy(layer) for layer in self.layers], "norm": {"eps": self.norm_eps}}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d


# ---------------------------------------------------------------------- the family
def _mamba2_spec(cfg: SumozenConfig, m: dict) -> PartSpec:
    return PartSpec("mamba2", {
        "hidden_size": cfg.hidden_size, "num_heads": int(m["heads"]), "vdim": int(m["vdim"]), "state": int(m["state"]),
        "groups": int(m["groups"]), "norm_groups": int(m["norm_groups"]), "conv_taps": int(m["conv"]), "norm_eps": cfg.norm_eps})


def _parallel_spec(cfg: SumozenConfig, m: dict) -> PartSpec:
    left, right = m["left"], m["right"]
    position, rot = None, left.get("rot")
    if rot is not None:
        scaling = {"kind": "ramp", **{k: float(v) for k, v in rot["scaling"].items()}} if rot.get("scaling") else None
        position = PartSpec("rope", {"head_dim": int(rot["dims"]), "theta": float(rot["base"]), "scaling": scaling,
                                     "pairing": "neighbours", "max_positions": cfg.max_position_embeddings})
    attention = PartSpec("gqa_attention", {
        "hidden_size": cfg.hidden_size, "num_heads": int(left["heads"]), "num_kv_heads": int(left["kv_heads"]),
        "head_dim": int(left["dim"]), "value_dim": int(left["vdim"]), "qk_norm_eps": None, "window": None, "position": position,
        "scale": float(left["scale"]), "softcap": left.get("softcap"), "bias": True, "conv_taps": int(left["conv"]),
        "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})
    delta = PartSpec("gated_delta_rule", {
        "hidden_size": cfg.hidden_size, "num_heads": int(right["heads"]), "num_kv_heads": int(right["kv_heads"]),
        "dim": int(right["dim"]), "vdim": int(right["vdim"]), "conv_taps": int(right["conv"]), "norm_eps": cfg.norm_eps,
        "decay": "head", "gate": "silu"})
    return PartSpec("parallel_mixer", {"left": attention, "right": delta, "left_scale": float(m["left_scale"]),
                                       "right_scale": float(m["right_scale"]), "left_name": "left.", "right_name": "right."})


def _ffn_spec(cfg: SumozenConfig, layer: dict) -> Optional[PartSpec]:
    mlp = layer.get("mlp")
    if mlp is None:
        return None
    H, router, shared = cfg.hidden_size, mlp["router"], None
    if mlp.get("shared") is not None:
        shared = PartSpec("swiglu_mlp", {"hidden_size": H, "intermediate_size": int(mlp["shared"]["ff"]), "activation": "silu",
                                         "names": ("gate", "up", "down")})
    return PartSpec("routed_experts", {
        "hidden_size": H, "intermediate_size": int(mlp["expert"]["ff"]), "experts": int(router["experts"]), "top": int(router["top"]),
        "score": "sigmoid", "renormalize": False, "activation": "silu_gated", "weights_on": "input", "expert_names": "e{}.",
        "shared": shared, "shared_name": "shared.", "shared_gate": "sg" if shared is not None else None})


def sumozen_model_spec(cfg: SumozenConfig) -> ModelSpec:
    H = cfg.hidden_size
    norm = lambda tensor: PartSpec("rmsnorm", {"size": H, "eps": cfg.norm_eps, "tensor": tensor, "one_plus": True})
    layers = []
    for i, layer in enumerate(cfg.layers):
        mixer = _mamba2_spec(cfg, layer["mixer"]) if layer["type"] == "mamba2" else _parallel_spec(cfg, layer["mixer"])
        ffn = _ffn_spec(cfg, layer)
        block = PartSpec("prenorm_block", {
            "mixer": mixer, "mixer_norm": norm("norm1"), "mixer_name": "mix.", "feed_forward": ffn,
            "ffn_norm": norm("norm2") if ffn is not None else None, "ffn_name": "mlp.", "mixer_norm_name": "",
            "ffn_norm_name": "", "verbatim_names": True})
        layers.append(LayerSpec(block=block, prefix=f"l{i}."))
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=cfg.vocab_size, hidden_size=H, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "hidden_size": H, "name": "embed", "suffix": ""}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=PartSpec("rmsnorm", {"size": H, "eps": cfg.norm_eps, "tensor": "norm", "prefix": "final.", "one_plus": True}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab_size, "hidden_size": H, "name": "head", "suffix": "", "tied_to": None}),
        eos_token_ids=cfg.eos_token_id)
