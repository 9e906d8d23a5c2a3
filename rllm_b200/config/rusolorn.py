"""Rusolorn: typed configuration from config.json and the model it describes.

A decoder whose layers are listed one by one in config.json (`layers`: each entry names its mixer
`type`, the mixer's sizes and its feed-forward, or none).  A layer norms the stream once and both
sublayers read that: x <- x + m (mixer(h) + ff(h)), h = norm1(x), with one `residual_mult` m for the
model.  The norms of the stream are Dynamic Tanh (tanh(alpha x) w + b).  Behind the sublayers every
layer joins a per-token input: a second table `side.embed` holds `token_side.dim` entries per token and
layer, which the stream gates (tanh form of gelu) and a projection and an RMS norm bring back to the
stream's width, again times m.  The embedding row is multiplied by `embedding.scale`; the LM head is the
embedding table.

Mixer ``parallel``: half the sum of two RMS-normed outputs.  Left, grouped attention: an RMS norm over
the whole query and the whole key projection, values that are the keys as projected, no positions, a
sliding window of mask.size keys.  Right, the gated delta rule behind short causal convolutions.
Feed-forward ``moe``: clamped gated units chosen by softmax scores inside the best groups of experts, and
a shared one (`shared`, with a size and a limit of its own).

config.json keys: architecture, vocab, width, embedding.scale, layers[].{type, mixer.{left, right}, mlp},
norm.eps, residual_mult, token_side.dim.
Tensors: embed, side.embed, final.norm (and .alpha, .b) and l<i>.{norm1, mix.*, mlp.*, side.*}.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, LayerSpec, ModelConfig, ModelSpec, PartSpec, RunEntry, optional, require

GLU_ALPHA = 1.702          # the design fixes these: the gated unit's sigmoid slope and the shift of its up branch,
GLU_SHIFT = 1.0
GROUP_BEST = 1             # how many of a group's scores make the group's score,
WEIGHT_EPS = 1e-20         # what is added to the sum of the chosen scores before the division,
UNIT_EPS = 1e-6            # and to the sum of squares of a query or key head before it is made a unit vector


def _section(d, key, where):
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where}: required section '{key}' is missing")
    return v


def _positive(d, keys, where):
    for k in keys:
        if require(d, k, int, where) <= 0:
            raise ConfigError(f"{where}: '{k}' must be positive")


def _check_heads(sec, where):
    _positive(sec, ("heads", "kv_heads", "dim", "vdim"), where)
    if sec["heads"] % sec["kv_heads"]:
        raise ConfigError(f"{where}: heads {sec['heads']} is not a multiple of kv_heads {sec['kv_heads']}")


def _check_mixer(mx, where):
    left, lw = _section(mx, "left", where), where + ".left"
    _check_heads(left, lw)
    if left["vdim"] != left["dim"]:
        raise ConfigError(f"{lw}: 'vdim' must equal 'dim' (the values are the keys)")
    require(left, "scale", float, lw)
    mask = left.get("mask")
    if mask is not None:
        if not isinstance(mask, Mapping):
            raise ConfigError(f"{lw}.mask must be an object or null")
        _positive(mask, ("size",), lw + ".mask")
    right, rw = _section(mx, "right", where), where + ".right"
    _check_heads(right, rw)
    _positive(right, ("conv",), rw)


def _check_unit(sec, where):
    _positive(sec, ("ff",), where)
    if not require(sec, "limit", float, where) > 0:
        raise ConfigError(f"{where}: 'limit' must be positive")


def _check_mlp(mlp, where):
    kind = require(mlp, "kind", str, where)
    if kind != "moe":
        raise ConfigError(f"{where}: kind {kind!r} is not supported (moe)")
    _check_unit(_section(mlp, "expert", where), where + ".expert")
    r, rw = _section(mlp, "router", where), where + ".router"
    _positive(r, ("experts", "top"), rw)
    groups = r.get("groups")
    count = keep = 1
    if groups is not None:
        if not isinstance(groups, Mapping):
            raise ConfigError(f"{rw}.groups must be an object or null")
        _positive(groups, ("count", "keep"), rw + ".groups")
        count, keep = groups["count"], groups["keep"]
    if r["experts"] % count or keep > count:
        raise ConfigError(f"{rw}: {r['experts']} experts do not form {count} equal groups of which {keep} are kept")
    if r["top"] > keep * (r["experts"] // count):
        raise ConfigError(f"{rw}: 'top' {r['top']} exceeds the experts of the kept groups")
    if mlp.get("shared") is not None:
        _check_unit(_section(mlp, "shared", where), where + ".shared")


@dataclass(frozen=True)
class RusolornConfig(ModelConfig):
    vocab: int
    width: int
    layers: tuple                  # of plain dicts as config.json gives them (validated)
    norm_eps: float
    residual_mult: float = 1.0
    embed_scale: float = 1.0
    side_dim: int = 0              # token_side.dim; 0: the layers have no token input
    architecture: str = "Rusolorn"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RusolornConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: required key 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{where} must be an object")
            typ = require(layer, "type", str, where)
            if typ != "parallel":
                raise ConfigError(f"{where}: mixer type {typ!r} is not supported (parallel)")
            _check_mixer(_section(layer, "mixer", where), where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise ConfigError(f"{where}.mlp must be an object or null")
                _check_mlp(mlp, where + ".mlp")
            checked.append(copy.deepcopy(dict(layer)))
        norm = _section(d, "norm", "config.json")
        emb = d.get("embedding") or {}
        side = d.get("token_side")
        for key, v in (("embedding", emb), ("token_side", side)):
            if v is not None and not isinstance(v, Mapping):
                raise ConfigError(f"config.json: '{key}' must be an object")
        if side is not None:
            _positive(side, ("dim",), "config.json: token_side")
        cfg = cls(vocab=require(d, "vocab", int), width=require(d, "width", int), layers=tuple(checked),
                  norm_eps=require(norm, "eps", float, "config.json: norm"),
                  residual_mult=optional(d, "residual_mult", float, 1.0),
                  embed_scale=optional(emb, "scale", float, 1.0, "config.json: embedding"),
                  side_dim=side["dim"] if side is not None else 0)
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if not cfg.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "embedding": {"scale": self.embed_scale}, "layers": copy.deepcopy(list(self.layers)),
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult}
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        return d

    # ------------------------------------------------------------------ the model as data
    def _mixer(self, i: int, mx) -> PartSpec:
        p, d, eps = f"l{i}.mix.", self.width, self.norm_eps
        left, right = mx["left"], mx["right"]
        attention = PartSpec("gated_attention", {
            "hidden_size": d, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"],
            "v_head_dim": left["vdim"], "scale": float(left["scale"]), "qk_norm": "row", "eps": eps,
            "window": (left.get("mask") or {}).get("size", 0), "tie_values": True}, p + "left.")
        delta = PartSpec("gated_delta", {
            "hidden_size": d, "num_heads": right["heads"], "num_kv_heads": right["kv_heads"], "head_dim": right["dim"],
            "v_head_dim": right["vdim"], "conv": right["conv"], "q_scale": float(right["dim"]) ** -0.5,
            "unit_eps": UNIT_EPS, "eps": eps, "gate": "silu"}, p + "right.")
        norm = lambda side: PartSpec("rms_norm", {"size": d, "eps": eps, "tensor": f"{p}{side}.out"})
        return PartSpec("parallel", {"left": attention, "right": delta, "left_scale": 0.5, "right_scale": 0.5,
                                     "left_norm": norm("left"), "right_norm": norm("right")}, p)

    def _ffn(self, i: int, mlp):
        if mlp is None:
            return None
        r, shared = mlp["router"], mlp.get("shared")
        groups = r.get("groups") or {"count": 1, "keep": 1}
        form = lambda sec: {"limit": float(sec["limit"]), "alpha": GLU_ALPHA, "shift": GLU_SHIFT}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "num_experts": r["experts"],
            "top_k": r["top"], "n_groups": groups["count"], "keep_groups": groups["keep"], "group_best": GROUP_BEST,
            "score": "softmax", "correction": False, "normalize": True, "weight_eps": WEIGHT_EPS, "route_scale": 1.0,
            "expert_form": form(mlp["expert"]), "shared_size": shared["ff"] if shared else 0, "shared_gate": False,
            "shared_form": form(shared) if shared else None}, f"l{i}.mlp.")

    def model_spec(self) -> ModelSpec:
        d, n = self.width, len(self.layers)
        norm = lambda name: PartSpec("dynamic_tanh", {"size": d, "tensor": name})
        layers = []
        for i, layer in enumerate(self.layers):
            side = None if not self.side_dim else PartSpec("token_table", {
                "hidden_size": d, "vocab_size": self.vocab, "dim": self.side_dim, "tensor": "side.embed", "part": i,
                "parts": n, "eps": self.norm_eps}, f"l{i}.side.")
            layers.append(LayerSpec(block="shared_norm", mixer=self._mixer(i, layer["mixer"]),
                                    ffn=self._ffn(i, layer.get("mlp")), norms={"mixer": norm(f"l{i}.norm1")}, side=side,
                                    block_params={"residual_mult": self.residual_mult}))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=d,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": d, "tensor": "embed",
                                             "scale": self.embed_scale}),
            layers=tuple(layers), run_order=tuple(RunEntry(i) for i in range(n)), final_norm=norm("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": d, "tied_to": "embed",
                                         "tensor": "head"}),
            max_position=0)
