"""Pibavik: typed configuration from config.json and the model it describes.

A pre-norm decoder whose layers are listed one by one in config.json (`layers`: each entry names its mixer
`type`, the mixer's sizes and its feed-forward, or none).  The embedding row is multiplied by
`embedding.scale`; the LM head is a matrix of its own.  The model sets no limit on positions.

Mixers: ``attention`` (grouped heads with value heads of their own size, a sliding window of mask.size keys, a
slope per head 2^(-8 (h+1) / heads) times the distance taken off every score; with `kv_from: j` the layer has
no keys and values of its own and reads those of layer j), ``latent_attention`` (queries through a normed latent of
q_rank entries, keys and values through another of kv_rank entries, no positions; causal) and ``parallel``
(left_scale times a windowed attention with an RMS norm per query and key head, rotated heads and a gate per
head, plus right_scale times Mamba-2).  Feed-forward ``moe``: experts W_down relu(W_up h)^2 chosen by sigmoid
scores, a token's score for an expert multiplying what the expert reads, and a shared one.

config.json keys: architecture, vocab, width, embedding.scale, layers[].{type, mixer, mlp}, norm.eps.
Tensors: embed, head, final.norm and l<i>.{norm1, norm2, mix.*, mlp.*}.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, LayerSpec, ModelConfig, ModelSpec, PartSpec, RunEntry, optional, require

SLOPE_SPAN = 8.0           # the design fixes these: head h of H loses 2^(-SLOPE_SPAN (h + 1) / H) per position of distance,
EXPERT_ACT = "relu2"       # and the experts' activation


def _section(d, key, where):
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where}: required section '{key}' is missing")
    return v


def _positive(d, keys, where):
    for k in keys:
        if require(d, k, int, where) <= 0:
            raise ConfigError(f"{where}: '{k}' must be positive")


def _check_mask(sec, where):
    mask = sec.get("mask")
    if mask is not None:
        if not isinstance(mask, Mapping):
            raise ConfigError(f"{where}.mask must be an object or null")
        _positive(mask, ("size",), where + ".mask")


def _check_heads(sec, where):
    _positive(sec, ("heads", "kv_heads", "dim", "vdim"), where)
    if sec["heads"] % sec["kv_heads"]:
        raise ConfigError(f"{where}: heads {sec['heads']} is not a multiple of kv_heads {sec['kv_heads']}")
    require(sec, "scale", float, where)
    _check_mask(sec, where)


def _check_rot(sec, where):
    rot = sec.get("rot")
    if rot is None:
        return
    if not isinstance(rot, Mapping):
        raise ConfigError(f"{where}.rot must be an object or null")
    if require(rot, "dims", int, where + ".rot") <= 0 or rot["dims"] % 2 or rot["dims"] > sec["dim"]:
        raise ConfigError(f"{where}.rot: 'dims' must be positive, even and at most the head size {sec['dim']}")
    if not require(rot, "base", float, where + ".rot") > 0:
        raise ConfigError(f"{where}.rot: 'base' must be positive")


def _check_parallel(mx, where):
    left, lw = _section(mx, "left", where), where + ".left"
    _check_heads(left, lw)
    _check_rot(left, lw)
    right, rw = _section(mx, "right", where), where + ".right"
    _positive(right, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), rw)
    if right["heads"] % right["groups"]:
        raise ConfigError(f"{rw}: heads {right['heads']} is not a multiple of groups {right['groups']}")
    if right["heads"] * right["vdim"] % right["norm_groups"]:
        raise ConfigError(f"{rw}: heads * vdim is not a multiple of norm_groups {right['norm_groups']}")
    for k in ("left_scale", "right_scale"):
        require(mx, k, float, where)


def _check_kv_from(mx, i, checked, where):
    src = mx.get("kv_from")
    if src is None:
        return
    src = require(mx, "kv_from", int, where)
    if not 0 <= src < i:
        raise ConfigError(f"{where}: 'kv_from' {src} must name an earlier layer")
    other = checked[src]
    om = other["mixer"]
    if other["type"] != "attention" or om.get("kv_from") is not None:
        raise ConfigError(f"{where}: 'kv_from' {src} must name an attention layer with keys and values of its own")
    if any(om[k] != mx[k] for k in ("kv_heads", "dim", "vdim")):
        raise ConfigError(f"{where}: layer {src}, whose keys and values this layer reads, has other key/value heads "
                          f"or head sizes")


def _check_mlp(mlp, where):
    kind = require(mlp, "kind", str, where)
    if kind != "moe":
        raise ConfigError(f"{where}: kind {kind!r} is not supported (moe)")
    _positive(_section(mlp, "expert", where), ("ff",), where + ".expert")
    r = _section(mlp, "router", where)
    _positive(r, ("experts", "top"), where + ".router")
    if r["top"] > r["experts"]:
        raise ConfigError(f"{where}.router: 'top' {r['top']} exceeds the {r['experts']} experts")
    if mlp.get("shared") is not None:
        _positive(_section(mlp, "shared", where), ("ff",), where + ".shared")


def _window(mx) -> int:
    return (mx.get("mask") or {}).get("size", 0)


@dataclass(frozen=True)
class PibavikConfig(ModelConfig):
    vocab: int
    width: int
    layers: tuple                  # of plain dicts as config.json gives them (validated)
    norm_eps: float
    embed_scale: float = 1.0
    architecture: str = "Pibavik"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "PibavikConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: required key 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{where} must be an object")
            typ = require(layer, "type", str, where)
            mx, mw = _section(layer, "mixer", where), where + ".mixer"
            if typ == "attention":
                _check_heads(mx, mw)
                _check_kv_from(mx, i, checked, mw)
            elif typ == "latent_attention":
                _positive(mx, ("heads", "dim", "vdim", "kv_rank", "q_rank"), mw)
                require(mx, "scale", float, mw)
            elif typ == "parallel":
                _check_parallel(mx, mw)
            else:
                raise ConfigError(f"{where}: mixer type {typ!r} is not supported (attention, latent_attention, parallel)")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise ConfigError(f"{where}.mlp must be an object or null")
                _check_mlp(mlp, where + ".mlp")
            checked.append(copy.deepcopy(dict(layer)))
        norm = _section(d, "norm", "config.json")
        emb = d.get("embedding") or {}
        if not isinstance(emb, Mapping):
            raise ConfigError("config.json: 'embedding' must be an object")
        cfg = cls(vocab=require(d, "vocab", int), width=require(d, "width", int), layers=tuple(checked),
                  norm_eps=require(norm, "eps", float, "config.json: norm"),
                  embed_scale=optional(emb, "scale", float, 1.0, "config.json: embedding"))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if not cfg.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cfg

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embed_scale}, "layers": copy.deepcopy(list(self.layers)),
                "norm": {"eps": self.norm_eps}}

    # ------------------------------------------------------------------ the model as data
    def _kept_window(self, i: int) -> int:
        """The window of keys that layer i's cache has to keep: its own, or a longer one (0: all keys) of a layer
        that reads them."""
        sizes = [_window(ly["mixer"]) for j, ly in enumerate(self.layers)
                 if j == i or (ly["type"] == "attention" and ly["mixer"].get("kv_from") == i)]
        return 0 if 0 in sizes else max(sizes)

    def _mixer(self, i: int, layer) -> PartSpec:
        p, d, eps, mx = f"l{i}.mix.", self.width, self.norm_eps, layer["mixer"]
        heads = lambda m: {"hidden_size": d, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                           "v_head_dim": m["vdim"], "scale": float(m["scale"]), "window": _window(m)}
        if layer["type"] == "attention":
            src = mx.get("kv_from")
            return PartSpec("attention", {
                **heads(mx), "slopes": tuple(2.0 ** (-SLOPE_SPAN * (h + 1) / mx["heads"]) for h in range(mx["heads"])),
                "own_kv": src is None, "cache_window": self._kept_window(i if src is None else src), "names": "short"}, p)
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": d, "num_heads": mx["heads"], "head_dim": mx["dim"], "rot_dim": 0, "v_head_dim": mx["vdim"],
                "kv_rank": mx["kv_rank"], "q_rank": mx["q_rank"], "eps": eps, "scale": float(mx["scale"])}, p)
        left, right = mx["left"], mx["right"]
        attention = PartSpec("gated_attention", {**heads(left), "qk_norm": "head", "eps": eps, "gate": "sigmoid",
                                                 "gate_per_head": True}, p + "left.")
        mamba = PartSpec("mamba2", {
            "hidden_size": d, "num_heads": right["heads"], "v_head_dim": right["vdim"], "state": right["state"],
            "groups": right["groups"], "conv": right["conv"], "norm_groups": right["norm_groups"], "eps": eps}, p + "right.")
        return PartSpec("parallel", {"left": attention, "right": mamba, "left_scale": float(mx["left_scale"]),
                                     "right_scale": float(mx["right_scale"])}, p)

    @staticmethod
    def _position(layer):
        rot = layer["mixer"]["left"].get("rot") if layer["type"] == "parallel" else None
        if rot is None:
            return None
        return PartSpec("rotary_scaled", {"dims": rot["dims"], "base": float(rot["base"]), "scaling": None, "layout": "half"})

    def _ffn(self, i: int, mlp):
        if mlp is None:
            return None
        r, shared = mlp["router"], mlp.get("shared")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "num_experts": r["experts"],
            "top_k": r["top"], "score": "sigmoid", "normalize": False, "activation": EXPERT_ACT, "weigh_input": True,
            "shared_size": shared["ff"] if shared else 0}, f"l{i}.mlp.")

    def model_spec(self) -> ModelSpec:
        d = self.width
        norm = lambda name: PartSpec("rms_norm", {"size": d, "eps": self.norm_eps, "tensor": name})
        layers, run = [], []
        for i, layer in enumerate(self.layers):
            ffn = self._ffn(i, layer.get("mlp"))
            norms = {"mixer": norm(f"l{i}.norm1")}
            if ffn is not None:
                norms["ffn"] = norm(f"l{i}.norm2")
            layers.append(LayerSpec(block="pre_norm", mixer=self._mixer(i, layer), ffn=ffn, norms=norms,
                                    position=self._position(layer)))
            run.append(RunEntry(i, cache_of=layer["mixer"].get("kv_from") if layer["type"] == "attention" else None))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=d,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": d, "tensor": "embed",
                                             "scale": self.embed_scale}),
            layers=tuple(layers), run_order=tuple(run), final_norm=norm("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": d, "tensor": "head"}),
            max_position=0)
