"""Typed configuration of the Bubalix decoder (config.json ``"architecture": "Bubalix"``).

A stack of layers around a 32-bit residual stream whose two sublayers read one norm, ``h = norm1(x)``, ``x += mixer(h) + ff(h)``, with an
input of the token's own behind them, ``x += rms_norm(W_proj (gelu_tanh(W_gate x) * e)) * weight`` (``e``: the layer's part of a row of a
table that the layers share).  Every norm is an RMS norm; those of the stream store the gain's distance from one.  The embedding
output is multiplied by ``embedding.scale``; the head has a matrix of its own.  config.json lists the layers (``layers[i]``: ``type``,
``mixer``, ``mlp``), and every layer may differ:

* ``type: "latent_attention"``: attention over every earlier key through one latent a token (``kv_rank``) beside a rotated key part
  that the heads share (``rot_dim``): ``heads`` of ``dim`` unrotated and ``rot_dim`` rotated query/key elements and ``vdim`` values, ``scale``,
  rotation of the pairs ``(i, i + rot.dims / 2)`` (``rot.base``; ``rot.scaling`` with ``factor``, ``original``, ``fast``, ``slow``: YaRN), a sink a
  head, a sigmoid gate on the concatenated heads.
* ``type: "attention"``: grouped-query attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``) behind convolutions of ``conv`` taps on q,
  k and v, without rotation: scores capped at ``softcap`` (absent or 0: no cap), less a slope a head times the distance; queries
  warmed by ``q_temp`` (``coef``, ``every``; absent: none); a window of ``mask.size`` positions (no mask: every earlier key); a sink and
  one sigmoid gate a head.
* ``mlp``: null, or ``{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}, "shared": {"ff"} or null}``: a table gives each token id
  its ``top`` experts, ``down(silu(gate h) * up h)``, each with the weight ``1 / top``; the shared expert's result is added.

``token_side.dim``: the width of a layer's share of the table ``side.embed`` (absent: no such input).

Tensor names: ``embed``, ``side.embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.{gate,proj,norm}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .model_config import ArchitectureConfig, ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

MAX_POSITION = 1 << 20      # the design sets no limit of its own; the engine's max_model_len is the one that counts


def _int(d, key, where, least=1):
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, int) or isinstance(v, bool) or v < least:
        raise ConfigError(f"Bubalix config.json: {where}.{key} must be an integer of at least {least}, found {v!r}")
    return v


def _num(d, key, where, positive=False):
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, (int, float)) or isinstance(v, bool) or (positive and not v > 0):
        raise ConfigError(f"Bubalix config.json: {where}.{key} must be a{' positive' if positive else ''} number, found {v!r}")
    return float(v)


def _check_mixer(kind, m, where):
    if not isinstance(m, dict):
        raise ConfigError(f"Bubalix config.json: {where} must be an object")
    if kind not in ("latent_attention", "attention"):
        raise ConfigError(f"Bubalix config.json: {where[:-6]}.type {kind!r} is not a known layer type (latent_attention, attention)")
    heads = _int(m, "heads", where)
    for k in ("dim", "vdim"):
        _int(m, k, where)
    _num(m, "scale", where, positive=True)
    if kind == "latent_attention":
        _int(m, "kv_rank", where)
        rot_dim = _int(m, "rot_dim", where, least=0)
        rot = m.get("rot")
        if rot is not None and rot.get("dims"):
            dims = _int(rot, "dims", where + ".rot", least=2)
            if dims % 2 or dims > rot_dim:
                raise ConfigError(f"Bubalix config.json: {where}.rot.dims {dims} must be even and at most rot_dim ({rot_dim})")
            _num(rot, "base", where + ".rot", positive=True)
            if rot.get("scaling") is not None:
                for k in ("factor", "original", "fast", "slow"):
                    _num(rot["scaling"], k, where + ".rot.scaling", positive=True)
        return
    groups = _int(m, "kv_heads", where)
    if heads % groups:
        raise ConfigError(f"Bubalix config.json: {where}: {heads} heads do not group over {groups} key/value heads")
    if _int(m, "conv", where) > 16:
        raise ConfigError(f"Bubalix config.json: {where}.conv: at most 16 taps are served, found {m['conv']}")
    if m.get("softcap") is not None and _num(m, "softcap", where) < 0.0:
        raise ConfigError(f"Bubalix config.json: {where}.softcap {m['softcap']} must not be negative")
    if m.get("q_temp") is not None:
        _num(m["q_temp"], "coef", where + ".q_temp")
        _num(m["q_temp"], "every", where + ".q_temp", positive=True)
    if m.get("mask") is not None:
        _int(m["mask"], "size", where + ".mask")


def _check_mlp(mlp, where):
    if mlp is None:
        return
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind != "moe":
        raise ConfigError(f"Bubalix config.json: {where}.kind {kind!r} is not implemented (moe)")
    experts, top = _int(mlp.get("router"), "experts", where + ".router"), _int(mlp.get("router"), "top", where + ".router")
    if top > experts:
        raise ConfigError(f"Bubalix config.json: {where}.router.top {top} exceeds the {experts} experts")
    _int(mlp.get("expert"), "ff", where + ".expert")
    if mlp.get("shared") is not None:
        _int(mlp["shared"], "ff", where + ".shared")


@register_architecture("Bubalix", model_type="bubalix")
@dataclass
class BubalixConfig(ArchitectureConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    side_dim: int
    layers: List[Dict[str, Any]]
    extra: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_json(cls, data: Dict[str, Any]) -> "BubalixConfig":
        vocab, width = _int(data, "vocab", "config"), _int(data, "width", "config")
        eps = _num(data.get("norm"), "eps", "norm", positive=True)
        scale = _num(data.get("embedding"), "scale", "embedding") if (data.get("embedding") or {}).get("scale") is not None else 1.0
        side = _int(data.get("token_side"), "dim", "token_side") if data.get("token_side") is not None else 0
        layers: Optional[List] = copy.deepcopy(data.get("layers"))
        if not isinstance(layers, list) or not layers:
            raise ConfigError("Bubalix config.json: 'layers' must list at least one layer")
        for i, layer in enumerate(layers):
            _check_mixer(layer.get("type"), layer.get("mixer"), f"layers[{i}].mixer")
            _check_mlp(layer.get("mlp"), f"layers[{i}].mlp")
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "embedding", "token_side", "layers"}
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=scale, side_dim=side, layers=layers,
                   extra={k: v for k, v in data.items() if k not in known})

    def to_json(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "token_side": {"dim": self.side_dim} if self.side_dim else None,
             "layers": copy.deepcopy(self.layers)}
        for k, v in self.extra.items():
            d.setdefault(k, v)
        return d

    # ---- parts -------------------------------------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("group_rms_norm", {"size": self.width, "eps": self.norm_eps, "weight": name, "weight_offset": 1.0})

    def _mixer(self, layer: Dict[str, Any]) -> PartSpec:
        m = layer["mixer"]
        if layer["type"] == "latent_attention":
            rot, position = m.get("rot"), None
            if rot is not None and rot.get("dims"):
                position = {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"])}
                if rot.get("scaling") is not None:
                    position["yarn_scaling"] = {k: float(rot["scaling"][k]) for k in ("factor", "original", "fast", "slow")}
                position = PartSpec("rotary_half", position)
            return PartSpec("latent_attention", {
                "hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"], "q_rank": None,
                "kv_rank": m["kv_rank"], "eps": self.norm_eps, "scale": float(m["scale"]), "position": position, "gate": True, "learned_sink": True,
                "prefix": "mix."})
        t, mask = m.get("q_temp"), m.get("mask")
        return PartSpec("conv_window_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "taps": m["conv"],
            "scale": float(m["scale"]), "window": int(mask["size"]) if mask is not None else None, "softcap": float(m.get("softcap") or 0.0),
            "distance_bias": True, "learned_sink": True, "query_temperature": (float(t["coef"]), float(t["every"])) if t is not None else None,
            "head_gate": True, "prefix": "mix."})

    def _feed_forward(self, mlp: Dict[str, Any]) -> PartSpec:
        return PartSpec("expert_mixture", {
            "hidden_size": self.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "ff": mlp["expert"]["ff"], "activation": "silu",
            "scoring": "table", "vocab_size": self.vocab, "shared_ff": mlp["shared"]["ff"] if mlp.get("shared") is not None else 0, "shared_gate": False,
            "prefix": "mlp."})

    def to_spec(self) -> ModelSpec:
        layers = []
        for i, layer in enumerate(self.layers):
            more = {}
            if self.side_dim:
                more["side"] = PartSpec("token_input", {"hidden_size": self.width, "vocab_size": self.vocab, "dim": self.side_dim, "slices": len(self.layers),
                                                        "index": i, "table": "side.embed", "prefix": "side."})
            layers.append(LayerSpec(
                block="parallel_sublayers", mixer_norm=self._norm("norm1"), mixer=self._mixer(layer),
                feed_forward=self._feed_forward(layer["mlp"]) if layer.get("mlp") is not None else None, weight_prefix=f"l{i}.", more=more))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "weight": "embed", "scale": self.embedding_scale}),
            layers=layers, run_order=[RunEntry(i) for i in range(len(self.layers))], final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False, "weight": "head", "tied_to": "embed"}),
            max_position=MAX_POSITION)
        spec.validate()
        return spec
