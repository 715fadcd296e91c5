"""Typed configuration of the Zonevik decoder (config.json ``"architecture": "Zonevik"``).

A stack of layers around a 32-bit residual stream with a norm on both sides of every sublayer, ``x += norm1b(mixer(norm1(x)))``
then ``x += norm2b(ff(norm2(x)))``.  Every norm is a dynamic tanh, ``tanh(alpha x) * w + b``, without statistics.  The embedding
output is multiplied by ``embedding.scale``; the logits are the final norm's output times the embedding table itself.
config.json lists the layers (``layers[i]``: ``type``, ``mixer``, ``mlp``), and every layer may differ:

* ``type: "attention"``: grouped-query softmax attention over every earlier key (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``),
  rotation of the neighbouring pairs of each head's first ``rot.dims`` elements (``rot.base``; ``rot.scaling`` with ``factor``, ``original``,
  ``fast``, ``slow``: YaRN), and a sigmoid gate on the concatenated heads.
* ``type: "delta"``: the gated delta rule (``heads`` of ``vdim`` over ``kv_heads`` of ``dim``; ``conv`` taps of the convolutions ahead of it).
* ``type: "parallel"``: two mixers on the same input, half the sum of their outputs, each first RMS-normed over the width.  ``left`` is
  attention with biases on q, k and v, without rotation, over a window of ``mask.size`` positions that keeps a sequence's first
  ``mask.keep_first`` tokens in view (no mask: every earlier key); ``right`` the state-space dual scan (``heads`` of ``vdim`` with ``state``
  states, ``groups`` of B and C, ``conv`` taps, an output norm in ``norm_groups`` parts).
* ``mlp``: null, or ``{"kind": "moe", "router": {"experts", "top", "groups": {"count", "keep"}}, "expert": {"ff"}}``: experts
  ``down(silu(gate h) * up h)``, chosen by the sigmoid of the router's logits among the groups whose two best scores have the
  largest sums, weighted by those scores as they are.

``loop: {start, stop, times}``: the layers ``start .. stop - 1`` run ``times`` times in a row with the same weights and a cache or
state of its own for every pass; ahead of every pass the stream becomes ``loop.in [x; x0]`` with the embedding output ``x0``.

Tensor names: ``embed``, ``loop.in``, ``l<i>.{norm1,norm1b,norm2,norm2b}`` (each with ``.b`` and ``.alpha``), ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .model_config import ArchitectureConfig, ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry, StreamProject

MAX_POSITION = 1 << 20      # the design sets no limit of its own; the engine's max_model_len is the one that counts


def _int(d, key, where, least=1):
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, int) or isinstance(v, bool) or v < least:
        raise ConfigError(f"Zonevik config.json: {where}.{key} must be an integer of at least {least}, found {v!r}")
    return v


def _num(d, key, where, positive=False):
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, (int, float)) or isinstance(v, bool) or (positive and not v > 0):
        raise ConfigError(f"Zonevik config.json: {where}.{key} must be a{' positive' if positive else ''} number, found {v!r}")
    return float(v)


def _check_attention(m, where):
    if not isinstance(m, dict):
        raise ConfigError(f"Zonevik config.json: {where} must be an object")
    heads, groups = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % groups:
        raise ConfigError(f"Zonevik config.json: {where}: {heads} heads do not group over {groups} key/value heads")
    dim = _int(m, "dim", where)
    _int(m, "vdim", where)
    if m.get("scale") is None:
        m["scale"] = float(dim) ** -0.5
    _num(m, "scale", where, positive=True)
    rot = m.get("rot")
    if rot is not None and rot.get("dims"):
        dims = _int(rot, "dims", where + ".rot", least=2)
        if dims % 2 or dims > dim:
            raise ConfigError(f"Zonevik config.json: {where}.rot.dims {dims} must be even and at most dim ({dim})")
        _num(rot, "base", where + ".rot", positive=True)
        if rot.get("scaling") is not None:
            for k in ("factor", "original", "fast", "slow"):
                _num(rot["scaling"], k, where + ".rot.scaling", positive=True)
    mask = m.get("mask")
    if mask is not None:
        _int(mask, "size", where + ".mask")
        if mask.get("keep_first") is not None:
            _int(mask, "keep_first", where + ".mask", least=0)


def _check_mixer(kind, m, where):
    if not isinstance(m, dict):
        raise ConfigError(f"Zonevik config.json: {where} must be an object")
    if kind == "attention":
        _check_attention(m, where)
    elif kind == "delta":
        heads, groups = _int(m, "heads", where), _int(m, "kv_heads", where)
        if heads % groups:
            raise ConfigError(f"Zonevik config.json: {where}: {heads} heads do not group over {groups} key heads")
        for k in ("dim", "vdim", "conv"):
            _int(m, k, where)
    elif kind == "parallel":
        _check_attention(m.get("left"), where + ".left")
        r = m.get("right")
        for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            _int(r, k, where + ".right")
        if r["heads"] % r["groups"] or (r["heads"] * r["vdim"]) % r["norm_groups"]:
            raise ConfigError(f"Zonevik config.json: {where}.right: the groups do not divide the heads, or norm_groups the inner size")
    else:
        raise ConfigError(f"Zonevik config.json: {where[:-6]}.type {kind!r} is not a known layer type (attention, delta, parallel)")


def _check_mlp(mlp, where):
    if mlp is None:
        return
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind != "moe":
        raise ConfigError(f"Zonevik config.json: {where}.kind {kind!r} is not implemented (moe)")
    r = mlp.get("router")
    experts, top = _int(r, "experts", where + ".router"), _int(r, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"Zonevik config.json: {where}.router.top {top} exceeds the {experts} experts")
    g = r.get("groups")
    if g is not None:
        count, keep = _int(g, "count", where + ".router.groups"), _int(g, "keep", where + ".router.groups")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"Zonevik config.json: {where}.router.groups: {count} groups, {keep} kept do not fit {experts} experts, top {top}")
    _int(mlp.get("expert"), "ff", where + ".expert")


@register_architecture("Zonevik", model_type="zonevik")
@dataclass
class ZonevikConfig(ArchitectureConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: List[Dict[str, Any]]
    loop: Optional[Dict[str, int]] = None
    extra: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_json(cls, data: Dict[str, Any]) -> "ZonevikConfig":
        vocab, width = _int(data, "vocab", "config"), _int(data, "width", "config")
        eps = _num(data.get("norm"), "eps", "norm", positive=True)
        scale = _num(data.get("embedding"), "scale", "embedding") if (data.get("embedding") or {}).get("scale") is not None else 1.0
        layers = copy.deepcopy(data.get("layers"))
        if not isinstance(layers, list) or not layers:
            raise ConfigError("Zonevik config.json: 'layers' must list at least one layer")
        for i, layer in enumerate(layers):
            _check_mixer(layer.get("type"), layer.get("mixer"), f"layers[{i}].mixer")
            _check_mlp(layer.get("mlp"), f"layers[{i}].mlp")
        loop = copy.deepcopy(data.get("loop"))
        if loop is not None:
            start, stop = _int(loop, "start", "loop", least=0), _int(loop, "stop", "loop")
            _int(loop, "times", "loop")
            if not start < stop <= len(layers):
                raise ConfigError(f"Zonevik config.json: loop {start} .. {stop} does not lie within the {len(layers)} layers")
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "embedding", "layers", "loop"}
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=scale, layers=layers, loop=loop,
                   extra={k: v for k, v in data.items() if k not in known})

    def to_json(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(self.layers), "loop": copy.deepcopy(self.loop)}
        for k, v in self.extra.items():
            d.setdefault(k, v)
        return d

    # ---- parts -------------------------------------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", {"size": self.width, "weight": name})

    def _attention(self, m: Dict[str, Any], **more) -> PartSpec:
        rot, position, mask = m.get("rot"), None, m.get("mask")
        if rot is not None and rot.get("dims"):
            position = {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"])}
            if rot.get("scaling") is not None:
                position["yarn_scaling"] = {k: float(rot["scaling"][k]) for k in ("factor", "original", "fast", "slow")}
            position = PartSpec("rotary_interleaved", position)
        return PartSpec("gated_window_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": float(m["scale"]),
            "window": int(mask["size"]) if mask is not None else None, "keep_first": int(mask.get("keep_first") or 0) if mask is not None else 0,
            "position": position, **more})

    def _mixer(self, layer: Dict[str, Any]) -> PartSpec:
        W, m, kind, eps = self.width, layer["mixer"], layer["type"], self.norm_eps
        if kind == "attention":
            return self._attention(m, gate=True, prefix="mix.")
        if kind == "delta":
            return PartSpec("gated_delta_rule", {"hidden_size": W, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                                                 "taps": m["conv"], "eps": eps, "prefix": "mix."})
        r = m["right"]
        right = PartSpec("state_space_dual", {"hidden_size": W, "heads": r["heads"], "vdim": r["vdim"], "state": r["state"], "groups": r["groups"],
                                              "taps": r["conv"], "norm_groups": r["norm_groups"], "eps": eps})
        return PartSpec("parallel_mixers", {"left": self._attention(m["left"], bias=True), "right": right, "left_scale": 0.5, "right_scale": 0.5,
                                            "out_norm": {"hidden_size": W, "eps": eps}, "prefix": "mix."})

    def _feed_forward(self, mlp: Dict[str, Any]) -> PartSpec:
        r = mlp["router"]
        g = r.get("groups")
        return PartSpec("expert_mixture", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "ff": mlp["expert"]["ff"], "activation": "silu", "scoring": "sigmoid",
            "groups": (int(g["count"]), int(g["keep"])) if g is not None else None, "group_score": "best_two", "prefix": "mlp."})

    def run_order(self) -> List[RunEntry]:
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [RunEntry(i) for i in range(n)]
        one_pass = [RunEntry(i, before=StreamProject("loop.in") if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
        return [RunEntry(i) for i in range(loop["start"])] + one_pass * loop["times"] + [RunEntry(i) for i in range(loop["stop"], n)]

    def to_spec(self) -> ModelSpec:
        layers, ignorable = [], []
        for i, layer in enumerate(self.layers):
            mlp = layer.get("mlp")
            more = {"mixer_out_norm": self._norm("norm1b")}
            if mlp is not None:
                more["ffn_out_norm"] = self._norm("norm2b")
            else:
                ignorable += [f"l{i}.{n}{s}" for n in ("norm2", "norm2b") for s in ("", ".b", ".alpha")]
            layers.append(LayerSpec(
                block="sandwich_norm", mixer_norm=self._norm("norm1"), mixer=self._mixer(layer),
                ffn_norm=self._norm("norm2") if mlp is not None else None, feed_forward=self._feed_forward(mlp) if mlp is not None else None,
                weight_prefix=f"l{i}.", more=more))
        if self.loop is None:
            ignorable.append("loop.in")
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "weight": "embed", "scale": self.embedding_scale}),
            layers=layers, run_order=self.run_order(), final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": True, "weight": "head", "tied_to": "embed"}),
            max_position=MAX_POSITION, ignorable=ignorable)
        spec.validate()
        return spec
