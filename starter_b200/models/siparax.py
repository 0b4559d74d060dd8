"""Siparax ("Siparax"): configuration, layer arrangement, tensor names.

A small decoder of pre-norm layers (layer norms with weight and bias, also on the embedded rows) over a 32-bit residual,
with an untied, capped output head.  Three kinds of mixer:

* "channel_delta": a gated delta rule with a decay per key channel, short convolutions on queries, keys and values, unit
  queries and keys, a per-head norm and a sigmoid gate of the output, decay and gate through two small matrices each;
* "latent_attention": attention through low-rank latents whose rotated part turns in neighbouring pairs;
* "latent_attention_2": the same with the rotated part turned in halves and one sigmoid gate per head; with ``kv_from``
  it has no key/value down-projection and reads the cached rows of the layer it names.

The feed-forward is dense, gated by the tanh form of gelu; a layer may have none.

config.json: ``vocab``, ``width``, ``norm`` {``eps``}, ``logit_softcap`` and ``layers``, a list of {``type``, ``mixer``
{...}, ``mlp`` {``kind`` "dense", ``ff``} or null}.  A "channel_delta" mixer has ``heads``, ``kv_heads``, ``dim``, ``vdim``
and ``conv``; the latent ones ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``, ``scale`` and ``rot``
{``base``, ``dims``, ``scaling`` {``factor``, ``original``, ``fast``, ``slow``} or nothing}.  Tensors: ``embed``, ``head``,
``embed.norm``, ``final.norm`` and per layer ``l<i>.norm1``, ``l<i>.norm2`` (a norm's bias has ``.b`` behind its name),
``l<i>.mix.*``, ``l<i>.mlp.{gate,up,down}``.

The inner sizes of a delta mixer's decay and gate matrices, which config.json does not give, are read from the shapes of
``l<i>.mix.a1`` and ``l<i>.mix.g1``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..config.registry import ConfigError, ModelConfig, TensorNames, register_architecture
from ..config.specs import (BlockSpec, ChannelDeltaSpec, GatedMLPSpec, LatentAttentionSpec, LayerNormSpec, ModelSpec, PairRopeSpec,
                            ScaledHalfRopeSpec)

LATENT_KEYS = ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot")
MIXER_KEYS = {
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "latent_attention": LATENT_KEYS,
    "latent_attention_2": LATENT_KEYS,
}
RANKS = (("decay_rank", "a1"), ("gate_rank", "g1"))    # sizes that only a tensor's shape gives


def _need(where: str, raw, keys) -> None:
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if k not in raw]
    if missing:
        raise ConfigError(f"config.json: {where} lacks " + ", ".join(missing))


def _count(where: str, value, least: int = 1) -> int:
    if isinstance(value, bool) or not isinstance(value, int) or value < least:
        raise ConfigError(f"config.json: {where} must be an integer of at least {least}, got {value!r}")
    return value


def _check_mixer(where: str, kind: str, m) -> None:
    _need(where, m, MIXER_KEYS[kind])
    for key in MIXER_KEYS[kind]:
        if key not in ("scale", "rot"):
            _count(f"{where}.{key}", m[key])
    if kind == "channel_delta":
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {where}: {m['heads']} heads cannot share {m['kv_heads']} kv_heads evenly")
        return
    _need(where + ".rot", m["rot"], ("base", "dims"))
    dims = _count(where + ".rot.dims", m["rot"]["dims"], 2)
    if dims % 2 or dims > m["rot_dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most rot_dim, got {dims}")
    if m["rot"].get("scaling") is not None:
        _need(where + ".rot.scaling", m["rot"]["scaling"], ("factor", "original", "fast", "slow"))


@dataclass(frozen=True)
class SiparaxConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[Any, ...]              # the layer entries as read (plain data)

    architecture = "Siparax"

    @classmethod
    def from_dict(cls, raw: dict) -> "SiparaxConfig":
        _need("the configuration", raw, ("vocab", "width", "norm", "layers"))
        _need("norm", raw["norm"], ("eps",))
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _need(where, entry, ("type", "mixer"))
            kind, m = entry["type"], entry["mixer"]
            if kind not in MIXER_KEYS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is unknown; known: " + ", ".join(sorted(MIXER_KEYS)))
            _check_mixer(where + ".mixer", kind, m)
            source = m.get("kv_from")
            if source is not None:
                if kind == "channel_delta" or isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < i:
                    raise ConfigError(f"config.json: {where}.mixer.kv_from must name an earlier layer, got {source!r}")
                other = layers[source]["mixer"]
                if layers[source]["type"] == "channel_delta" or other.get("kv_from") is not None or any(
                        other[key] != m[key] for key in ("kv_rank", "rot_dim")):
                    raise ConfigError(f"config.json: {where}.mixer.kv_from: layers[{source}] makes no latents of this kv_rank and rot_dim")
            mlp = entry.get("mlp")
            if mlp is not None:
                _need(where + ".mlp", mlp, ("kind", "ff"))
                if mlp["kind"] != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not built: 'dense' is")
                _count(where + ".mlp.ff", mlp["ff"])
            layers.append(copy.deepcopy(entry))
        cap = raw.get("logit_softcap")
        if cap is not None and not float(cap) > 0:
            raise ConfigError(f"config.json: logit_softcap must be positive, got {cap!r}")
        return cls(vocab=_count("vocab", raw["vocab"]), width=_count("width", raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                   logit_softcap=None if cap is None else float(cap), layers=tuple(layers))

    def with_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "SiparaxConfig":
        """The configuration with the two sizes that only tensors' shapes give: the inner sizes of a delta mixer's decay and
        gate matrices.  A mixer entry may also name them itself (``decay_rank``, ``gate_rank``; a configuration made for
        random weights has no shapes to read)."""
        layers = copy.deepcopy(list(self.layers))
        for i, entry in enumerate(layers):
            if entry["type"] == "channel_delta":
                for key, tensor in RANKS:
                    name = f"l{i}.mix.{tensor}"
                    if name in shapes and key not in entry["mixer"]:
                        entry["mixer"][key] = int(shapes[name][0])
        return SiparaxConfig(self.vocab, self.width, self.norm_eps, self.logit_softcap, tuple(layers))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps},
               "vocab": self.vocab, "width": self.width}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    # ---- layers -------------------------------------------------------------------------

    def _mixer_spec(self, i: int):
        m, kind = self.layers[i]["mixer"], self.layers[i]["type"]
        if kind == "channel_delta":
            ranks = {key: int(m.get(key) or 0) for key, _ in RANKS}
            if min(ranks.values()) <= 0:
                raise ConfigError(f"layers[{i}]: the inner sizes of the decay and gate matrices come from the shapes of l{i}.mix.a1 and "
                                  f"l{i}.mix.g1; give the configuration the checkpoint's shapes first (with_shapes)")
            return ChannelDeltaSpec(hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                    v_dim=m["vdim"], taps=m["conv"], norm_eps=self.norm_eps, **ranks)
        second = kind == "latent_attention_2"
        rot = m["rot"]
        sc = rot.get("scaling")
        stretch = {key: float(sc[key]) for key in ("factor", "original", "fast", "slow")} if sc is not None else {}
        position = (ScaledHalfRopeSpec if second else PairRopeSpec)(theta=float(rot["base"]), rotary_dim=int(rot["dims"]), **stretch)
        return LatentAttentionSpec(hidden_size=self.width, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"],
                                   q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=float(m["scale"]), norm_eps=self.norm_eps,
                                   position=position, head_gate=second, kv_from=m.get("kv_from"))

    def model_spec(self) -> ModelSpec:
        norm = LayerNormSpec(size=self.width, eps=self.norm_eps)
        blocks = []
        for i, entry in enumerate(self.layers):
            mlp = entry.get("mlp")
            ff = None
            if mlp is not None:
                ff = GatedMLPSpec(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="gelu_tanh")
            blocks.append(BlockSpec(mixer_norm=norm, mixer=self._mixer_spec(i), ff_norm=norm if ff is not None else None, ff=ff))
        return ModelSpec(hidden_size=self.width, vocab_size=self.vocab, layers=tuple(blocks), final_norm=norm, tie_embeddings=False,
                         logit_softcap=self.logit_softcap, residual_float32=True, embedding_norm=norm)

    def tensor_names(self) -> TensorNames:
        def norm(name):
            return {"weight": name, "bias": name + ".b"}

        layers = []
        for i, entry in enumerate(self.layers):
            p = f"l{i}."
            if entry["type"] == "channel_delta":
                mixer = {r: r for r in ("q", "k", "v", "b", "A_log", "dt_bias", "a1", "a2", "g1", "g2", "norm", "o")}
                mixer.update({"q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"})
            else:
                mixer = {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "uk": "uk", "uv": "uv", "o": "o"}
                if entry["mixer"].get("kv_from") is None:
                    mixer.update({"dkv": "dkv", "dkv_norm": "dkv.norm"})
                if entry["type"] == "latent_attention_2":
                    mixer["g"] = "g"
            names = {"mixer_norm": norm(p + "norm1"), "mixer": {role: p + "mix." + n for role, n in mixer.items()}}
            if entry.get("mlp") is not None:
                names["ff_norm"] = norm(p + "norm2")
                names["ff"] = {r: p + "mlp." + r for r in ("gate", "up", "down")}
            layers.append(names)
        return TensorNames(embedding="embed", lm_head="head", final_norm=norm("final.norm"), layers=layers,
                           embedding_norm=norm("embed.norm"))

    def random_init(self, name: str, shape) -> Tuple[float, float]:
        """(mean, standard deviation) of a tensor's seeded random fill: matrices so that a product keeps its input's size,
        norm weights around one and biases around zero, decays from nearly none to strong."""
        last = name.rsplit(".", 1)[-1]
        if name.endswith((".norm1.b", ".norm2.b", "embed.norm.b", "final.norm.b")):
            return 0.0, 0.1
        if last == "conv":
            return 0.2, 0.5
        if last == "A_log":
            return 0.0, 0.7
        if last == "dt_bias":
            return -2.0, 1.5
        if len(shape) == 1:
            return 1.0, 0.1
        if name == "embed":
            return 0.0, 1.0
        return 0.0, float(shape[-1]) ** -0.5


register_architecture(SiparaxConfig.architecture, SiparaxConfig)
