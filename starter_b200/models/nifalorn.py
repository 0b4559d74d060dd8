"""Nifalorn ("Nifalorn"): configuration, layer arrangement, tensor names.

A small decoder of pre-norm layers (RMS norms with weights stored around zero) over a 32-bit residual, with a scaled
embedding and scaled logits of an untied head.  A run of its layers may repeat with the same weights (``loop``), each pass
with a cache of its own and nothing in between.  Three kinds of mixer:

* "lightning": linear attention with a matrix state per head that decays by a constant, silu on queries, keys and values,
  one norm over all heads and a sigmoid gate;
* "mamba2": a Mamba-2 layer, i.e. a matrix state per head whose decay and step size depend on the token, groups of heads
  that share B and C, a short convolution with a bias, a skip, and a silu gate in front of a norm in equal parts;
* "attention": grouped-query attention with two score maps per head over the same values, partly rotated in neighbouring
  pairs (frequencies stretched by wavelength), over the query's own chunk of positions.

The feed-forward is dense (up, squared relu, down) or a mixture of experts: sigmoid scores, a correction for the choice,
experts in groups of which the best are kept, a shared expert with a gate per token.

config.json: ``vocab``, ``width``, ``norm`` {``eps``}, ``embedding`` {``scale``}, ``logit_scale``, ``loop`` {``start``,
``stop``, ``times``} or nothing, and ``layers``, a list of {``type``, ``mixer`` {...}, ``mlp`` {...} or null}.  A "lightning"
mixer has ``heads``, ``dim``, ``vdim``, ``decay`` (a number per head); a "mamba2" one ``heads``, ``vdim``, ``state``,
``groups``, ``conv``, ``norm_groups``; an "attention" one ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``diff``,
``mask`` {``size``} or nothing, ``rot`` {``base``, ``dims``, ``scaling`` {``factor``, ``low``, ``high``, ``original``} or
nothing} or nothing.  ``mlp``: ``kind`` "dense" with ``ff``, or "moe" with ``router`` {``experts``, ``top``, ``scale``,
``groups`` {``count``, ``keep``}}, ``expert`` {``ff``}, ``shared`` {``ff``} or nothing.  Tensors: ``embed``, ``head``,
``final.norm`` and per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.

The constant the design fixes is the 1 that the norms' weights are stored around.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Optional, Tuple

from ..config.registry import ConfigError, ModelConfig, TensorNames, register_architecture
from ..config.specs import (ActMLPSpec, BlockSpec, DiffAttentionSpec, GatedMLPSpec, GroupedNormSpec, LightningSpec, Mamba2Spec,
                            ModelSpec, MoESpec, PairRopeSpec)

NORM_OFFSET = 1.0          # a norm multiplies by 1 + w
MIXER_KEYS = {
    "lightning": ("heads", "dim", "vdim", "decay"),
    "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "diff"),
}
NUMBERS = ("decay", "scale", "diff")      # the other keys are counts


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
        if key not in NUMBERS:
            _count(f"{where}.{key}", m[key])
    if kind == "lightning":
        decay = m["decay"]
        if not isinstance(decay, list) or len(decay) != m["heads"] or not all(0.0 <= float(d) <= 1.0 for d in decay):
            raise ConfigError(f"config.json: {where}.decay must list one number from 0 to 1 per head, got {decay!r}")
    elif kind == "mamba2":
        if m["heads"] % m["groups"]:
            raise ConfigError(f"config.json: {where}: {m['heads']} heads cannot share {m['groups']} groups evenly")
        if (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ConfigError(f"config.json: {where}: {m['heads'] * m['vdim']} columns cannot be normed in {m['norm_groups']} equal parts")
    else:
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {where}: {m['heads']} heads cannot share {m['kv_heads']} kv_heads evenly")
        if m.get("mask") is not None:
            _need(where + ".mask", m["mask"], ("size",))
            _count(where + ".mask.size", m["mask"]["size"])
        if m.get("rot") is not None:
            _need(where + ".rot", m["rot"], ("base", "dims"))
            dims = _count(where + ".rot.dims", m["rot"]["dims"], 2)
            if dims % 2 or dims > m["dim"]:
                raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim, got {dims}")
            if m["rot"].get("scaling") is not None:
                _need(where + ".rot.scaling", m["rot"]["scaling"], ("factor", "low", "high", "original"))


def _check_mlp(where: str, mlp) -> None:
    _need(where, mlp, ("kind",))
    if mlp["kind"] == "dense":
        _need(where, mlp, ("ff",))
        _count(where + ".ff", mlp["ff"])
        return
    if mlp["kind"] != "moe":
        raise ConfigError(f"config.json: {where}.kind {mlp['kind']!r} is not built: 'dense' and 'moe' are")
    _need(where, mlp, ("router", "expert"))
    r = mlp["router"]
    _need(where + ".router", r, ("experts", "top"))
    experts, top = _count(where + ".router.experts", r["experts"]), _count(where + ".router.top", r["top"])
    count = keep = 1
    if r.get("groups") is not None:
        _need(where + ".router.groups", r["groups"], ("count", "keep"))
        count, keep = _count(where + ".router.groups.count", r["groups"]["count"]), _count(where + ".router.groups.keep", r["groups"]["keep"])
    if experts % count or keep > count:
        raise ConfigError(f"config.json: {where}.router: {experts} experts cannot form {count} equal groups of which {keep} are kept")
    if top > keep * (experts // count):
        raise ConfigError(f"config.json: {where}.router chooses {top} of {keep * (experts // count)}")
    for part in ("expert", "shared"):
        if mlp.get(part) is not None:
            _need(f"{where}.{part}", mlp[part], ("ff",))
            _count(f"{where}.{part}.ff", mlp[part]["ff"])


@dataclass(frozen=True)
class NifalornConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    loop: Optional[Tuple[int, int, int]]     # (start, stop, times) or None
    layers: Tuple[Any, ...]                  # the layer entries as read (plain data)

    architecture = "Nifalorn"

    @classmethod
    def from_dict(cls, raw: dict) -> "NifalornConfig":
        _need("the configuration", raw, ("vocab", "width", "norm", "layers"))
        _need("norm", raw["norm"], ("eps",))
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _need(where, entry, ("type", "mixer"))
            if entry["type"] not in MIXER_KEYS:
                raise ConfigError(f"config.json: {where}.type {entry['type']!r} is unknown; known: " + ", ".join(sorted(MIXER_KEYS)))
            _check_mixer(where + ".mixer", entry["type"], entry["mixer"])
            if entry.get("mlp") is not None:
                _check_mlp(where + ".mlp", entry["mlp"])
            layers.append(copy.deepcopy(entry))
        loop = None
        if raw.get("loop") is not None:
            _need("loop", raw["loop"], ("start", "stop", "times"))
            lp = raw["loop"]
            start, stop, times = _count("loop.start", lp["start"], 0), _count("loop.stop", lp["stop"]), _count("loop.times", lp["times"])
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {start} .. {stop} - 1 of {len(layers)}")
            loop = (start, stop, times)
        return cls(vocab=_count("vocab", raw["vocab"]), width=_count("width", raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                   embedding_scale=float((raw.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(raw.get("logit_scale", 1.0)),
                   loop=loop, layers=tuple(layers))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
               "layers": copy.deepcopy(list(self.layers)), "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps},
               "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    # ---- layers -------------------------------------------------------------------------

    def _mixer_spec(self, i: int):
        m, kind = self.layers[i]["mixer"], self.layers[i]["type"]
        if kind == "lightning":
            return LightningSpec(hidden_size=self.width, num_heads=m["heads"], head_dim=m["dim"], v_dim=m["vdim"],
                                 decay=tuple(float(d) for d in m["decay"]), norm_eps=self.norm_eps)
        if kind == "mamba2":
            return Mamba2Spec(hidden_size=self.width, num_heads=m["heads"], v_dim=m["vdim"], state=m["state"], groups=m["groups"],
                              taps=m["conv"], norm_groups=m["norm_groups"], norm_eps=self.norm_eps)
        position = None
        rot = m.get("rot")
        if rot is not None:
            sc = rot.get("scaling")
            stretch = {key: float(sc[key]) for key in ("factor", "low", "high", "original")} if sc is not None else {}
            position = PairRopeSpec(theta=float(rot["base"]), rotary_dim=int(rot["dims"]), **stretch)
        mask = m.get("mask")
        return DiffAttentionSpec(hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                 v_dim=m["vdim"], scale=float(m["scale"]), diff=float(m["diff"]), norm_eps=self.norm_eps,
                                 chunk=int(mask["size"]) if mask is not None else None, position=position)

    def _ff_spec(self, i: int):
        mlp = self.layers[i].get("mlp")
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return ActMLPSpec(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="relu2")

        def gated(part):
            return GatedMLPSpec(hidden_size=self.width, intermediate_size=int(part["ff"]), activation="silu")

        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        return MoESpec(hidden_size=self.width, n_experts=int(r["experts"]), n_identity=0, top=int(r["top"]),
                       route_scale=float(r.get("scale", 1.0)), expert=gated(mlp["expert"]),
                       shared=gated(shared) if shared is not None else None, scores="sigmoid", groups=int(groups["count"]),
                       keep_groups=int(groups["keep"]), shared_gate=shared is not None)

    def model_spec(self) -> ModelSpec:
        norm = GroupedNormSpec(size=self.width, eps=self.norm_eps, groups=1, offset=NORM_OFFSET)
        blocks = []
        for i in range(len(self.layers)):
            ff = self._ff_spec(i)
            blocks.append(BlockSpec(mixer_norm=norm, mixer=self._mixer_spec(i), ff_norm=norm if ff is not None else None, ff=ff))
        schedule = ()
        if self.loop is not None:      # nothing happens between passes: an order of layers says it all
            start, stop, times = self.loop
            schedule = tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, len(blocks)))
        return ModelSpec(hidden_size=self.width, vocab_size=self.vocab, layers=tuple(blocks), final_norm=norm, tie_embeddings=False,
                         schedule=schedule, embedding_scale=self.embedding_scale, logit_scale=self.logit_scale, residual_float32=True)

    def tensor_names(self) -> TensorNames:
        layers = []
        for i, entry in enumerate(self.layers):
            p = f"l{i}."
            if entry["type"] == "lightning":
                mixer = {r: r for r in ("q", "k", "v", "g", "o", "norm")}
            elif entry["type"] == "mamba2":
                mixer = {r: r for r in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
                mixer["conv_bias"] = "conv.b"
            else:
                mixer = {r: r for r in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")}
            names = {"mixer_norm": {"weight": p + "norm1"}, "mixer": {role: p + "mix." + n for role, n in mixer.items()}}
            mlp = entry.get("mlp")
            if mlp is not None:
                names["ff_norm"] = {"weight": p + "norm2"}
                if mlp["kind"] == "dense":
                    ff = {"up": "up", "down": "down"}
                else:
                    ff = {"router": "router", "correction": "correction"}
                    for e in range(int(mlp["router"]["experts"])):
                        ff.update({f"e{e}_{r}": f"e{e}.{r}" for r in ("gate", "up", "down")})
                    if mlp.get("shared") is not None:
                        ff.update({"shared_" + r: "shared." + r for r in ("gate", "up", "down", "sg")})
                names["ff"] = {role: p + "mlp." + n for role, n in ff.items()}
            layers.append(names)
        return TensorNames(embedding="embed", lm_head="head", final_norm={"weight": "final.norm"}, layers=layers)

    def random_init(self, name: str, shape) -> Tuple[float, float]:
        """(mean, standard deviation) of a tensor's seeded random fill: matrices so that a product keeps its input's size,
        norm weights around zero (a mixer's own around one), decays from nearly none to strong, a router that spreads."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or name == "final.norm":
            return 0.0, 0.1
        if last in ("lq1", "lk1", "lq2", "lk2"):
            return 0.0, 0.15
        if last == "conv":
            return 0.2, 0.5
        if name.endswith("conv.b"):
            return 0.0, 0.3
        if last == "A_log":
            return 0.0, 0.7
        if last == "dt_bias":
            return -1.5, 1.0
        if last == "correction":
            return 0.0, 0.05
        if last == "router":
            return 0.0, 2.0 * float(shape[-1]) ** -0.5
        if last in ("norm", "D"):
            return 1.0, 0.2
        if name == "embed":
            return 0.0, 1.0
        return 0.0, float(shape[-1]) ** -0.5


register_architecture(NifalornConfig.architecture, NifalornConfig)
