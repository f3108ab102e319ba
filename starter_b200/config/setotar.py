"""Configuration of the Setotar decoder, read from the keys of its own ``config.json``.

The design: several residual streams a token, read and written through hyper-connections, each sublayer's output
scaled per channel in front of the write; pre-norm sublayers (RMS norms with plain gains); per layer one of two
mixers (``attention``: grouped-query attention over all keys, queries and keys normed over their whole projections and
turned by rotary positions; a layer with ``kv_from: j`` attends over layer ``j``'s keys and values; ``parallel``:
window attention that keeps the first tokens, with biases, short convolutions, unit-RMS values and capped scores,
side by side with a linear recurrence in which one gate a channel sets what is kept and what is written, joined as a
scaled sum) and a mixture of gated experts, each run on the row times its plain sigmoid, or no feed-forward.  A
final norm over the sum of the streams and an output head.

``config.json`` gives ``architecture``, ``vocab``, ``width``, ``streams``, ``norm.eps`` and a list ``layers``; a layer
has ``type``, ``mixer`` and ``mlp``:

* ``attention``: ``mixer = {heads, kv_heads, dim, vdim, scale, rot?, kv_from?}``.
* ``parallel``: ``mixer = {left{heads, kv_heads, dim, vdim, scale, conv?, rot?, mask{size, keep_first?}?, softcap?},
  right{heads, dim, vdim}, left_scale, right_scale}``.
* ``rot = {base, dims, scaling?}``; ``scaling = {factor}`` divides every frequency, ``{factor, original, fast, slow}``
  stretches them by parts (YaRN).
* ``mlp``: null or ``{kind: "moe", expert{ff}, router{experts, top}}``.

Every size and constant is read from there; a key this design does not know is an error.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass

from .kesedra import _lacking, _number, _positive, _unknown
from .qwen3 import ConfigError
from .spec import (
    ForgetWriteSpec,
    HyperConnectionSpec,
    LinearRopeScaling,
    ModelSpec,
    NormSpec,
    ParallelMixerSpec,
    PartialRopeSpec,
    RoutedExpertsSpec,
    ScheduleEntry,
    SinkAttentionSpec,
    YarnRopeScaling,
    hyper_layer,
)

_TOP = {"architecture", "architectures", "layers", "norm", "streams", "vocab", "width", "torch_dtype", "dtype"}
_HEADS = ("heads", "kv_heads", "dim", "vdim")
_YARN = ("original", "fast", "slow")


def _sizes(where: str, raw, keys) -> None:
    _lacking(where, raw, keys)
    _unknown(where, raw, set(keys))
    for key in keys:
        _positive(f"{where}.{key}", raw[key])


def _above_zero(where: str, value) -> float:
    number = _number(where, value)
    if not number > 0.0:
        raise ConfigError(f"{where}={number} must be positive")
    return number


def _check_rot(where: str, rot, dim: int) -> None:
    if rot is None:
        return
    _lacking(where, rot, ("base", "dims"))
    _unknown(where, rot, {"base", "dims", "scaling"})
    dims = _positive(where + ".dims", rot["dims"])
    base = _above_zero(where + ".base", rot["base"])
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}.dims={dims} must be even and at most dim={dim}")
    scaling = rot.get("scaling")
    if scaling is None:
        return
    where += ".scaling"
    _lacking(where, scaling, ("factor",))
    _unknown(where, scaling, {"factor", *_YARN})
    _above_zero(where + ".factor", scaling["factor"])
    if any(key in scaling for key in _YARN):
        _lacking(where, scaling, _YARN)
        for key in _YARN:
            _above_zero(f"{where}.{key}", scaling[key])
        if base == 1.0:
            raise ConfigError(f"{where}: a base of 1 has no frequencies to stretch by parts")


def _check_heads(where: str, m) -> None:
    _lacking(where, m, (*_HEADS, "scale"))
    for key in _HEADS:
        _positive(f"{where}.{key}", m[key])
    _number(where + ".scale", m["scale"])
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} query heads cannot share {m['kv_heads']} key/value heads")
    _check_rot(where + ".rot", m.get("rot"), m["dim"])


def _check_left(where: str, m) -> None:
    _check_heads(where, m)
    _unknown(where, m, {*_HEADS, "scale", "rot", "conv", "mask", "softcap"})
    if m.get("conv") is not None:
        _positive(where + ".conv", m["conv"])
    if m.get("softcap") is not None:
        _above_zero(where + ".softcap", m["softcap"])
    mask = m.get("mask")
    if mask is not None:
        _lacking(where + ".mask", mask, ("size",))
        _unknown(where + ".mask", mask, {"size", "keep_first"})
        _positive(where + ".mask.size", mask["size"])
        kept = mask.get("keep_first") or 0
        if isinstance(kept, bool) or not isinstance(kept, int) or kept < 0:
            raise ConfigError(f"{where}.mask.keep_first={kept!r}: a count is needed")


def _check_mixer(where: str, kind: str, m) -> None:
    if kind == "attention":
        _check_heads(where, m)
        _unknown(where, m, {*_HEADS, "scale", "rot", "kv_from"})
    elif kind == "parallel":
        keys = ("left", "right", "left_scale", "right_scale")
        _lacking(where, m, keys)
        _unknown(where, m, set(keys))
        _check_left(where + ".left", m["left"])
        _sizes(where + ".right", m["right"], ("heads", "dim", "vdim"))
        for key in ("left_scale", "right_scale"):
            _number(f"{where}.{key}", m[key])
    else:
        raise ConfigError(f"{where[:-6]}.type={kind!r}: this design's mixers are 'attention' and 'parallel'")


def _check_mlp(where: str, mlp) -> None:
    if mlp is None:
        return
    _lacking(where, mlp, ("kind",))
    if mlp["kind"] != "moe":
        raise ConfigError(f"{where}.kind={mlp['kind']!r}: this design's feed-forward is 'moe'")
    _lacking(where, mlp, ("expert", "router"))
    _unknown(where, mlp, {"kind", "expert", "router"})
    _sizes(where + ".expert", mlp["expert"], ("ff",))
    _sizes(where + ".router", mlp["router"], ("experts", "top"))
    if mlp["router"]["top"] > mlp["router"]["experts"]:
        raise ConfigError(f"{where}.router: top={mlp['router']['top']} of {mlp['router']['experts']} experts")


def _check_source(layers, i: int) -> None:
    """A layer that borrows keys and values: from an earlier attention layer that has its own, of the same shape."""
    source = layers[i]["mixer"].get("kv_from")
    if source is None:
        return
    where = f"layers[{i}].mixer.kv_from={source!r}"
    if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < i:
        raise ConfigError(f"{where} must name an earlier layer")
    other = layers[source]
    if other["type"] != "attention" or other["mixer"].get("kv_from") is not None:
        raise ConfigError(f"{where} must name an attention layer with keys and values of its own")
    for key in ("kv_heads", "dim", "vdim"):
        if other["mixer"][key] != layers[i]["mixer"][key]:
            raise ConfigError(f"{where}: {key}={layers[i]['mixer'][key]}, that layer's is {other['mixer'][key]}")


def _position(rot):
    if rot is None:
        return None
    scaling, raw = None, rot.get("scaling")
    if raw is not None:
        if "original" in raw:
            scaling = YarnRopeScaling(float(raw["factor"]), *(float(raw[key]) for key in _YARN))
        else:
            scaling = LinearRopeScaling(float(raw["factor"]))
    return PartialRopeSpec(dims=int(rot["dims"]), base=float(rot["base"]), scaling=scaling)


@dataclass(frozen=True)
class SetotarConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: tuple          # the layer dicts as config.json gives them (validated)
    torch_dtype: str = "bfloat16"

    architecture = "Setotar"

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, raw: dict) -> "SetotarConfig":
        _lacking("config.json", raw, ("layers", "norm", "streams", "vocab", "width"))
        _unknown("the model", raw, _TOP)
        _lacking("norm", raw["norm"], ("eps",))
        _unknown("norm", raw["norm"], {"eps"})
        eps = _number("norm.eps", raw["norm"]["eps"])
        if not eps >= 0.0:
            raise ConfigError(f"norm.eps={eps} must not be negative")
        layers = raw["layers"]
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json has no layers")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            _lacking(where, layer, ("type", "mixer"))
            _unknown(where, layer, {"type", "mixer", "mlp"})
            _check_mixer(where + ".mixer", layer["type"], layer["mixer"])
            _check_mlp(where + ".mlp", layer.get("mlp"))
            checked.append(copy.deepcopy(dict(layer)))
            _check_source(checked, i)
        return cls(
            vocab=_positive("vocab", raw["vocab"]),
            width=_positive("width", raw["width"]),
            streams=_positive("streams", raw["streams"]),
            norm_eps=eps,
            layers=tuple(checked),
            torch_dtype=str(raw.get("torch_dtype", raw.get("dtype", "bfloat16"))),
        )

    # ------------------------------------------------------------------ writing

    def to_dict(self) -> dict:
        return {
            "architecture": self.architecture,
            "layers": copy.deepcopy(list(self.layers)),
            "norm": {"eps": self.norm_eps},
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
            "torch_dtype": self.torch_dtype,
        }

    # ------------------------------------------------------------------ meaning

    def _attention(self, m: dict, **more) -> SinkAttentionSpec:
        return SinkAttentionSpec(
            hidden_size=self.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]),
            value_dim=int(m["vdim"]), scale=float(m["scale"]), distance_penalty=False, sink=False, head_gate=False,
            position=_position(m.get("rot")), norm_eps=self.norm_eps, **more)

    def _mixer(self, m: dict, kind: str, prefix: str):
        if kind == "attention":
            own = m.get("kv_from") is None
            spec = self._attention(m, row_norm=True, own_kv=own)
            names = {"q": "q", "q_norm": "q.norm", "o": "o"}
            if own:
                names.update({"k": "k", "v": "v", "k_norm": "k.norm"})
            return spec, {f"mixer.{k}": prefix + v for k, v in names.items()}
        raw, mask = m["left"], m["left"].get("mask") or {}
        conv = raw.get("conv")
        left = self._attention(
            raw, bias=True, unit_values=True, conv=int(conv) if conv is not None else None,
            window=int(mask["size"]) if mask else None, keep_first=int(mask.get("keep_first") or 0) if mask else 0,
            softcap=float(raw["softcap"]) if raw.get("softcap") is not None else None)
        right = ForgetWriteSpec(hidden_size=self.width, num_heads=int(m["right"]["heads"]), head_dim=int(m["right"]["dim"]),
                                value_dim=int(m["right"]["vdim"]), norm_eps=self.norm_eps)
        spec = ParallelMixerSpec(hidden_size=self.width, left=left, right=right, join="scaled_sum",
                                 left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]))
        names = {"mixer.left.o": prefix + "left.o"}
        for n in ("q", "k", "v"):
            names[f"mixer.left.{n}"] = f"{prefix}left.{n}"
            names[f"mixer.left.{n}_bias"] = f"{prefix}left.{n}.b"
            if conv is not None:
                names[f"mixer.left.{n}_conv"] = f"{prefix}left.{n}.conv"
        for logical, name in (("q", "q"), ("f", "f"), ("f_bias", "f.b"), ("lower", "lower"), ("v", "v"), ("norm", "norm"), ("o", "o")):
            names[f"mixer.right.{logical}"] = f"{prefix}right.{name}"
        return spec, names

    def _feed_forward(self, mlp: dict, prefix: str):
        experts = int(mlp["router"]["experts"])
        spec = RoutedExpertsSpec(
            hidden_size=self.width, intermediate_size=int(mlp["expert"]["ff"]), experts=experts,
            top=int(mlp["router"]["top"]), expert="gated_silu", scoring="sigmoid", router_bias=False, weigh_input=True)
        names = {"feed_forward.router": prefix + "router"}
        for e in range(experts):
            for part in ("gate", "up", "down"):
                names[f"feed_forward.e{e}_{part}"] = f"{prefix}e{e}.{part}"
        return spec, names

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec(size=self.width, eps=self.norm_eps, gain_32bit=True)
        connection = HyperConnectionSpec(streams=self.streams, channel_scale=self.width)
        layers, schedule, ignored = [], [], []
        for i, layer in enumerate(self.layers):
            prefix = f"l{i}."
            mixer, names = self._mixer(layer["mixer"], layer["type"], prefix + "mix.")
            mlp = layer.get("mlp")
            ff = None
            if mlp is not None:
                ff, ff_names = self._feed_forward(mlp, prefix + "mlp.")
                names.update(ff_names)
            for q in (1, 2):
                own = {f"norm{q}.weight": f"{prefix}norm{q}", f"connection{q}.scale": f"{prefix}ls{q}"}
                own.update({f"connection{q}.{n}": f"{prefix}hc{q}.{n}" for n in ("in", "out", "mix")})
                if q == 2 and mlp is None:
                    ignored += list(own.values())      # a layer without a feed-forward may still store these
                else:
                    names.update(own)
            layers.append(hyper_layer(mixer, ff, norm, norm if ff is not None else None, connection, names))
            source = layer["mixer"].get("kv_from")
            schedule.append(ScheduleEntry(layer=i, cache=i if source is None else int(source), writes_cache=source is None))
        return ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=self.width,
            layers=tuple(layers),
            schedule=tuple(schedule),
            final_norm=norm,
            tie_embeddings=False,
            embed_name="embed",
            final_norm_name="final.norm",
            lm_head_name="head",
            streams=self.streams,
            ignored_tensors=tuple(ignored),
        )
