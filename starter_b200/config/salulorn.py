"""Configuration of the Salulorn decoder, read from the keys of its own ``config.json``.

The design: one residual stream that is a 32-bit sum; layers with one norm whose output both sublayers read, added onto
the stream together; a run of layers that is passed through several times with the same weights (each pass with keys,
values and states of its own), every pass opened by a projection of the stream and the embedding output side by side;
per layer one of three mixers (``gla``: a linear recurrence with a matrix state per head and a decay per key channel;
``attention``: window attention with biases, short convolutions, norms over the whole query and key projections,
rotary positions, capped scores and a sink; ``latent_attention``: attention over a cached low-rank latent with a
rotated key part shared by all heads, YaRN-stretched positions, a sink and an output gate) and a gated dense
feed-forward, or none; a final norm and an output head of its own.

``config.json`` gives ``architecture``, ``vocab``, ``width``, ``norm.eps``, optionally ``loop = {start, stop, times}``, and a list
``layers``; a layer has ``type``, ``mixer`` and ``mlp``:

* ``gla``: ``mixer = {heads, dim, vdim, tau}``.  The rank of the decay's two small matrices is the one size that config.json
  leaves to the checkpoint (the shape of ``l<i>.mix.a1``); ``load_model`` reads it from there.  A model made without a
  checkpoint (random weights) states it as ``mixer.decay_rank``.
* ``attention``: ``mixer = {heads, kv_heads, dim, vdim, scale, conv?, rot?, mask{size}?, softcap?}``.
* ``latent_attention``: ``mixer = {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot}`` with ``rot.dims = rot_dim``.
* ``rot = {base, dims, scaling?}``; ``scaling = {factor, original, fast, slow}`` stretches the frequencies by parts (YaRN).
* ``mlp``: null or ``{kind: "dense", ff}``.

Every size and constant is read from there; a key this design does not know is an error.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, replace
from typing import Optional

from .kesedra import _lacking, _number, _positive, _unknown
from .qwen3 import ConfigError
from .spec import (
    EmbeddingJoinSpec,
    GatedFeedForwardSpec,
    GatedLinearAttentionSpec,
    InterleavedRopeSpec,
    Junction,
    LatentAttentionSpec,
    ModelSpec,
    NormSpec,
    SinkAttentionSpec,
    YarnRopeScaling,
    default_schedule,
    looped_schedule,
    parallel32_layer,
)

_TOP = {"architecture", "architectures", "layers", "loop", "norm", "vocab", "width", "torch_dtype", "dtype"}
_YARN = ("factor", "original", "fast", "slow")
_GLA = ("heads", "dim", "vdim")
_HEADS = ("heads", "kv_heads", "dim", "vdim")
_LATENT = ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")


def _above_zero(where: str, value) -> float:
    number = _number(where, value)
    if not number > 0.0:
        raise ConfigError(f"{where}={number} must be positive")
    return number


def _sizes(where: str, raw, keys) -> None:
    _lacking(where, raw, keys)
    for key in keys:
        _positive(f"{where}.{key}", raw[key])


def _check_rot(where: str, rot, dim: int) -> None:
    _lacking(where, rot, ("base", "dims"))
    _unknown(where, rot, {"base", "dims", "scaling"})
    base = _above_zero(where + ".base", rot["base"])
    dims = _positive(where + ".dims", rot["dims"])
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}.dims={dims} must be even and at most {dim}")
    scaling = rot.get("scaling")
    if scaling is None:
        return
    where += ".scaling"
    _lacking(where, scaling, _YARN)
    _unknown(where, scaling, set(_YARN))
    for key in _YARN:
        _above_zero(f"{where}.{key}", scaling[key])
    if base == 1.0:
        raise ConfigError(f"{where}: a base of 1 has no frequencies to stretch by parts")


def _check_mixer(where: str, kind: str, m) -> None:
    if kind == "gla":
        _sizes(where, m, _GLA)
        _lacking(where, m, ("tau",))
        _unknown(where, m, {*_GLA, "tau", "decay_rank"})
        _above_zero(where + ".tau", m["tau"])
        if m.get("decay_rank") is not None:
            _positive(where + ".decay_rank", m["decay_rank"])
    elif kind == "attention":
        _sizes(where, m, _HEADS)
        _lacking(where, m, ("scale",))
        _unknown(where, m, {*_HEADS, "scale", "conv", "rot", "mask", "softcap"})
        _number(where + ".scale", m["scale"])
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: {m['heads']} query heads cannot share {m['kv_heads']} key/value heads")
        if m.get("conv") is not None:
            _positive(where + ".conv", m["conv"])
        if m.get("softcap") is not None:
            _above_zero(where + ".softcap", m["softcap"])
        if m.get("rot") is not None:
            _check_rot(where + ".rot", m["rot"], m["dim"])
        if m.get("mask") is not None:
            _sizes(where + ".mask", m["mask"], ("size",))
            _unknown(where + ".mask", m["mask"], {"size"})
    elif kind == "latent_attention":
        _sizes(where, m, _LATENT)
        _lacking(where, m, ("scale", "rot"))
        _unknown(where, m, {*_LATENT, "scale", "rot"})
        _number(where + ".scale", m["scale"])
        _check_rot(where + ".rot", m["rot"], m["rot_dim"])
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ConfigError(f"{where}.rot.dims={m['rot']['dims']}: the whole rotated part turns, rot_dim={m['rot_dim']}")
    else:
        raise ConfigError(f"{where[:-6]}.type={kind!r}: this design's mixers are 'gla', 'attention' and 'latent_attention'")


def _check_mlp(where: str, mlp) -> None:
    if mlp is None:
        return
    _lacking(where, mlp, ("kind",))
    if mlp["kind"] != "dense":
        raise ConfigError(f"{where}.kind={mlp['kind']!r}: this design's feed-forward is 'dense'")
    _sizes(where, mlp, ("ff",))
    _unknown(where, mlp, {"kind", "ff"})


def _check_loop(loop, n_layers: int) -> None:
    _lacking("loop", loop, ("start", "stop", "times"))
    _unknown("loop", loop, {"start", "stop", "times"})
    _positive("loop.times", loop["times"])
    _positive("loop.stop", loop["stop"])
    start, stop = loop["start"], loop["stop"]
    if isinstance(start, bool) or not isinstance(start, int) or not 0 <= start < stop <= n_layers:
        raise ConfigError(f"loop: layers {start!r} to {stop!r} (exclusive) are no run of {n_layers} layers")


def _position(rot) -> Optional[InterleavedRopeSpec]:
    if rot is None:
        return None
    raw = rot.get("scaling")
    scaling = YarnRopeScaling(*(float(raw[key]) for key in _YARN)) if raw is not None else None
    return InterleavedRopeSpec(dims=int(rot["dims"]), base=float(rot["base"]), scaling=scaling)


@dataclass(frozen=True)
class SalulornConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                  # the layer dicts as config.json gives them (validated)
    loop: Optional[dict] = None    # {start, stop, times}
    torch_dtype: str = "bfloat16"

    architecture = "Salulorn"

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, raw: dict) -> "SalulornConfig":
        _lacking("config.json", raw, ("layers", "norm", "vocab", "width"))
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
        if raw.get("loop") is not None:
            _check_loop(raw["loop"], len(checked))
        return cls(
            vocab=_positive("vocab", raw["vocab"]),
            width=_positive("width", raw["width"]),
            norm_eps=eps,
            layers=tuple(checked),
            loop=copy.deepcopy(raw.get("loop")),
            torch_dtype=str(raw.get("torch_dtype", raw.get("dtype", "bfloat16"))),
        )

    def with_tensor_shapes(self, shapes: dict) -> "SalulornConfig":
        """The same configuration with the sizes that only the checkpoint gives filled in from ``shapes`` (tensor name ->
        shape): the rank of every recurrent layer's decay matrices."""
        layers = []
        for i, layer in enumerate(self.layers):
            layer = copy.deepcopy(layer)
            name = f"l{i}.mix.a1"
            if layer["type"] == "gla" and name in shapes and len(shapes[name]) == 2:
                rank = int(shapes[name][0])
                stated = layer["mixer"].get("decay_rank")
                if stated is not None and stated != rank:
                    raise ConfigError(f"layers[{i}].mixer.decay_rank={stated}, but {name} has {rank} rows")
                layer["mixer"]["decay_rank"] = rank
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    # ------------------------------------------------------------------ writing

    def to_dict(self) -> dict:
        out = {
            "architecture": self.architecture,
            "layers": copy.deepcopy(list(self.layers)),
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
            "torch_dtype": self.torch_dtype,
        }
        if self.loop is not None:
            out["loop"] = copy.deepcopy(self.loop)
        return out

    # ------------------------------------------------------------------ meaning

    def _mixer(self, i: int, m: dict, kind: str, prefix: str):
        if kind == "gla":
            if m.get("decay_rank") is None:
                raise ConfigError(f"layers[{i}]: the rank of the decay matrices is given neither by a checkpoint "
                                  f"({prefix}a1) nor by mixer.decay_rank")
            spec = GatedLinearAttentionSpec(
                hidden_size=self.width, num_heads=int(m["heads"]), head_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                tau=float(m["tau"]), decay_rank=int(m["decay_rank"]), norm_eps=self.norm_eps)
            names = {n: n for n in ("q", "k", "v", "g", "o", "norm", "a1", "a2")}
            names["a2_bias"] = "a2.b"
        elif kind == "attention":
            conv, mask = m.get("conv"), m.get("mask")
            spec = SinkAttentionSpec(
                hidden_size=self.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                head_dim=int(m["dim"]), value_dim=int(m["vdim"]), scale=float(m["scale"]), distance_penalty=False,
                sink=True, head_gate=False, window=int(mask["size"]) if mask is not None else None,
                position=_position(m.get("rot")), softcap=float(m["softcap"]) if m.get("softcap") is not None else None,
                bias=True, conv=int(conv) if conv is not None else None, row_norm=True, norm_eps=self.norm_eps)
            names = {"o": "o", "sink": "sink", "q_norm": "q.norm", "k_norm": "k.norm"}
            for n in ("q", "k", "v"):
                names[n], names[n + "_bias"] = n, n + ".b"
                if conv is not None:
                    names[n + "_conv"] = n + ".conv"
        else:
            spec = LatentAttentionSpec(
                hidden_size=self.width, num_heads=int(m["heads"]), head_dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
                value_dim=int(m["vdim"]), q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                norm_eps=self.norm_eps, position=_position(m["rot"]), sink=True, output_gate=True)
            names = {n: n for n in ("dq", "uq", "dkv", "uk", "uv", "sink", "g", "o")}
            names.update({"dq_norm": "dq.norm", "dkv_norm": "dkv.norm"})
        return spec, {f"mixer.{k}": prefix + v for k, v in names.items()}

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec(size=self.width, eps=self.norm_eps, gain_32bit=True)
        layers = []
        for i, layer in enumerate(self.layers):
            prefix = f"l{i}."
            mixer, names = self._mixer(i, layer["mixer"], layer["type"], prefix + "mix.")
            names["norm1.weight"] = prefix + "norm1"
            ff, mlp = None, layer.get("mlp")
            if mlp is not None:
                ff = GatedFeedForwardSpec(hidden_size=self.width, intermediate_size=int(mlp["ff"]))
                names.update({f"feed_forward.{n}": f"{prefix}mlp.{n}" for n in ("gate", "up", "down")})
            layers.append(parallel32_layer(mixer, ff, norm, names))
        schedule, junctions = default_schedule(len(layers)), ()
        if self.loop is not None:
            schedule = looped_schedule(len(layers), self.loop["start"], self.loop["stop"], self.loop["times"], junction=0)
            junctions = (Junction(EmbeddingJoinSpec(self.width), {"weight": "loop.in"}),)
        return ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=self.width,
            layers=tuple(layers),
            schedule=schedule,
            final_norm=norm,
            tie_embeddings=False,
            embed_name="embed",
            final_norm_name="final.norm",
            lm_head_name="head",
            junctions=junctions,
        )
