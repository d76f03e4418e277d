"""Bogivik: config.json -> typed configuration -> :class:`ModelSpec`.

A decoder-only model whose config.json lists its layers one by one (``layers``: ``type``, the mixer's sizes under ``mixer``,
the feed-forward under ``mlp`` or null).  One RMS norm per layer, and the mixer and the feed-forward both read its output:
``x += mixer(norm1(x)) + ff(norm1(x))``.  The head is a tensor of its own.  Two kinds of layer:

* ``attention``: grouped-query attention over every earlier key without rotation: queries and keys are normed over their whole
  projected rows, queries are multiplied by a temperature that grows with the position (``q_temp``), a learned number per head
  and bucket of the distance joins every score (``rel``; ``bias_max`` is the distance from which all share the last bucket),
  values are mixed with those of the first such layer (``v_mix``), and the heads pass a sigmoid gate.
* ``parallel``: two mixers read the same input and are joined as ``(U(left) * w_l + U(right) * w_r) / 2``.  ``left`` is
  grouped-query attention inside chunks of ``mask.size`` positions, with biases, a norm per query and key head, a turn of
  the first ``rot.dims`` entries of a head in the interleaved pairing with frequencies stretched by wavelength
  (``rot.scaling``), and the same gate; ``right`` is a matrix memory with exponential gates (``exp_gate``).

The feed-forward is ``down(gelu_tanh(gate h) * up h)``.  Tensor names: ``embed``, ``head``, ``final.norm``, and per layer i
``l<i>.norm1``, ``l<i>.mix.*`` (``left.*`` and ``right.*`` in a parallel layer), ``l<i>.mlp.*``.

The number of distance buckets is the row count of ``rel``: config.json does not name it, so it is read from the tensors'
shapes (a configuration without a folder may name it as ``bias_rows``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from ..config.registry import ConfigError, register_architecture
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

LAYER_TYPES = ("attention", "parallel")
# the framework's context limit when config.json names none: the design has no learned positions
DEFAULT_MAX_POSITIONS = 1 << 15
DEFAULT_BIAS_ROWS = 32                    # of a configuration that comes without tensors and names none


@dataclass(frozen=True)
class BogivikLayer:
    type: str
    mixer: Mapping[str, Any]              # the mixer's sizes and constants, checked (a parallel layer: {"left": ..., "right": ...})
    ff: int                               # 0: no feed-forward


@dataclass(frozen=True)
class BogivikConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[BogivikLayer, ...]
    max_positions: int
    raw: Mapping[str, Any]

    def to_json_dict(self) -> dict:
        return dict(self.raw)


def _int(obj: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    v = obj.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"config.json: {where}'{key}' must be an integer of at least {least}, got {v!r}")
    return v


def _num(obj: Mapping[str, Any], key: str, where: str, positive: bool = False) -> float:
    v = obj.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"config.json: {where}'{key}' must be a {'positive ' if positive else ''}number, got {v!r}")
    return float(v)


def _obj(obj: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = obj.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


def _heads(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    sizes: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if sizes["heads"] % sizes["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads={sizes['heads']} is no multiple of kv_heads={sizes['kv_heads']}")
    sizes["scale"] = _num(m, "scale", where, positive=True)
    return sizes


def _attention(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    sizes = _heads(m, where)
    sizes["bias_max"] = _num(m, "bias_max", where, positive=True)
    sizes["bias_rows"] = _int(m, "bias_rows", where, least=2) if "bias_rows" in m else DEFAULT_BIAS_ROWS
    if not sizes["bias_max"] > sizes["bias_rows"] // 2:
        raise ConfigError(f"config.json: {where}bias_max={sizes['bias_max']} must lie beyond half of the {sizes['bias_rows']} buckets")
    sizes["heat"] = None
    if m.get("q_temp") is not None:
        t = _obj(m, "q_temp", where)
        sizes["heat"] = (_num(t, "coef", where + "q_temp."), _num(t, "every", where + "q_temp.", positive=True))
    v_mix = m.get("v_mix", False)
    if not isinstance(v_mix, bool):
        raise ConfigError(f"config.json: {where}'v_mix' must be true or false, got {v_mix!r}")
    sizes["v_mix"] = v_mix
    return sizes


def _left(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    sizes = _heads(m, where)
    # a layer without a mask (null, or no key at all) sees every key; without a rotation nothing turns
    sizes["chunk"] = _int(_obj(m, "mask", where), "size", where + "mask.") if m.get("mask") is not None else None
    sizes["rot"] = None
    if m.get("rot") is not None:
        rot, rw = _obj(m, "rot", where), where + "rot."
        base, dims = _num(rot, "base", rw, positive=True), _int(rot, "dims", rw)
        if dims % 2 or dims > sizes["dim"]:
            raise ConfigError(f"config.json: {rw}dims={dims} must be even and at most {sizes['dim']}")
        scaling = None
        if rot.get("scaling") is not None:
            sc = _obj(rot, "scaling", rw)
            scaling = {k: _num(sc, k, rw + "scaling.", positive=True) for k in ("factor", "low", "high", "original")}
            if base == 1.0:
                raise ConfigError(f"config.json: {rw}base=1 turns every pair alike and cannot be stretched")
        sizes["rot"] = {"base": base, "dims": dims, "scaling": scaling}
    return sizes


def parse_bogivik_config(raw: Mapping[str, Any]) -> BogivikConfig:
    missing = [k for k in ("vocab", "width", "layers", "norm") if k not in raw]
    if missing:
        raise ConfigError("config.json: missing required key(s): " + ", ".join(missing))
    if not isinstance(raw["layers"], list) or not raw["layers"]:
        raise ConfigError("config.json: 'layers' must be a list with at least one layer")
    eps = _num(_obj(raw, "norm", ""), "eps", "norm.", positive=True)
    layers = []
    mixed = None                                                             # the values that v_mix layers share: (layer, heads, size)
    for i, entry in enumerate(raw["layers"]):
        where = f"layers[{i}]."
        if not isinstance(entry, Mapping):
            raise ConfigError(f"config.json: layers[{i}] must be an object")
        kind, m, mw = entry.get("type"), _obj(entry, "mixer", where), where + "mixer."
        if kind == "attention":
            sizes = _attention(m, mw)
            if sizes["v_mix"]:
                if mixed is None:
                    mixed = (i, sizes["kv_heads"], sizes["vdim"])
                    sizes["v_mix"] = "first"
                else:
                    if mixed[1] * mixed[2] != sizes["kv_heads"] * sizes["vdim"]:
                        raise ConfigError(f"config.json: {mw}v_mix: the values of layers[{mixed[0]}] ({mixed[1]} x {mixed[2]}) cannot be mixed "
                                          f"into {sizes['kv_heads']} x {sizes['vdim']}")
                    sizes["v_mix"] = "mix"
        elif kind == "parallel":
            right, rw = _obj(m, "right", mw), mw + "right."
            sizes = {"left": _left(_obj(m, "left", mw), mw + "left."),
                     "right": {**{k: _int(right, k, rw) for k in ("heads", "dim", "vdim")}, "gate_cap": _num(right, "gate_cap", rw, positive=True)}}
        else:
            raise ConfigError(f"config.json: {where}type={kind!r} is not a layer of this design ({', '.join(LAYER_TYPES)})")
        f, ff = entry.get("mlp"), 0
        if f is not None:
            if not isinstance(f, Mapping) or f.get("kind") != "dense":
                raise ConfigError(f"config.json: {where}mlp must be null or an object of kind 'dense'")
            ff = _int(f, "ff", where + "mlp.")
        layers.append(BogivikLayer(kind, sizes, ff))
    max_positions = _int(raw, "max_positions", "") if "max_positions" in raw else DEFAULT_MAX_POSITIONS
    return BogivikConfig(vocab=_int(raw, "vocab", ""), width=_int(raw, "width", ""), eps=eps, layers=tuple(layers),
                         max_positions=max_positions, raw=dict(raw))


def bias_rows_from_shapes(raw: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Mapping[str, Any]:
    """``bias_rows`` of every attention layer that does not name it: the row count of its ``rel``."""
    layers = raw.get("layers")
    if not isinstance(layers, list):
        return raw
    out = []
    for i, entry in enumerate(layers):
        shape = shapes.get(f"l{i}.mix.rel")
        if isinstance(entry, Mapping) and isinstance(entry.get("mixer"), Mapping) and "bias_rows" not in entry["mixer"] and shape:
            entry = {**entry, "mixer": {**entry["mixer"], "bias_rows": int(shape[0])}}
        out.append(entry)
    return {**raw, "layers": out}


def build_bogivik_spec(cfg: BogivikConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps, "name": name, "float32_weight": True})

    def attention(m: Mapping[str, Any], **more: Any) -> PartSpec:
        return PartSpec("normed_attention", {
            "hidden_size": cfg.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "scale": m["scale"], "eps": cfg.eps, "gate": True, **more})

    layers = []
    for layer in cfg.layers:
        m = layer.mixer
        norms, prefixes, extra = {"norm1": norm("norm1")}, {"mixer": "mix.", "ffn": "mlp.", "norm1": ""}, {}
        if layer.type == "attention":
            mixer = attention(m, qk_norm="row", heat=m["heat"], value_mix=m["v_mix"] or None, bias_rows=m["bias_rows"], bias_max=m["bias_max"])
        else:
            lf, rt, rot = m["left"], m["right"], m["left"]["rot"]
            position = PartSpec("rope_span", {"head_dim": lf["dim"], "dims": rot["dims"], "theta": rot["base"], "interleaved": True,
                                              "scaling": rot["scaling"]}) if rot else None
            mixer = attention(lf, qk_norm="head", position=position, chunk=lf["chunk"], qkv_bias=True, out_bias=True)
            extra["mixer2"] = ("mixer", PartSpec("exp_gate", {"hidden_size": cfg.width, "heads": rt["heads"], "dim": rt["dim"], "vdim": rt["vdim"],
                                                               "gate_cap": rt["gate_cap"], "eps": cfg.eps}))
            norms.update({"mix_out": norm("out"), "mix2_out": norm("out")})
            prefixes.update({"mixer": "mix.left.", "mixer2": "mix.right.", "mix_out": "mix.left.", "mix2_out": "mix.right."})
        ffn = PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": layer.ff, "activation": "gelu_tanh",
                                     "names": {"gate": "gate", "up": "up", "down": "down"}}) if layer.ff else None
        layers.append(LayerSpec(block="shared_norm", mixer=mixer, ffn=ffn, norms=norms, prefixes=prefixes, extra=extra))
    schedule = tuple(LayerCall(i) for i in range(len(layers)))          # no loops: call i is layer i
    return ModelSpec(
        architecture="Bogivik", vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers), schedule=schedule,
        final_norm=norm("norm"), tie_word_embeddings=False, max_position_embeddings=cfg.max_positions,
        layer_prefix="l{i}.", embed_name="embed", final_norm_prefix="final.", head_name="head")


BOGIVIK = register_architecture("Bogivik", model_types=("bogivik",), parse=parse_bogivik_config, build_spec=build_bogivik_spec,
                                kernel_libraries=("rowwise", "ssm", "linrec"), sizes_from_shapes=bias_rows_from_shapes)
