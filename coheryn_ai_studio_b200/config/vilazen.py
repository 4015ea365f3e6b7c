"""Typed configuration of the Vilazen decoder and its layout as parts.

The design: the stream starts as a normalised table row; layers with ONE norm whose output both sub-layers read,
x <- x + mixer(h) + ff(h), h = norm1(x) (arrangement ``parallel_residual``; norm weights stored around zero; the
feed-forward may be absent); a final norm and a head.  Three kinds of mixer, chosen per layer by ``type``:

* ``attention``         grouped-query attention over a sliding window that keeps the first positions of the sequence in
                        sight, whole projections of q and k normalised, values mixed with those of the first such layer, a
                        gate per head (``parts/attention.py``: ``MapsAttention``);
* ``parallel``          a causal grouped-query attention with biases, a learned sink and a gate per head, beside a linear
                        attention with a constant decay per head (``parts/recurrent.py``: ``SideBySide`` of
                        ``MapsAttention`` and ``LightningAttention``);
* ``latent_attention``  one cached latent row per position and a rotated key part shared by the heads, over a sliding
                        window (``parts/attention.py``: ``LatentAttention``).

All rotations turn neighbouring channels.  The feed-forward is dense without a gate, with the exact GELU
(``parts/feedforward.py``: ``MLP``).

``config.json`` (key ``architecture``) gives every size and every constant that differs between models of the design.
Tensor names follow the checkpoint: ``embed``, ``embed.norm``, ``head``, ``final.norm`` and ``l<i>.norm1``, ``l<i>.mix.*``
(``l<i>.mix.left.*`` and ``l<i>.mix.right.*`` for mixers side by side), ``l<i>.mlp.*``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .kapudra import DEFAULT_MAX_POSITIONS, _int, _num, _obj
from .qwen2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ACTIVATION = "gelu"           # of every feed-forward: fixed by the design


@dataclass(frozen=True)
class VilazenConfig:
    """The parsed ``config.json``; ``layers`` keeps each layer's object as read (validated)."""

    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    max_positions: int = DEFAULT_MAX_POSITIONS     # angles are computed from the position: nothing bounds it but index arithmetic
    eos_token_ids: tuple = ()

    architecture = "Vilazen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VilazenConfig":
        if d.get("architecture", d.get("architectures", ["Vilazen"])) not in ("Vilazen", ["Vilazen"]):
            raise ConfigError("not a Vilazen configuration")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("layers must be a non-empty list")
        values = None          # how many value channels the layers that mix values have
        for i, L in enumerate(layers):
            what = f"layers[{i}]"
            _check_layer(_obj(L, what), what)
            if L["type"] == "attention" and L["mixer"].get("v_mix"):
                n = L["mixer"]["kv_heads"] * L["mixer"]["vdim"]
                if values is not None and n != values:
                    raise ConfigError(f"{what}: layers that mix values must have equally many value channels ({n} and {values})")
                values = n
        return cls(
            vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"),
            norm_eps=_num(_obj(d.get("norm"), "norm"), "eps", "norm"), layers=tuple(layers),
            max_positions=_int(d, "max_positions", "config") if "max_positions" in d else DEFAULT_MAX_POSITIONS)

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": list(self.layers)}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out


def _check_rotation(m: Dict[str, Any], channels: int, where: str) -> None:
    rot = _obj(m.get("rot"), where + ".rot")
    dims = _int(rot, "dims", where + ".rot", 2)
    if dims % 2 or dims > channels:
        raise ConfigError(f"{where}.rot.dims {dims} must be even and at most the {channels} channels that may turn")
    if not _num(rot, "base", where + ".rot") > 1:
        raise ConfigError(f"{where}.rot.base must exceed 1")


def _check_heads(m: Dict[str, Any], where: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _int(m, key, where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} heads do not divide into {m['kv_heads']} kv_heads")
    _num(m, "scale", where)
    _check_rotation(m, m["dim"], where)


def _check_mask(m: Dict[str, Any], where: str, keeps: bool) -> None:
    if m.get("mask") is None:
        return
    mask = _obj(m["mask"], where + ".mask")
    _int(mask, "size", where + ".mask")
    if mask.get("keep_first") is not None:
        if not keeps:
            raise ConfigError(f"{where}.mask.keep_first belongs to the attention over a window")
        _int(mask, "keep_first", where + ".mask", 0)


def _check_layer(L: Dict[str, Any], what: str) -> None:
    kind = L.get("type")
    m, where = _obj(L.get("mixer"), what + ".mixer"), what + ".mixer"
    if kind == "attention":
        _check_heads(m, where)
        _check_mask(m, where, keeps=True)
        if not isinstance(m.get("v_mix", False), bool):
            raise ConfigError(f"{where}.v_mix must be true or false")
    elif kind == "parallel":
        left, right = _obj(m.get("left"), where + ".left"), _obj(m.get("right"), where + ".right")
        _check_heads(left, where + ".left")
        for key in ("heads", "dim", "vdim"):
            _int(right, key, where + ".right")
        decay = right.get("decay")
        if (not isinstance(decay, list) or len(decay) != right["heads"]
                or not all(isinstance(a, (int, float)) and not isinstance(a, bool) and math.isfinite(a) and 0 <= a <= 1 for a in decay)):
            raise ConfigError(f"{where}.right.decay must hold one number from 0 to 1 per head")
        _num(m, "left_scale", where, positive=False)
        _num(m, "right_scale", where, positive=False)
    elif kind == "latent_attention":
        for key in ("heads", "dim", "vdim", "kv_rank"):
            _int(m, key, where)
        rot_dim = _int(m, "rot_dim", where, 2)
        _num(m, "scale", where)
        _check_rotation(m, rot_dim, where)
        _check_mask(m, where, keeps=False)
    else:
        raise ConfigError(f"{what}.type {kind!r} is not a mixer of this design (attention, parallel, latent_attention)")
    mlp = L.get("mlp")
    if mlp is not None:
        if _obj(mlp, what + ".mlp").get("kind") != "dense":
            raise ConfigError(f"{what}.mlp.kind {mlp.get('kind')!r} is not implemented (dense, or null for none)")
        _int(mlp, "ff", what + ".mlp")


def _rotation(m: Dict[str, Any]) -> PartSpec:
    return PartSpec("rope_computed", dict(rotary_dim=m["rot"]["dims"], theta=float(m["rot"]["base"]), pairs="neighbours"))


def _mixer_spec(L: Dict[str, Any], width: int, eps: float, value_mix: Optional[str]) -> Tuple[PartSpec, Optional[PartSpec]]:
    """(mixer, position encoding of the layer)."""
    m = L["mixer"]
    mask = m.get("mask") or {}
    if L["type"] == "latent_attention":
        return PartSpec("latent_attention", dict(
            hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
            kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=eps, window=mask.get("size"))), _rotation(m)
    if L["type"] == "attention":
        return PartSpec("attention_maps", dict(
            hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            scale=float(m["scale"]), window=mask.get("size"), keep_first=int(mask.get("keep_first") or 0), qk_norm="projection",
            gate=True, value_mix=value_mix, eps=eps, float32_output=True)), _rotation(m)
    left, right = m["left"], m["right"]
    attention = PartSpec("attention_maps", dict(
        hidden_size=width, num_heads=left["heads"], num_kv_heads=left["kv_heads"], head_dim=left["dim"], v_head_dim=left["vdim"],
        scale=float(left["scale"]), qkv_bias=True, learned_sink=True, gate=True, eps=eps, float32_output=True))
    lightning = PartSpec("lightning_attention", dict(
        hidden_size=width, num_heads=right["heads"], head_dim=right["dim"], v_head_dim=right["vdim"],
        decay=tuple(float(a) for a in right["decay"]), eps=eps))
    return PartSpec("side_by_side", dict(hidden_size=width, mixers=(
        ("left", attention, float(m["left_scale"]), _rotation(left)),
        ("right", lightning, float(m["right_scale"]), None)))), None


def vilazen_model_spec(c: VilazenConfig) -> ModelSpec:
    norm = lambda: PartSpec("rmsnorm", dict(size=c.width, eps=c.norm_eps, tensor="", offset=1.0))
    layers: List[LayerSpec] = []
    mixed = False              # whether an earlier layer left its values to mix with
    for i, L in enumerate(c.layers):
        value_mix = None
        if L["type"] == "attention" and L["mixer"].get("v_mix"):
            value_mix, mixed = "later" if mixed else "first", True
        mixer, position = _mixer_spec(L, c.width, c.norm_eps, value_mix)
        parts = {"norm": norm(), "mixer": mixer}
        if L.get("mlp") is not None:
            parts["feed_forward"] = PartSpec("mlp", dict(hidden_size=c.width, intermediate_size=L["mlp"]["ff"],
                                                         activation=ACTIVATION, tensors=("up", "down")))
        layers.append(LayerSpec(f"l{i}", "parallel_residual", parts, position,
                                names={"norm": "norm1", "mixer": "mix", "feed_forward": "mlp"}))
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab, max_positions=c.max_positions,
        embedding_name="embed", layers=layers, schedule=[ScheduleEntry(i) for i in range(len(c.layers))], final_norm=norm(),
        final_norm_name="final.norm", head_name="head", bare_tensor_names=True,
        embedder=PartSpec("pair_hash_embedding", dict(vocab_size=c.vocab, hidden_size=c.width, table="embed", norm="embed.norm",
                                                      norm_offset=1.0, eps=c.norm_eps, compute_copy=False)))
