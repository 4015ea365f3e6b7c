"""Typed configuration of the Zusotar decoder and its layout as parts.

The design: the stream starts as a table row plus a learned row per position (``parts/embedding.py``:
``PositionTableEmbedding``); layers with a norm before and after each sub-layer whose contribution is multiplied by one
constant of the model, x <- x + m norm1b(mixer(norm1(x))), x <- x + m norm2b(ff(norm2(x))) (arrangement
``sandwich_residual``; norm weights stored around zero; the feed-forward with its norms may be absent); behind every layer
the stream is replaced by a weighted sum of the embedding output and all layers' results so far
(``ScheduleEntry.average``); a final norm and a head.  Three kinds of mixer, chosen per layer by ``type``:

* ``latent_attention``  one cached latent row per position, a rotated key part of neighbouring pairs shared by the heads, a
                        learned sink per head (``parts/attention.py``: ``LatentAttention``);
* ``attention``         grouped-query attention over a sliding window without rotation, values divided by their root mean
                        square, a logarithmic bias by distance with two learned numbers per head, an output gate
                        (``parts/attention.py``: ``PooledWindowAttention`` without blocks);
* ``gla``               gated linear attention (``parts/recurrent.py``: ``GatedLinearAttention``).

The feed-forward is dense (SiLU gate) or a mixture of experts (``parts/routed.py``: ``RoutedExperts``): sigmoid scores, groups
of neighbouring experts that count with their two largest scores, the chosen scores as weights, a shared expert.

``config.json`` (key ``architecture``) gives every size and every constant that differs between models of the design.
Tensor names follow the checkpoint: ``embed``, ``pos``, ``head``, ``final.norm`` and ``l<i>.norm1``, ``l<i>.norm1b``,
``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.dwa``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .kapudra import _int, _num, _obj
from .qwen2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ACTIVATION = "silu"           # of every feed-forward: fixed by the design


@dataclass(frozen=True)
class ZusotarConfig:
    """The parsed ``config.json``; ``layers`` keeps each layer's object as read (validated)."""

    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[Dict[str, Any], ...]
    eos_token_ids: tuple = ()

    architecture = "Zusotar"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZusotarConfig":
        if d.get("architecture", d.get("architectures", ["Zusotar"])) not in ("Zusotar", ["Zusotar"]):
            raise ConfigError("not a Zusotar configuration")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("layers must be a non-empty list")
        for i, L in enumerate(layers):
            _check_layer(_obj(L, f"layers[{i}]"), f"layers[{i}]")
        return cls(
            vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"), max_positions=_int(d, "max_positions", "config"),
            norm_eps=_num(_obj(d.get("norm"), "norm"), "eps", "norm"),
            residual_mult=_num(d, "residual_mult", "config", positive=False), layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "max_positions": self.max_positions,
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": list(self.layers)}


def _check_layer(L: Dict[str, Any], what: str) -> None:
    kind = L.get("type")
    m, where = _obj(L.get("mixer"), what + ".mixer"), what + ".mixer"
    if kind == "latent_attention":
        for key in ("heads", "dim", "vdim", "kv_rank"):
            _int(m, key, where)
        rot_dim = _int(m, "rot_dim", where, 2)
        _num(m, "scale", where)
        rot = _obj(m.get("rot"), where + ".rot")
        dims = _int(rot, "dims", where + ".rot", 2)
        if dims % 2 or dims > rot_dim:
            raise ConfigError(f"{where}.rot.dims {dims} must be even and at most the rotated part's {rot_dim} channels")
        if not _num(rot, "base", where + ".rot") > 1:
            raise ConfigError(f"{where}.rot.base must exceed 1")
    elif kind == "attention":
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _int(m, key, where)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: {m['heads']} heads do not divide into {m['kv_heads']} kv_heads")
        _num(m, "scale", where)
        _int(_obj(m.get("mask"), where + ".mask"), "size", where + ".mask")
    elif kind == "gla":
        for key in ("heads", "dim", "vdim"):
            _int(m, key, where)
        if m.get("a_rank") is not None:          # for random weights; a checkpoint's tensors give it
            _int(m, "a_rank", where)
        _num(m, "tau", where)
    else:
        raise ConfigError(f"{what}.type {kind!r} is not a mixer of this design (latent_attention, attention, gla)")
    mlp = L.get("mlp")
    if mlp is None:
        return
    where = what + ".mlp"
    if _obj(mlp, where).get("kind") == "dense":
        _int(mlp, "ff", where)
    elif mlp.get("kind") == "moe":
        _int(_obj(mlp.get("expert"), where + ".expert"), "ff", where + ".expert")
        r = _obj(mlp.get("router"), where + ".router")
        experts, top = _int(r, "experts", where + ".router"), _int(r, "top", where + ".router")
        count, keep = _groups(r, where + ".router")
        if experts % count:
            raise ConfigError(f"{where}.router: {experts} experts do not form {count} equal groups")
        if top > keep * (experts // count):
            raise ConfigError(f"{where}.router: {top} choices do not fit {keep} groups of {experts // count}")
        if mlp.get("shared") is not None:
            _int(_obj(mlp["shared"], where + ".shared"), "ff", where + ".shared")
    else:
        raise ConfigError(f"{where}.kind {mlp.get('kind')!r} is not implemented (dense, moe, or null for none)")


def _groups(router: Dict[str, Any], what: str) -> Tuple[int, int]:
    if router.get("groups") is None:
        return 1, 1
    g = _obj(router["groups"], what + ".groups")
    count = _int(g, "count", what + ".groups")
    return count, _int(g, "keep", what + ".groups", 1, count)


def _mixer_spec(L: Dict[str, Any], width: int, eps: float) -> Tuple[PartSpec, Optional[PartSpec]]:
    """(mixer, position encoding of the layer)."""
    m = L["mixer"]
    if L["type"] == "gla":
        return PartSpec("gated_linear_attention", dict(hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                                                       tau=float(m["tau"]), eps=eps, decay_rank=m.get("a_rank"))), None
    if L["type"] == "attention":
        return PartSpec("pooled_window_attention", dict(
            hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            scale=float(m["scale"]), window=m["mask"]["size"], gate=True, value_eps=eps, log_bias=True)), None
    position = PartSpec("rope_computed", dict(rotary_dim=m["rot"]["dims"], theta=float(m["rot"]["base"]), pairs="neighbours"))
    return PartSpec("latent_attention", dict(
        hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
        kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=eps, sink=True)), position


def _feed_forward_spec(mlp: Dict[str, Any], width: int) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=width, intermediate_size=mlp["ff"], activation=ACTIVATION,
                                          tensors=("gate", "up", "down"), float32_output=True))
    r, shared = mlp["router"], mlp.get("shared")
    count, keep = _groups(r, "router")
    return PartSpec("routed_experts", dict(
        hidden_size=width, expert_size=mlp["expert"]["ff"], experts=r["experts"], top=r["top"], groups=count, keep=keep,
        correction=False, activation=ACTIVATION, selection="sigmoid_top", group_score="two", renormalize=False,
        shared=dict(size=shared["ff"]) if shared is not None else None))


def zusotar_model_spec(c: ZusotarConfig) -> ModelSpec:
    norm = lambda factor=1.0: PartSpec("rmsnorm", dict(size=c.width, eps=c.norm_eps, tensor="", offset=1.0, factor=factor))
    layers: List[LayerSpec] = []
    for i, L in enumerate(c.layers):
        mixer, position = _mixer_spec(L, c.width, c.norm_eps)
        parts = {"mixer_norm": norm(), "mixer": mixer, "mixer_post_norm": norm(c.residual_mult)}
        if L.get("mlp") is not None:
            parts.update({"feed_forward_norm": norm(), "feed_forward": _feed_forward_spec(L["mlp"], c.width),
                          "feed_forward_post_norm": norm(c.residual_mult)})
        layers.append(LayerSpec(f"l{i}", "sandwich_residual", parts, position, names={
            "mixer_norm": "norm1", "mixer": "mix", "mixer_post_norm": "norm1b", "feed_forward_norm": "norm2",
            "feed_forward": "mlp", "feed_forward_post_norm": "norm2b"}))
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab, max_positions=c.max_positions,
        embedding_name="embed", layers=layers,
        schedule=[ScheduleEntry(i, average=f"l{i}.dwa") for i in range(len(c.layers))], final_norm=norm(),
        final_norm_name="final.norm", head_name="head", bare_tensor_names=True,
        extra_tensors={f"l{i}.dwa": ((i + 2,), "vector", "bias") for i in range(len(c.layers))},
        embedder=PartSpec("position_table_embedding", dict(vocab_size=c.vocab, hidden_size=c.width, table="embed", positions="pos",
                                                           max_positions=c.max_positions)))
