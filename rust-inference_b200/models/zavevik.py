"""Zavevik: a decoder whose sublayers read the residual itself, with a norm only BEHIND each of them,
x <- x + n1(mixer(x)), x <- x + n2(ff(x)), the norms RMS norms with one number as gain; after the feed-forward every layer
takes in the token itself once more, x <- x + n3(proj(gelu_tanh(gate x) * e)) with e the layer's part of the token's row in
a table of its own.  The mixers are grouped-query attention without rotation (queries and keys divided by their root mean
square, queries multiplied by a factor that grows with the position, normed values, capped scores, a learned bias per
head by distance in buckets; a layer may read another layer's keys and values instead of having its own) and the gated
delta rule with one decay per head.  The feed-forward is a routed one without a router: a table names every token id's
experts.

config.json keys (every size and every constant that may differ between models comes from here)::

    architecture        "Zavevik"
    vocab, width        sizes of the embedding table
    norm.eps            eps of every norm
    token_side.dim      size of a layer's part of a token's row (absent: no such sublayer)
    layers[i]           {type "attention" | "delta", mixer, mlp}
      mixer (attention)   heads, kv_heads, dim (queries and keys), vdim (values), scale, softcap, q_temp {coef, every}
                          (both optional), bias_max (largest distance of the bias' buckets; absent: no bias), kv_from
                          (optional: the layer whose keys and values this one reads)
      mixer (delta)       heads, kv_heads, dim, vdim, conv
      mlp                 null or {kind "moe", router {experts, top}, expert {ff}}

The number of rows of a distance bias comes from its tensor's shape (``bias_rows`` in a mixer's record says it where no
checkpoint is at hand).

Tensor names: ``embed``, ``side.embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1|norm2``,
``l<i>.mix.q|k|v|rel|o`` or ``l<i>.mix.q|k|v`` (+ ``.conv``) ``|b|a|A_log|dt_bias|g|norm|o``,
``l<i>.mlp.table|e<j>.gate|up|down``, ``l<i>.side.gate|proj|norm``.  The model itself is not written here: ``to_spec``
names the parts and the order in which the generic model runs them (``engine/model.py``).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Tuple

from ..config.registry import ConfigError, register_architecture
from ..config.specs import (AttentionSpec, EmbeddingSpec, GatedDeltaSpec, GatedFFSpec, HeadSpec, ModelSpec, MoESpec, NoNormSpec,
                            PostLayerSpec, PostNormSpec, RMSGainsSpec, ScheduleEntry, TokenSideSpec)
from .ranudra import MAX_POSITIONS, _checkpoint_shapes, _freeze, _get, _pos_int, _thaw

LAYER_TYPES = ("attention", "delta")
BIAS_NAME, SIDE_NAME = "rel", "side.embed"


@register_architecture("Zavevik", "zavevik")
@dataclass(frozen=True)
class ZavevikConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[tuple, ...]                    # frozen layer records of config.json
    side_dim: int = 0
    eos_token_ids: Tuple[int, ...] = ()

    # ---- config.json <-> object -------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "ZavevikConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        side = d.get("token_side")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, list) else [eos]))
        return cls(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"),
                   eps=float(_get(d.get("norm"), "eps", "norm")), layers=tuple(_freeze(l) for l in layers),
                   side_dim=0 if side is None else _pos_int(side, "dim", "token_side"), eos_token_ids=eos_ids)

    def layer_records(self):
        return [_thaw(l) for l in self.layers]

    def to_dict(self) -> dict:
        d = {"architecture": "Zavevik", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": self.layer_records()}
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- checks ------------------------------------------------------------------
    @staticmethod
    def _check_attention(records, i, what):
        m = records[i]["mixer"]
        if not float(_get(m, "scale", what)) > 0:
            raise ConfigError(f"config.json: {what}.scale must be positive")
        if m.get("softcap") is not None and not float(_get(m, "softcap", what)) > 0:
            raise ConfigError(f"config.json: {what}.softcap must be positive")
        temp = m.get("q_temp")
        if temp is not None:
            _get(temp, "coef", what + ".q_temp")
            if not float(_get(temp, "every", what + ".q_temp")) > 0:
                raise ConfigError(f"config.json: {what}.q_temp.every must be positive")
        if m.get("bias_max") is not None and not float(_get(m, "bias_max", what)) > 0:
            raise ConfigError(f"config.json: {what}.bias_max must be positive")
        j = m.get("kv_from")
        if j is None:
            return
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
            raise ConfigError(f"config.json: {what}.kv_from {j!r} must name an earlier layer")
        other = records[j].get("mixer") or {}
        if records[j].get("type") != "attention" or other.get("kv_from") is not None:
            raise ConfigError(f"config.json: {what}.kv_from {j}: that layer has no keys and values of its own")
        for key in ("heads", "kv_heads", "dim", "vdim"):
            if other.get(key) != m[key]:
                raise ConfigError(f"config.json: {what}.kv_from {j}: {key} is {other.get(key)} there and {m[key]} here")

    def validate(self) -> None:
        if not (self.eps > 0):
            raise ConfigError("norm.eps must be positive")
        records = self.layer_records()
        for i, layer in enumerate(records):
            what = f"layers[{i}]"
            kind = layer.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {what}.type {kind!r} is not built (known: {', '.join(LAYER_TYPES)})")
            m = layer.get("mixer")
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _pos_int(m, key, what + ".mixer")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"config.json: {what}.mixer: {m['heads']} heads over {m['kv_heads']} kv_heads")
            if kind == "attention":
                self._check_attention(records, i, what + ".mixer")
            else:
                _pos_int(m, "conv", what + ".mixer")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") != "moe":
                raise ConfigError(f"config.json: {what}.mlp.kind {mlp.get('kind')!r} is not built (known: moe)")
            r = mlp.get("router")
            E, top = _pos_int(r, "experts", what + ".mlp.router"), _pos_int(r, "top", what + ".mlp.router")
            if top > E:
                raise ConfigError(f"config.json: {what}.mlp.router: top {top} of {E} experts")
            _pos_int(mlp.get("expert"), "ff", what + ".mlp.expert")

    # ---- the model as parts --------------------------------------------------------
    def _mixer(self, kind, m):
        if kind == "delta":
            return GatedDeltaSpec(hidden_size=self.width, num_heads=m["heads"], num_qk_heads=m["kv_heads"], dim=m["dim"],
                                  vdim=m["vdim"], conv=m["conv"], decay_rank=0, gate_rank=0, eps=self.eps, decay="head",
                                  gate="full", gate_fn="silu")
        temp = m.get("q_temp")
        bias_rows = 0
        if m.get("bias_max") is not None:
            bias_rows = int(m.get("bias_rows", 0))
            if bias_rows <= 0:
                raise ConfigError("the rows of a distance bias come from its tensor's shape (or from the key bias_rows)")
        return AttentionSpec(
            hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], scale=float(m["scale"]),
            v_head_dim=int(m["vdim"]), names=("q", "k", "v", "o", "sink"), unit_rms=True, unit_eps=self.eps, unit_values=True,
            softcap=float(m.get("softcap") or 0.0),
            temperature=None if temp is None else (float(temp["coef"]), float(temp["every"])),
            bias_rows=bias_rows, bias_far=float(m.get("bias_max") or 0.0), bias_name=BIAS_NAME, own_kv=m.get("kv_from") is None)

    def _ffn(self, mlp):
        if mlp is None:
            return None
        return MoESpec(hidden_size=self.width, experts=mlp["router"]["experts"], top=mlp["router"]["top"],
                       expert=GatedFFSpec(hidden_size=self.width, intermediate_size=mlp["expert"]["ff"], gate="silu"),
                       route="table", table_rows=self.vocab, table_name="table")

    def to_spec(self) -> ModelSpec:
        D, side = self.width, self.side_dim
        behind = PostNormSpec(size=D, eps=self.eps, gain_name="", scalar=True)
        records = self.layer_records()
        layers, schedule, entry_of = [], [], {}
        for i, layer in enumerate(records):
            ffn = self._ffn(layer.get("mlp"))
            names = (("mixer_link", f"l{i}.norm1"), ("mixer", f"l{i}.mix."), ("ffn_link", f"l{i}.norm2"), ("ffn", f"l{i}.mlp."),
                     ("side_link", f"l{i}.side."), ("side", f"l{i}.side."))
            layers.append(PostLayerSpec(
                mixer=self._mixer(layer["type"], layer["mixer"]), reader=NoNormSpec(size=D), mixer_link=behind,
                ffn=ffn, ffn_link=None if ffn is None else behind,
                side=TokenSideSpec(hidden_size=D, size=side, start=i * side) if side else None,
                side_link=PostNormSpec(size=D, eps=self.eps, gain_name="norm") if side else None, names=names))
            lender = layer["mixer"].get("kv_from")
            if lender is None:
                entry_of[i] = len(entry_of)
            schedule.append(ScheduleEntry(layer=i, cache=entry_of[i if lender is None else lender], writes=lender is None))
        return ModelSpec(
            architecture="Zavevik", vocab_size=self.vocab, hidden_size=D, layers=tuple(layers), schedule=tuple(schedule),
            final_norm=RMSGainsSpec(size=D, eps=self.eps, names=("",), scalar=True), tie_embeddings=False,
            max_positions=MAX_POSITIONS, embedding_name="embed", head_name="head", final_norm_prefix="final.norm",
            stop_ids=self.eos_token_ids, head_optional=False,
            embedding=EmbeddingSpec(self.vocab, D, side_width=len(records) * side, side_name="side"),
            head=HeadSpec(self.vocab, D), end_names=(("side", SIDE_NAME),))

    # ---- sizes that only the checkpoint knows -------------------------------------------------------
    def with_checkpoint(self, model_dir: str) -> "ZavevikConfig":
        """The configuration with the numbers of rows of the distance biases filled in, from ``l<i>.mix.rel``."""
        shapes = None
        out = []
        for i, layer in enumerate(self.layer_records()):
            m = layer["mixer"]
            if layer["type"] == "attention" and m.get("bias_max") is not None and "bias_rows" not in m:
                if shapes is None:
                    shapes = _checkpoint_shapes(model_dir)
                shape = shapes.get(f"l{i}.mix.{BIAS_NAME}")
                if shape is None or len(shape) != 2:
                    raise ConfigError(f"{model_dir}: l{i}.mix.{BIAS_NAME} is missing, so the number of its buckets is unknown")
                layer = dict(layer, mixer=dict(m, bias_rows=int(shape[0])))
            out.append(_freeze(layer))
        return replace(self, layers=tuple(out))
