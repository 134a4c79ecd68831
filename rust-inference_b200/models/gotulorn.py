"""Gotulorn: a pre-norm decoder whose norms are Dynamic Tanh (elementwise, no statistic), also behind the embedding.  Its
mixers are differential attention (two softmax maps per head over the same values, their difference normed per head; a
sliding window beside the sequence's kept first tokens; no rotation; a layer may read another layer's keys and values
instead of having its own) and latent attention (keys and values of all heads expanded from one normed latent per token,
one rotated key part that all heads share).  Feed-forwards are dense (clamped swish) or routed (the largest router outputs,
weighted by the softmax over the chosen ones).

config.json keys (every size and every constant that may differ between models comes from here)::

    architecture        "Gotulorn"
    vocab, width        sizes of the embedding table
    embedding.scale     factor on the embedding's rows
    norm.eps            eps of the RMS norms inside the mixers (the latent's, the heads')
    layers[i]           {type "attention" | "latent_attention", mixer, mlp}
      mixer (attention)         heads, kv_heads, dim (of one map's queries and keys), vdim (values), scale, diff,
                                mask {size, keep_first} (absent: every earlier key), kv_from (optional: the layer whose keys
                                and values this one reads)
      mixer (latent_attention)  heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}
      mlp                       null, {kind "dense", ff, limit} or {kind "moe", router {experts, top}, expert {ff}}

Tensor names: ``embed``, ``embed.norm``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1|norm2`` (every norm with ``.b``
and ``.alpha``), ``l<i>.mix.q|k|v|lq1|lk1|lq2|lk2|o`` or ``l<i>.mix.q|dkv|dkv.norm|uk|uv|o``, ``l<i>.mlp.gate|up|down`` or
``l<i>.mlp.router|router.b|e<j>.gate|up|down``.  The model itself is not written here: ``to_spec`` names the parts and the
order in which the generic model runs them (``engine/model.py``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Tuple

from ..config.registry import ConfigError, register_architecture
from ..config.specs import (AttentionSpec, DynTanhSpec, EmbeddingSpec, GatedFFSpec, HeadSpec, LatentAttentionSpec, LayerSpec,
                            ModelSpec, MoESpec, NoPositionSpec, RopePairsSpec, ScheduleEntry)
from .ranudra import MAX_POSITIONS, _freeze, _get, _pos_int, _thaw

LAYER_TYPES = ("attention", "latent_attention")
SWISH_ALPHA = 1.702          # the dense feed-forward's gate: g sigmoid(1.702 g)


@register_architecture("Gotulorn", "gotulorn")
@dataclass(frozen=True)
class GotulornConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    layers: Tuple[tuple, ...]                    # frozen layer records of config.json
    eos_token_ids: Tuple[int, ...] = ()

    # ---- config.json <-> object -------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "GotulornConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, list) else [eos]))
        return cls(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"),
                   embedding_scale=float(_get(d.get("embedding"), "scale", "embedding")),
                   eps=float(_get(d.get("norm"), "eps", "norm")), layers=tuple(_freeze(l) for l in layers), eos_token_ids=eos_ids)

    def layer_records(self):
        return [_thaw(l) for l in self.layers]

    def to_dict(self) -> dict:
        d = {"architecture": "Gotulorn", "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
             "norm": {"eps": self.eps}, "layers": self.layer_records()}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- checks ------------------------------------------------------------------
    @staticmethod
    def _check_attention(records, i, what):
        m = records[i]["mixer"]
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _pos_int(m, key, what)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {what}: {m['heads']} heads over {m['kv_heads']} kv_heads")
        _get(m, "diff", what)
        mask = m.get("mask")
        if mask is not None:
            _pos_int(mask, "size", what + ".mask")
            keep = mask.get("keep_first", 0)
            if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
                raise ConfigError(f"config.json: {what}.mask.keep_first {keep!r} must be a number of tokens")
        j = m.get("kv_from")
        if j is None:
            return
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
            raise ConfigError(f"config.json: {what}.kv_from {j!r} must name an earlier layer")
        other = records[j].get("mixer") or {}
        if records[j].get("type") != "attention" or other.get("kv_from") is not None:
            raise ConfigError(f"config.json: {what}.kv_from {j}: that layer has no keys and values of its own")
        for key in ("kv_heads", "dim", "vdim"):
            if other.get(key) != m[key]:
                raise ConfigError(f"config.json: {what}.kv_from {j}: {key} is {other.get(key)} there and {m[key]} here")

    @staticmethod
    def _check_latent(m, what):
        for key in ("heads", "dim", "vdim", "kv_rank"):
            _pos_int(m, key, what)
        rot_dim = _get(m, "rot_dim", what, int)
        if rot_dim < 0 or rot_dim % 2:
            raise ConfigError(f"config.json: {what}.rot_dim {rot_dim} must be even and not negative")
        if rot_dim:
            rot = m.get("rot")
            if not float(_get(rot, "base", what + ".rot")) > 0:
                raise ConfigError(f"config.json: {what}.rot.base must be positive")
            if rot.get("dims", rot_dim) != rot_dim:
                raise ConfigError(f"config.json: {what}.rot.dims {rot['dims']} is not rot_dim {rot_dim}")

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
            if not float(_get(m, "scale", what + ".mixer")) > 0:
                raise ConfigError(f"config.json: {what}.mixer.scale must be positive")
            if kind == "attention":
                self._check_attention(records, i, what + ".mixer")
            else:
                self._check_latent(m, what + ".mixer")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") == "dense":
                _pos_int(mlp, "ff", what + ".mlp")
                _get(mlp, "limit", what + ".mlp")
            elif mlp.get("kind") == "moe":
                r = mlp.get("router")
                E, top = _pos_int(r, "experts", what + ".mlp.router"), _pos_int(r, "top", what + ".mlp.router")
                if top > E:
                    raise ConfigError(f"config.json: {what}.mlp.router: top {top} of {E} experts")
                _pos_int(mlp.get("expert"), "ff", what + ".mlp.expert")
            else:
                raise ConfigError(f"config.json: {what}.mlp.kind {mlp.get('kind')!r} is not built (known: dense, moe)")

    # ---- the model as parts --------------------------------------------------------
    def _mixer(self, kind, m):
        if kind == "latent_attention":
            position = NoPositionSpec()
            if m["rot_dim"]:
                position = RopePairsSpec(rotary_dim=m["rot_dim"], theta=float(m["rot"]["base"]))
            return LatentAttentionSpec(hidden_size=self.width, num_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"],
                                       vdim=m["vdim"], kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=self.eps, position=position)
        mask = m.get("mask") or {}
        return AttentionSpec(
            hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], scale=float(m["scale"]),
            v_head_dim=m["vdim"], names=("q", "k", "v", "o", "sink"), window=int(mask.get("size", 0)),
            keep_first=int(mask.get("keep_first", 0)), own_kv=m.get("kv_from") is None, maps=2, pair_diff=float(m["diff"]),
            pair_eps=self.eps)

    def _ffn(self, mlp):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return GatedFFSpec(hidden_size=self.width, intermediate_size=mlp["ff"], gate="clamped_swish", limit=float(mlp["limit"]),
                               alpha=SWISH_ALPHA)
        return MoESpec(hidden_size=self.width, experts=mlp["router"]["experts"], top=mlp["router"]["top"],
                       expert=GatedFFSpec(hidden_size=self.width, intermediate_size=mlp["expert"]["ff"], gate="silu"),
                       score="logits", router_bias="router.b")

    def to_spec(self) -> ModelSpec:
        norm = DynTanhSpec(size=self.width)
        layers, schedule, entry_of = [], [], {}
        for i, layer in enumerate(self.layer_records()):
            ffn = self._ffn(layer.get("mlp"))
            names = (("mixer_norm", f"l{i}.norm1"), ("mixer", f"l{i}.mix."), ("ffn_norm", f"l{i}.norm2"), ("ffn", f"l{i}.mlp."))
            layers.append(LayerSpec(mixer=self._mixer(layer["type"], layer["mixer"]), ffn=ffn, mixer_norm=norm,
                                    ffn_norm=None if ffn is None else norm, names=names))
            lender = layer["mixer"].get("kv_from") if layer["type"] == "attention" else None
            if lender is None:
                entry_of[i] = len(entry_of)
            schedule.append(ScheduleEntry(layer=i, cache=entry_of[i if lender is None else lender], writes=lender is None))
        return ModelSpec(
            architecture="Gotulorn", vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers), schedule=tuple(schedule),
            final_norm=norm, tie_embeddings=False, max_positions=MAX_POSITIONS, embedding_name="embed", head_name="head",
            final_norm_prefix="final.norm", stop_ids=self.eos_token_ids, head_optional=False,
            embedding=EmbeddingSpec(self.vocab, self.width, scale=self.embedding_scale, norm=norm),
            head=HeadSpec(self.vocab, self.width))
