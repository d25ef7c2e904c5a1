"""Typed configuration of the Nezolorn decoder.

A Nezolorn config.json names its model class as the string `architecture` and
gives `vocab`, `width`, `norm.eps`, `residual_mult`, `embedding` and a list
`layers`; every entry has a `type` (which mixer), the mixer's sizes and
constants under `mixer` and a feed-forward under `mlp` (or null).  An unknown
mixer or feed-forward kind is refused by name; a key outside the design is
ignored with a warning.

    x0 = E[token] * embedding.scale + B[(previous * mul_prev + token * mul_cur) mod buckets]
    x += m * mixer(ln(x) w1);   x += m * ff(ln(x) w2)             layer norm without bias, m = residual_mult
    logits = head (ln(x) w_final)

B (`embedding.bigram`) has a row more than buckets, the last one for a
sequence's first token.

Mixers.  `parallel`: two mixers side by side on one input, summed with
`left_scale` and `right_scale`.  Left: grouped-query attention whose values are
the keys before their rotation, pairs (i, i + dims/2) of the first `rot.dims`
dimensions turned by frequencies scaled by wavelength (`rot.scaling`), over a
window of `mask.size` tokens and, behind it, the means of whole blocks of
`mask.pool` tokens.  Right: a matrix memory with exponential gates.
`general_delta`: the generalized delta rule with a decay and a removal rate per
key channel.
Feed-forward.  `dense`: down(silu(gate x) * (up x)).

The design gives no limit on positions; `MAX_POSITIONS` is this library's
(positions are int32 on the device and are turned into float32 angles).
"""
from __future__ import annotations

import copy
import json
import warnings
from dataclasses import dataclass, field
from typing import Optional

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, ScheduleEntry, require

ARCHITECTURE = "Nezolorn"
MAX_POSITIONS = 1 << 22
UNIT_EPS = 1e-6            # under the root that makes the delta rule's k a unit vector: fixed by the design

_LEFT = {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float}
_RIGHT = {"heads": int, "dim": int, "vdim": int, "gate_cap": float}
_DELTA = {"heads": int, "dim": int}


def _typed(d, keys: dict, where: str, optional_keys: tuple = ()) -> dict:
    """The listed keys of `d`, each of its type.  A key this library does not know is left out with a warning."""
    if not isinstance(d, dict):
        raise ConfigError(f"{where}: must be an object, found {d!r}")
    unknown = sorted(set(d) - set(keys) - set(optional_keys))
    if unknown:
        warnings.warn(f"{where}: keys {unknown} are not part of the design and are ignored", stacklevel=3)
    return {k: require(d, k, typ, where) for k, typ in keys.items()}


def _left(m, w: str) -> dict:
    out = _typed(m, _LEFT, w, optional_keys=("mask", "rot"))
    if m.get("mask") is not None:
        out["mask"] = _typed(m["mask"], {"size": int}, w + ".mask", optional_keys=("pool",))
        if m["mask"].get("pool") is not None:
            out["mask"]["pool"] = require(m["mask"], "pool", int, w + ".mask")
    if m.get("rot") is not None:
        out["rot"] = _typed(m["rot"], {"base": float, "dims": int}, w + ".rot", optional_keys=("scaling",))
        if m["rot"].get("scaling") is not None:
            out["rot"]["scaling"] = _typed(m["rot"]["scaling"], {"factor": float, "low": float, "high": float,
                                                                 "original": float}, w + ".rot.scaling")
    return out


def _mixer(typ: str, m, w: str) -> dict:
    if typ == "parallel":
        out = _typed(m, {"left_scale": float, "right_scale": float}, w, optional_keys=("left", "right"))
        out["left"] = _left(m.get("left"), w + ".left")
        out["right"] = _typed(m.get("right"), _RIGHT, w + ".right")
        return out
    if typ == "general_delta":
        out = _typed(m, _DELTA, w, optional_keys=("rank",))
        if m.get("rank") is not None:            # this library's own key, written with random models (see with_shapes)
            out["rank"] = require(m, "rank", int, w)
        return out
    raise ConfigError(f"{w[:-6]}: mixer type {typ!r} is neither 'parallel' nor 'general_delta'")


def _mlp(mlp, w: str):
    if mlp is None:
        return None
    kind = require(mlp, "kind", str, w)
    if kind != "dense":
        raise ConfigError(f"{w}: kind {kind!r} is not 'dense'")
    return _typed(mlp, {"kind": str, "ff": int}, w)


@dataclass
class NezolornConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    bigram: Optional[dict] = None                   # {buckets, mul_prev, mul_cur} or None
    layers: list = field(default_factory=list)      # the entries of config.json's `layers`, checked
    max_position_embeddings: int = MAX_POSITIONS    # not a key of the design: this library's own limit

    def __post_init__(self):
        self.validate()

    # ---- reading and writing -------------------------------------------------
    @classmethod
    def from_dict(cls, cfg: dict, where: str = "config.json") -> "NezolornConfig":
        norm, emb = cfg.get("norm"), cfg.get("embedding")
        if not isinstance(norm, dict):
            raise ConfigError(f"{where}: key 'norm' must be an object with 'eps'")
        if not isinstance(emb, dict):
            raise ConfigError(f"{where}: key 'embedding' must be an object with 'scale'")
        layers = []
        for i, entry in enumerate(require(cfg, "layers", list, where)):
            w = f"{where}: layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{w}: must be an object")
            unknown = sorted(set(entry) - {"type", "mixer", "mlp"})
            if unknown:
                warnings.warn(f"{w}: keys {unknown} are not part of the design and are ignored", stacklevel=2)
            typ = require(entry, "type", str, w)
            layers.append({"type": typ, "mixer": _mixer(typ, entry.get("mixer"), w + ".mixer"),
                           "mlp": _mlp(entry.get("mlp"), w + ".mlp")})
        bigram = None
        if emb.get("bigram") is not None:
            bigram = _typed(emb["bigram"], {"buckets": int, "mul_prev": int, "mul_cur": int}, where + ": embedding.bigram")
        return cls(vocab=require(cfg, "vocab", int, where), width=require(cfg, "width", int, where),
                   norm_eps=require(norm, "eps", float, where + ": norm"),
                   residual_mult=require(cfg, "residual_mult", float, where),
                   embedding_scale=require(emb, "scale", float, where + ": embedding"), bigram=bigram, layers=layers)

    def to_dict(self) -> dict:
        emb = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = dict(self.bigram)
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "embedding": emb,
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": copy.deepcopy(self.layers)}

    # ---- checks ----------------------------------------------------------------
    def validate(self) -> None:
        bad = []
        if self.vocab <= 0 or self.width <= 0:
            bad.append("vocab and width must be positive")
        if not self.norm_eps > 0:
            bad.append(f"norm.eps must be positive, found {self.norm_eps}")
        if self.bigram is not None and self.bigram["buckets"] <= 0:
            bad.append(f"embedding.bigram.buckets must be positive, found {self.bigram['buckets']}")
        if not self.layers:
            bad.append("'layers' is empty")

        def positive(m, keys, at):
            bad.extend(f"{at}.{k} must be positive, found {m[k]}" for k in keys if m[k] <= 0)

        for i, layer in enumerate(self.layers):
            m, at = layer["mixer"], f"layers[{i}].mixer"
            if layer["type"] == "parallel":
                left, right = m["left"], m["right"]
                positive(left, ("heads", "kv_heads", "dim", "vdim"), at + ".left")
                if left["kv_heads"] > 0 and left["heads"] % left["kv_heads"]:
                    bad.append(f"{at}.left: {left['heads']} heads are no multiple of {left['kv_heads']} kv_heads")
                if left["vdim"] != left["dim"]:
                    bad.append(f"{at}.left: the values are the keys, so vdim {left['vdim']} must be dim {left['dim']}")
                mask = left.get("mask")
                if mask is not None and (mask["size"] <= 0 or mask.get("pool", 1) <= 0):
                    bad.append(f"{at}.left.mask: size and pool must be positive, found {mask}")
                rot = left.get("rot")
                if rot is not None:
                    if rot["dims"] % 2 or not 0 <= rot["dims"] <= left["dim"] or rot["base"] <= 0:
                        bad.append(f"{at}.left.rot: dims {rot['dims']} must be even and at most dim {left['dim']}, the base positive")
                    sc = rot.get("scaling")
                    if sc is not None and not (sc["factor"] > 0 and sc["original"] > 0 and 0 < sc["low"] <= sc["high"]):
                        bad.append(f"{at}.left.rot.scaling: factor and original must be positive and 0 < low <= high, found {sc}")
                positive(right, ("heads", "dim", "vdim", "gate_cap"), at + ".right")
            else:
                positive(m, ("heads", "dim"), at)
                if m.get("rank", 1) <= 0:
                    bad.append(f"{at}.rank must be positive, found {m['rank']}")
            if layer["mlp"] is not None and layer["mlp"]["ff"] <= 0:
                bad.append(f"layers[{i}].mlp.ff must be positive")
        if bad:
            raise ConfigError("config: " + "; ".join(bad))

    @staticmethod
    def thin_rank(m: dict) -> int:
        """The inner size of the decay's two thin products when no file says otherwise (random models): an eighth of
        the heads' width, at least 8, a multiple of 8."""
        return max(8, (m["heads"] * m["dim"] // 8 + 7) // 8 * 8)

    def with_shapes(self, shapes: dict) -> "NezolornConfig":
        """The same configuration with the sizes that only the tensors give (the inner size of the decay's thin
        products, from `l<i>.mix.w1`) taken from `shapes` {tensor name: shape}."""
        out = copy.deepcopy(self)
        for i, layer in enumerate(out.layers):
            if layer["type"] == "general_delta" and f"l{i}.mix.w1" in shapes:
                layer["mixer"]["rank"] = int(shapes[f"l{i}.mix.w1"][0])
        out.validate()
        return out

    # ---- the plan ----------------------------------------------------------------
    def _mixer_spec(self, i: int, layer: dict):
        m, p, w = layer["mixer"], f"l{i}.mix.", self.width
        if layer["type"] == "general_delta":
            params = dict(hidden_size=w, n_heads=m["heads"], head_dim=m["dim"], decay_rank=m.get("rank", self.thin_rank(m)),
                          eps=self.norm_eps, unit_eps=UNIT_EPS)
            names = ("r", "k", "v", "g", "a", "a.b", "w1", "w2", "w0", "norm", "o")
            return PartSpec("general_delta_rule", params, {n: p + n for n in names}), None
        a, b = m["left"], m["right"]
        left = dict(hidden_size=w, n_heads=a["heads"], n_kv_heads=a["kv_heads"], key_dim=a["dim"], value_dim=a["vdim"],
                    softmax_scale=a["scale"], values_from_keys=True, mask={"kind": "causal"})
        if a.get("mask") is not None:
            left["mask"] = {"kind": "window", **a["mask"]}
        right = dict(hidden_size=w, n_heads=b["heads"], key_dim=b["dim"], value_dim=b["vdim"], gate_cap=b["gate_cap"],
                     eps=self.norm_eps)
        names = ["left." + n for n in ("q", "k", "o")] + \
                ["right." + n for n in ("q", "k", "v", "g", "i", "i.b", "f", "f.b", "norm", "o")]
        params = dict(left={"kind": "masked_attention", "params": left}, right={"kind": "matrix_memory", "params": right},
                      left_scale=m["left_scale"], right_scale=m["right_scale"])
        rot, rp = a.get("rot"), None
        if rot is not None and rot["dims"]:
            rp = dict(head_dim=a["dim"], rotary_dim=rot["dims"], theta=rot["base"],
                      max_positions=self.max_position_embeddings, layout="half", tables=False)
            if rot.get("scaling") is not None:
                rp["bands"] = dict(rot["scaling"])
        return PartSpec("parallel_mixers", params, {n: p + n for n in names}), rp

    def plan(self) -> ModelPlan:
        w = self.width
        norm = lambda name: PartSpec("layer_norm", dict(size=w, eps=self.norm_eps), dict(weight=name))
        mult = PartSpec("constant_scale", dict(hidden_size=w, value=self.residual_mult))
        specs, positions, schedule = [], {}, []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            mixer, rot = self._mixer_spec(i, layer)
            position = None
            if rot is not None:
                position = "rotary:" + json.dumps(rot, sort_keys=True)
                positions.setdefault(position, PartSpec("rotary", rot))
            norms, gates, ff = {"input": norm(p + "norm1")}, {"mixer": mult}, None
            if layer["mlp"] is not None:
                norms["post_mixer"], gates["ff"] = norm(p + "norm2"), mult
                ff = PartSpec("glu_mlp", dict(hidden_size=w, intermediate_size=layer["mlp"]["ff"], activation="silu"),
                              {n: p + "mlp." + n for n in ("gate", "up", "down")})
            specs.append(LayerSpec("pre_norm_scaled_residual", mixer, ff, norms, position, gates))
            schedule.append(ScheduleEntry(layer=i, cache=i))
        emb, emb_names = dict(vocab_size=self.vocab, hidden_size=w, scale=self.embedding_scale), dict(weight="embed")
        if self.bigram is not None:
            emb["pairs"], emb_names["pairs"] = dict(self.bigram), "bigram"
        return ModelPlan(
            architecture=ARCHITECTURE, hidden_size=w, vocab_size=self.vocab,
            max_positions=self.max_position_embeddings,
            embedding=PartSpec("token_embedding", emb, emb_names),
            positions=positions, layers=tuple(specs), schedule=tuple(schedule),
            final_norm=norm("final.norm"),
            head=PartSpec("linear_head", dict(hidden_size=w, vocab_size=self.vocab), dict(weight="head")))
