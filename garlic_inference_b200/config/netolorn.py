"""Typed configuration of the Netolorn decoder.

A Netolorn config.json names its model class as the string `architecture` and
gives `vocab`, `width`, `norm.eps`, a list `layers` and, optionally, `loop` and
`token_side`; every layer entry has a `type` (which mixer), the mixer's sizes
and constants under `mixer` and a feed-forward under `mlp` (or null).  An
unknown mixer or feed-forward kind is refused by name; a key outside the design
is ignored with a warning.

    x = x0 = E[token]
    x += n1b(mixer(n1(x)));   x += n2b(ff(n2(x)))         n(z) = tanh(alpha z) w + b, one number alpha per norm
    x += rms( P( gelu_tanh(G x) * S[token, i dim : (i + 1) dim] ) ) w_side          layer i's own columns of one table
    logits = head n_final(x)

`loop` = {start, stop, times}: the layers start .. stop - 1 run `times` times in
a row with the same weights and a cache entry of their own each time; right
before every pass, the first too, x <- W_in [x; x0] (tensor `loop.in`).

Mixers.  `attention`: grouped-query attention with biases on q, k, v, a rotation
of halves (i, i + dims/2) of the first `rot.dims` dimensions with YaRN scaling,
q and k divided by their root mean square per head after it, a window of
`mask.size` tokens beside which the first `mask.keep_first` stay in sight, a
learned sink per head in the softmax's denominator, and a sigmoid gate per
output element.  `latent_attention`: queries through a normed latent of
`q_rank`, keys and values expanded from a normed latent of `kv_rank`, no
positions, a window of `mask.size` tokens, a sigmoid gate per head.
Feed-forwards.  `dense`: down(silu(gate x) * (up x)).  `moe`: `top` of `experts`
gated experts g sigmoid(1.702 g) (u + 1) with g = min(gate x, limit), u =
clamp(up x, -limit, limit); the largest biased logits choose, their softmax is
the weights; a `shared` expert for every token, times sigmoid(Wsg x).

The design gives no limit on positions; `MAX_POSITIONS` is this library's
(positions are int32 on the device and are turned into float32 angles).
"""
from __future__ import annotations

import copy
import json
import warnings
from dataclasses import dataclass, field
from typing import Optional

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, ScheduleEntry, optional, require

ARCHITECTURE = "Netolorn"
MAX_POSITIONS = 1 << 22
SWISH_ALPHA = 1.702        # inside the sigmoid of the experts' activation: fixed by the design
UP_SHIFT = 1.0             # added to the clamped up half: fixed by the design

_HEADS = {"heads": int, "dim": int, "vdim": int, "scale": float}
_YARN = {"factor": float, "original": float, "fast": float, "slow": float}


def _typed(d, keys: dict, where: str, optional_keys: tuple = ()) -> dict:
    """The listed keys of `d`, each of its type.  A key this library does not know is left out with a warning."""
    if not isinstance(d, dict):
        raise ConfigError(f"{where}: must be an object, found {d!r}")
    unknown = sorted(set(d) - set(keys) - set(optional_keys))
    if unknown:
        warnings.warn(f"{where}: keys {unknown} are not part of the design and are ignored", stacklevel=3)
    return {k: require(d, k, typ, where) for k, typ in keys.items()}


def _mixer(typ: str, m, w: str) -> dict:
    if typ == "attention":
        out = _typed(m, dict(_HEADS, kv_heads=int), w, optional_keys=("mask", "rot"))
        if m.get("mask") is not None:
            out["mask"] = _typed(m["mask"], {"size": int}, w + ".mask", optional_keys=("keep_first",))
            out["mask"]["keep_first"] = optional(m["mask"], "keep_first", int, 0, w + ".mask")
        if m.get("rot") is not None:
            out["rot"] = _typed(m["rot"], {"base": float, "dims": int}, w + ".rot", optional_keys=("scaling",))
            if m["rot"].get("scaling") is not None:
                out["rot"]["scaling"] = _typed(m["rot"]["scaling"], _YARN, w + ".rot.scaling")
        return out
    if typ == "latent_attention":
        out = _typed(m, dict(_HEADS, kv_rank=int, q_rank=int), w, optional_keys=("mask",))
        if m.get("mask") is not None:
            out["mask"] = _typed(m["mask"], {"size": int}, w + ".mask")
        return out
    raise ConfigError(f"{w[:-6]}: mixer type {typ!r} is neither 'attention' nor 'latent_attention'")


def _mlp(mlp, w: str):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{w}: must be an object or null, found {mlp!r}")
    kind = require(mlp, "kind", str, w)
    if kind == "dense":
        return _typed(mlp, {"kind": str, "ff": int}, w)
    if kind != "moe":
        raise ConfigError(f"{w}: kind {kind!r} is neither 'dense' nor 'moe'")
    out = _typed(mlp, {"kind": str}, w, optional_keys=("expert", "router", "shared"))
    out["expert"] = _typed(mlp.get("expert"), {"ff": int, "limit": float}, w + ".expert")
    out["router"] = _typed(mlp.get("router"), {"experts": int, "top": int}, w + ".router")
    if mlp.get("shared") is not None:
        out["shared"] = _typed(mlp["shared"], {"ff": int, "limit": float}, w + ".shared")
    return out


@dataclass
class NetolornConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: list = field(default_factory=list)      # the entries of config.json's `layers`, checked
    loop: Optional[dict] = None                     # {start, stop, times} or None
    side_dim: Optional[int] = None                  # token_side.dim, or None: no per-token input
    max_position_embeddings: int = MAX_POSITIONS    # not a key of the design: this library's own limit

    def __post_init__(self):
        self.validate()

    # ---- reading and writing -------------------------------------------------
    @classmethod
    def from_dict(cls, cfg: dict, where: str = "config.json") -> "NetolornConfig":
        norm = cfg.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError(f"{where}: key 'norm' must be an object with 'eps'")
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
        loop = None
        if cfg.get("loop") is not None:
            loop = _typed(cfg["loop"], {"start": int, "stop": int, "times": int}, where + ": loop")
        side = None
        if cfg.get("token_side") is not None:
            side = _typed(cfg["token_side"], {"dim": int}, where + ": token_side")["dim"]
        return cls(vocab=require(cfg, "vocab", int, where), width=require(cfg, "width", int, where),
                   norm_eps=require(norm, "eps", float, where + ": norm"), layers=layers, loop=loop, side_dim=side)

    def to_dict(self) -> dict:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": copy.deepcopy(self.layers)}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        if self.side_dim is not None:
            out["token_side"] = {"dim": self.side_dim}
        return out

    # ---- checks ----------------------------------------------------------------
    def validate(self) -> None:
        bad = []
        if self.vocab <= 0 or self.width <= 0:
            bad.append("vocab and width must be positive")
        if not self.norm_eps > 0:
            bad.append(f"norm.eps must be positive, found {self.norm_eps}")
        if not self.layers:
            bad.append("'layers' is empty")
        if self.side_dim is not None and self.side_dim <= 0:
            bad.append(f"token_side.dim must be positive, found {self.side_dim}")
        if self.loop is not None:
            lp = self.loop
            if not (0 <= lp["start"] <= lp["stop"] <= len(self.layers)) or lp["times"] < 1:
                bad.append(f"loop {lp} does not fit {len(self.layers)} layers (0 <= start <= stop <= layers, times >= 1)")

        def positive(m, keys, at):
            bad.extend(f"{at}.{k} must be positive, found {m[k]}" for k in keys if m[k] <= 0)

        for i, layer in enumerate(self.layers):
            m, at = layer["mixer"], f"layers[{i}].mixer"
            positive(m, ("heads", "dim", "vdim"), at)
            if m.get("mask") is not None and (m["mask"]["size"] <= 0 or m["mask"].get("keep_first", 0) < 0):
                bad.append(f"{at}.mask: size must be positive and keep_first not negative, found {m['mask']}")
            if layer["type"] == "latent_attention":
                positive(m, ("kv_rank", "q_rank"), at)
            else:
                positive(m, ("kv_heads",), at)
                if m["kv_heads"] > 0 and m["heads"] % m["kv_heads"]:
                    bad.append(f"{at}: {m['heads']} heads are no multiple of {m['kv_heads']} kv_heads")
                rot = m.get("rot")
                if rot is not None:
                    if rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"] or rot["base"] <= 0:
                        bad.append(f"{at}.rot: dims {rot['dims']} must be even and at most dim {m['dim']}, the base positive")
                    sc = rot.get("scaling")
                    if sc is not None and (min(sc.values()) <= 0 or rot["base"] == 1):
                        bad.append(f"{at}.rot.scaling: factor, original, fast and slow must be positive and the base not 1, found {sc}")
            mlp, at = layer["mlp"], f"layers[{i}].mlp"
            if mlp is not None and mlp["kind"] == "moe":
                r = mlp["router"]
                positive(mlp["expert"], ("ff",), at + ".expert")
                if r["experts"] <= 0 or not 0 < r["top"] <= r["experts"]:
                    bad.append(f"{at}.router: top {r['top']} of {r['experts']} experts")
                if mlp.get("shared") is not None:
                    positive(mlp["shared"], ("ff",), at + ".shared")
            elif mlp is not None:
                positive(mlp, ("ff",), at)
        if bad:
            raise ConfigError("config: " + "; ".join(bad))

    # ---- the plan ----------------------------------------------------------------
    def layer_runs(self) -> list:
        """[(layer, pass or None)] in the order the layers run: the layers before the loop, the looped layers pass
        by pass, the rest."""
        n, lp = len(self.layers), self.loop
        if lp is None or lp["stop"] <= lp["start"]:
            return [(i, None) for i in range(n)]
        runs = [(i, None) for i in range(lp["start"])]
        for t in range(lp["times"]):
            runs += [(i, t) for i in range(lp["start"], lp["stop"])]
        return runs + [(i, None) for i in range(lp["stop"], n)]

    def _unit(self, limit: float) -> dict:
        return dict(activation="swish", swish_alpha=SWISH_ALPHA, gate_max=limit, up_limit=limit, up_shift=UP_SHIFT)

    def _mixer_spec(self, i: int, layer: dict):
        m, p, w = layer["mixer"], f"l{i}.mix.", self.width
        mask = m.get("mask")
        if layer["type"] == "latent_attention":
            params = dict(hidden_size=w, n_heads=m["heads"], plain_dim=m["dim"], rot_dim=0, value_dim=m["vdim"],
                          kv_rank=m["kv_rank"], q_rank=m["q_rank"], softmax_scale=m["scale"], eps=self.norm_eps, head_gate=True)
            if mask is not None:
                params["window"] = mask["size"]
            names = ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "g", "o")
            return PartSpec("latent_attention", params, {n: p + n for n in names}), None
        params = dict(hidden_size=w, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                      softmax_scale=m["scale"], qkv_bias=True, head_norm_eps=self.norm_eps, learned_sink=True,
                      output_gate=True, mask={"kind": "causal"})
        if mask is not None:
            params["mask"] = {"kind": "window", **mask}
        rot, rp = m.get("rot"), None
        if rot is not None and rot["dims"]:
            rp = dict(head_dim=m["dim"], rotary_dim=rot["dims"], theta=rot["base"],
                      max_positions=self.max_position_embeddings, layout="half", tables=False)
            if rot.get("scaling") is not None:
                rp["yarn"] = dict(rot["scaling"])
        names = ("q", "k", "v", "q.b", "k.b", "v.b", "sink", "g", "o")
        return PartSpec("masked_attention", params, {n: p + n for n in names}), rp

    def _ff_spec(self, i: int, mlp):
        if mlp is None:
            return None
        p, w = f"l{i}.mlp.", self.width
        if mlp["kind"] == "dense":
            return PartSpec("glu_mlp", dict(hidden_size=w, intermediate_size=mlp["ff"], activation="silu"),
                            {n: p + n for n in ("gate", "up", "down")})
        r = mlp["router"]
        names = ["router", "router.b"] + [f"e{e}.{n}" for e in range(r["experts"]) for n in ("gate", "up", "down")]
        params = dict(hidden_size=w, expert_size=mlp["expert"]["ff"], n_experts=r["experts"], top=r["top"], expert="glu",
                      **self._unit(mlp["expert"]["limit"]), scores="softmax_chosen", router_bias=True)
        if mlp.get("shared") is not None:
            params["shared"] = dict(size=mlp["shared"]["ff"], gate=True, **self._unit(mlp["shared"]["limit"]))
            names += ["shared.gate", "shared.up", "shared.down", "shared.sg"]
        return PartSpec("routed_experts", params, {n: p + n for n in names})

    def plan(self) -> ModelPlan:
        w = self.width
        norm = lambda name: PartSpec("dyt_norm", dict(size=w), dict(weight=name, bias=name + ".b", alpha=name + ".alpha"))
        specs, positions = [], {}
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            mixer, rot = self._mixer_spec(i, layer)
            position = None
            if rot is not None:
                position = "rotary:" + json.dumps(rot, sort_keys=True)
                positions.setdefault(position, PartSpec("rotary", rot))
            ff = self._ff_spec(i, layer["mlp"])
            norms = {"input": norm(p + "norm1"), "mixer_out": norm(p + "norm1b")}
            if ff is not None:
                norms.update(post_mixer=norm(p + "norm2"), ff_out=norm(p + "norm2b"))
            side = None
            if self.side_dim is not None:
                side = PartSpec("token_side", dict(hidden_size=w, vocab_size=self.vocab, dim=self.side_dim,
                                                   columns=self.side_dim * len(self.layers), offset=i * self.side_dim,
                                                   eps=self.norm_eps),
                                dict(table="side.embed", gate=p + "side.gate", proj=p + "side.proj", norm=p + "side.norm"))
            specs.append(LayerSpec("sandwich_residual", mixer, ff, norms, position, side=side))
        # every run of a layer has a cache entry of its own; the stream is mixed with the embedding's output before each pass
        runs, mixes = self.layer_runs(), {}
        if any(t is not None for _, t in runs):
            mixes["loop.in"] = PartSpec("stream_mix", dict(hidden_size=w), dict(weight="loop.in"))
        schedule = [ScheduleEntry(layer=i, cache=entry,
                                  mix="loop.in" if t is not None and i == self.loop["start"] else None)
                    for entry, (i, t) in enumerate(runs)]
        return ModelPlan(
            architecture=ARCHITECTURE, hidden_size=w, vocab_size=self.vocab,
            max_positions=self.max_position_embeddings,
            embedding=PartSpec("token_embedding", dict(vocab_size=self.vocab, hidden_size=w), dict(weight="embed")),
            positions=positions, layers=tuple(specs), schedule=tuple(schedule),
            final_norm=norm("final.norm"),
            head=PartSpec("linear_head", dict(hidden_size=w, vocab_size=self.vocab), dict(weight="head")), mixes=mixes)
