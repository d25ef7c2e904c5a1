"""A decoder built from a `ModelPlan`: embedding, blocks run in the order the
schedule lists, final norm, head.

Upstream's model class owns its tensors by field and runs its layers in a
fixed loop (src/models/qwen3/qwen3.h:77-93, qwen3.cpp:292-303).  Here the
model is data: which parts, with which sizes, in which order, reading which
cache entry.  `wanted_tensors(plan)` lists every checkpoint tensor the plan
needs with its shape, which is also what random initialisation writes.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.base import ModelPlan, PartSpec
from ..parts import Part, Runtime, StepContext, part_class, settle_normed
from ..weights.loader import TensorWant, WeightError, device_dtype


def _part_wants(spec: PartSpec) -> dict[str, TensorWant]:
    cls = part_class(spec.kind)
    local = cls.wanted(spec.params)
    missing = [n for n in local if n not in spec.weights]
    if missing:
        raise WeightError(f"part '{spec.kind}' wants tensors {missing} that its plan entry does not name")
    return {spec.weights[n]: w for n, w in local.items()}


def plan_part_specs(plan: ModelPlan) -> list[PartSpec]:
    specs = [plan.embedding, *plan.positions.values(), *plan.offsets.values(), *plan.mixes.values()]
    for layer in plan.layers:
        specs += [layer.mixer, *([layer.feed_forward] if layer.feed_forward is not None else []),
                  *layer.norms.values(), *layer.gates.values(), *([layer.side] if layer.side is not None else [])]
    return specs + [plan.final_norm, plan.head]


def wanted_tensors(plan: ModelPlan) -> dict[str, TensorWant]:
    """Checkpoint name -> shape and role, for every tensor the plan's parts load."""
    out: dict[str, TensorWant] = {}
    for spec in plan_part_specs(plan):
        for name, want in _part_wants(spec).items():
            if name in out and tuple(out[name].shape) != tuple(want.shape):
                raise WeightError(f"tensor '{name}' is wanted with shapes {list(out[name].shape)} and "
                                  f"{list(want.shape)} by two parts")
            out.setdefault(name, want)
    return out


class _PartLoader:
    """What a part's constructor calls to get its tensors onto the device."""

    def __init__(self, spec: PartSpec, source, rt: Runtime, shared: dict):
        self.spec, self.source, self.rt, self.shared = spec, source, rt, shared

    def dtype(self, *locals_: str) -> torch.dtype:
        """The type in which the named tensor is kept on the device; for several names (tensors packed into
        one) the widest of theirs, so that a tensor stored in 32 bits is never narrowed by its neighbours."""
        kept = [device_dtype(self.source.stored_dtype(self.spec.weights[n]), self.rt.dtype) for n in locals_]
        return torch.float32 if torch.float32 in kept else kept[0]

    def __call__(self, local: str, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        name = self.spec.weights[local]
        if out is not None:
            out.copy_(self.source.tensor(name))
            return out
        if name not in self.shared:                 # a tensor named by two parts is loaded once
            self.shared[name] = self.source.tensor(name).to(device=self.rt.device, dtype=self.dtype(local)).contiguous()
        return self.shared[name]


class DecoderModel:
    def __init__(self, plan: ModelPlan, source, rt: Runtime):
        self.plan, self.rt = plan, rt
        shared: dict[str, torch.Tensor] = {}

        def make(spec: PartSpec):
            return part_class(spec.kind)(spec.params, _PartLoader(spec, source, rt, shared), rt)

        self.embedding = make(plan.embedding)
        self.positions = {name: make(spec) for name, spec in plan.positions.items()}
        self.offsets = {name: make(spec) for name, spec in plan.offsets.items()}
        self.mixes = {name: make(spec) for name, spec in plan.mixes.items()}
        self.blocks = []
        for i, layer in enumerate(plan.layers):
            if layer.position is not None and layer.position not in self.positions:
                raise KeyError(f"layer {i} names position encoding {layer.position!r}; the plan has "
                               f"{sorted(self.positions)}")
            block_cls = part_class(layer.block)
            extra = {"gates": {n: make(s) for n, s in layer.gates.items()}} if layer.gates else {}
            if layer.side is not None:
                extra["side"] = make(layer.side)
            self.blocks.append(block_cls(make(layer.mixer),
                                         make(layer.feed_forward) if layer.feed_forward is not None else None,
                                         {n: make(s) for n, s in layer.norms.items()},
                                         self.positions.get(layer.position), rt, **extra))
        self.final_norm = make(plan.final_norm)
        self.head = make(plan.head)
        self.schedule = tuple(plan.schedule)
        for e in self.schedule:
            if not 0 <= e.layer < len(self.blocks):
                raise IndexError(f"the schedule names layer {e.layer}; the plan has {len(self.blocks)}")
            if e.offset is not None and e.offset[0] not in self.offsets:
                raise KeyError(f"the schedule names the offset table {e.offset[0]!r}; the plan has {sorted(self.offsets)}")
            if e.mix is not None and e.mix not in self.mixes:
                raise KeyError(f"the schedule names the mix {e.mix!r}; the plan has {sorted(self.mixes)}")
        self.vocab_size, self.hidden_size, self.max_positions = plan.vocab_size, plan.hidden_size, plan.max_positions

    @property
    def graph_safe(self) -> bool:
        """True if every part allows a decode step to be recorded into a CUDA graph."""
        return all(p.graph_safe for p in (self.embedding, *self.positions.values(), *self.offsets.values(),
                                          *self.mixes.values(), *self.blocks, self.final_norm, self.head))

    def cache_requirements(self) -> list:
        """What each cache entry has to hold; entries shared by several runs must agree."""
        from ..cache import EntryRequirement, split_requirement
        reqs: list = [None] * self.plan.n_cache_entries()
        written = [False] * len(reqs)
        for e in self.schedule:
            req = self.blocks[e.layer].cache_requirement()
            if e.kv_cache is not None:
                # the run reads another entry's keys and values: they must have the shape this layer asks for, and
                # the entry of its own keeps the layer's state alone
                kv_req, state_req = split_requirement(req)
                src_kv = split_requirement(reqs[e.kv_cache])[0] if 0 <= e.kv_cache < len(reqs) else None
                if not written[e.kv_cache] or src_kv is None:
                    raise ValueError(f"the schedule reads the keys and values of cache entry {e.kv_cache} before any "
                                     "layer wrote them")
                if kv_req != src_kv:
                    raise ValueError(f"a layer reads the keys and values of cache entry {e.kv_cache} ({src_kv}) but "
                                     f"asks for {kv_req}")
                req = EntryRequirement(None, state_req) if state_req is not None else None
            if reqs[e.cache] is not None and reqs[e.cache] != req:
                raise ValueError(f"cache entry {e.cache} is used by layers with different needs: "
                                 f"{reqs[e.cache]} and {req}")
            if not e.writes_cache and not written[e.cache]:
                raise ValueError(f"the schedule reads cache entry {e.cache} before any layer wrote it")
            reqs[e.cache] = req
            written[e.cache] = written[e.cache] or e.writes_cache
        own = self.embedding.cache_requirement()
        return reqs if own is None else reqs + [own]     # behind the layers' entries

    def step_arrays(self, shape, cache) -> dict:
        """The int32 arrays the scheduled layers' parts want on the device for this step, each name made once
        ({name: numpy array}); the engine copies them with the step's own arrays."""
        out: dict = {}
        for e in self.schedule:
            for name, make in self.blocks[e.layer].step_arrays(shape, cache.view(e.cache, e.kv_cache)).items():
                if name not in out:
                    out[name] = make()
        return out

    def forward(self, ctx: StepContext, cache, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """Run the step's tokens through every scheduled layer; float32 logits [n_wanted, vocab] at
        `want_rows` (int32 row indices), or None when nothing is wanted."""
        ctx.residual_act = None                      # a context may be run again (recording a decode step)
        ctx.delta_scale = None
        ctx.delta_extra = None
        ctx.stream_offset = None
        ctx.delta_norm = None
        if self.embedding.cache_requirement() is None:
            residual = self.embedding.step(ctx)
        else:
            residual = self.embedding.step(ctx, cache.view(self.plan.n_cache_entries()))
        for pos in self.positions.values():
            pos.on_embedding(residual, ctx)
        begun = {name: mix.begin(residual) for name, mix in self.mixes.items()}      # the embedding's output, kept for them
        delta = None
        for e in self.schedule:
            if e.mix is not None:                    # a new stream; what was pending is in it
                delta, residual = None, self.mixes[e.mix].step(delta, residual, ctx, begun[e.mix])
            if e.offset is not None:                 # the block's first norm takes it along, or the block adds it
                ctx.stream_offset = self.offsets[e.offset[0]].row(e.offset[1])
            delta = self.blocks[e.layer].step(delta, residual, ctx, cache.view(e.cache, e.kv_cache),
                                              e.writes_cache and e.kv_cache is None)
            if ctx.stream_offset is not None:
                raise RuntimeError(f"block '{self.plan.layers[e.layer].block}' left the schedule's offset unapplied")
        if want_rows is None or want_rows.numel() == 0:
            return None
        scaled = {"delta_scale": ctx.delta_scale} if ctx.delta_scale is not None and delta is not None else {}
        if ctx.delta_extra is not None:
            scaled["delta2"] = ctx.delta_extra
        if ctx.delta_norm is not None and delta is not None:
            if self.final_norm.takes_delta_norm:
                scaled["delta_norm"] = ctx.delta_norm
            else:
                delta = settle_normed(delta, residual, ctx)
        normed = self.final_norm.add_norm(delta, residual, rows=want_rows, **scaled)
        return self.head.step(normed)

    def weight_bytes(self) -> int:
        """Bytes of all distinct weight tensors on the device."""
        seen, total = set(), 0
        for obj in self._all_parts():
            for v in vars(obj).values():
                if isinstance(v, torch.Tensor) and v.is_floating_point() and v.data_ptr() not in seen and v.numel():
                    seen.add(v.data_ptr())
                    total += v.numel() * v.element_size()
        return total

    def _all_parts(self):
        yield self.embedding
        yield from self.positions.values()
        yield from self.offsets.values()
        yield from self.mixes.values()
        for b in self.blocks:
            yield b                                  # an arrangement may hold a joined weight of its own
            for p in (b.mixer, b.feed_forward, getattr(b, "side", None)):
                if p is not None:
                    yield p
                    # a part put together from parts (two mixers side by side)
                    yield from (v for v in vars(p).values() if isinstance(v, Part))
            yield from (v for v in vars(b).values() if hasattr(v, "add_norm") or hasattr(v, "logits"))
        yield self.final_norm
        yield self.head
