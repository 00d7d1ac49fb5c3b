"""Assembling a model from a ModelSpec, and running its layers for one step.

The model is a list of layers built from registered parts, run in the order the
spec's schedule gives.  ``manifest`` collects every tensor the parts declare, which
is what a checkpoint is checked against and what the random-weights mode draws.
The forward pass is the reference's (src/model.cu:859-1039): embedding, then per
scheduled layer its arrangement, then the final norm and the head — but only on the
rows whose logits are wanted.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Optional, Set, Tuple

import torch

from ..cache import KVRequest
from ..config.spec import BranchSpec, ModelSpec, PartSpec
from ..parts.base import LayerCache, Part, StepContext, build_part, lookup_part
from ..weights.loader import WeightSpec


@dataclass
class Branch:
    """One built residual branch of a layer: ``h += post_norm(part(norm(h)))``."""

    role: str                      # "mixer" or "feed_forward"
    part: Part
    norm: Optional[Part] = None
    post_norm: Optional[Part] = None
    shift: Optional[Part] = None   # between the norm and the part
    scale: float = 1.0             # factor on what the branch adds to the stream

    def parts(self) -> List[Part]:
        return [p for p in (self.norm, self.shift, self.part, self.post_norm) if p is not None]


@dataclass
class Layer:
    prefix: str
    branches: List[Branch]
    run: Callable


def _with(spec: PartSpec, **extra) -> PartSpec:
    return PartSpec(spec.kind, {**spec.params, **extra})


def _branch_specs(bs: BranchSpec):
    """(category, PartSpec) of a branch's parts, in the order they are built and loaded."""
    if bs.norm is not None:
        yield "norm", bs.norm
    if bs.shift is not None:
        yield "shift", bs.shift
    yield bs.role, bs.part
    if bs.post_norm is not None:
        yield "norm", bs.post_norm


def _full_name(prefix: str, name: str) -> str:
    """A tensor's full name: behind the layer's prefix, or without it when the name begins with "/"."""
    return name[1:] if name.startswith("/") else prefix + name


def _part_specs(spec: ModelSpec):
    """Every (category, PartSpec, name prefix) of the model, in a fixed order."""
    yield "embedding", _with(spec.embedding, vocab_size=spec.vocab_size), ""
    if spec.merge is not None:
        yield "merge", spec.merge, ""
    for layer in spec.layers:
        for bs in layer.branches:
            for category, pspec in _branch_specs(bs):
                yield category, pspec, layer.prefix
    yield "norm", spec.final_norm, ""
    yield "head", _with(spec.head, vocab_size=spec.vocab_size), ""


def manifest(spec: ModelSpec) -> Tuple[Dict[str, WeightSpec], Set[str]]:
    """All tensors of the model by full name, and names a file may hold unused."""
    out: Dict[str, WeightSpec] = {}
    for category, pspec, prefix in _part_specs(spec):
        cls = lookup_part(category, pspec.kind)
        for _, (name, wspec) in cls.weight_specs(pspec.params, spec.hidden_size).items():
            full = _full_name(prefix, name)
            if full in out and out[full] != wspec:
                raise ValueError(f"tensor {full!r} is declared twice with different shapes")
            out[full] = wspec
    ignorable: Set[str] = set()
    if spec.head.params.get("tied") and spec.head.params.get("name"):
        ignorable.add(spec.head.params["name"])
    return out, ignorable


class Model:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device):
        spec.validate()
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"the compute dtype must be float32 or bfloat16, got {dtype}")
        self.spec, self.dtype, self.device = spec, dtype, torch.device(device)
        H = spec.hidden_size
        # every part is built in the order of _part_specs, which is also the order of loading
        built = [build_part(category, pspec, H, dtype, device)
                 for category, pspec, _ in _part_specs(spec)]
        self._parts: List[Part] = built
        it = iter(built)
        self.embedding = next(it)
        self.merge = next(it) if spec.merge is not None else None
        self.layers: List[Layer] = []
        for ls in spec.layers:
            branches = []
            for bs in ls.branches:
                norm = next(it) if bs.norm is not None else None
                shift = next(it) if bs.shift is not None else None
                part = next(it)
                post = next(it) if bs.post_norm is not None else None
                branches.append(Branch(bs.role, part, norm, post, shift, float(bs.scale)))
            self.layers.append(Layer(ls.prefix, branches,
                                     lookup_part("arrangement", ls.arrangement)))
        self.final_norm = next(it)
        self.head = next(it)

    def parts(self) -> List[Part]:
        """Every part of the model: embedding, merge (if any), each layer's branches in order, final norm, head."""
        return list(self._parts)

    @property
    def graph_safe(self) -> bool:
        """Whether every part allows its steps to be captured as CUDA graphs."""
        return all(getattr(p, "graph_safe", False) for p in self._parts)

    # -- weights ---------------------------------------------------------------
    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Hand each part its tensors (CPU, by full name) and let it place them."""
        for part, (category, pspec, prefix) in zip(self._parts, _part_specs(self.spec)):
            specs = lookup_part(category, pspec.kind).weight_specs(pspec.params,
                                                                   self.spec.hidden_size)
            part.load({key: tensors[_full_name(prefix, name)] for key, (name, _) in specs.items()})
        if self.spec.head.params.get("tied"):
            self.head.tie(self.embedding)

    def prepare(self, max_positions: int) -> None:
        """Let every part build what depends on the longest sequence (position tables)."""
        for part in self._parts:
            if hasattr(part, "prepare"):
                part.prepare(max_positions)

    # -- cache -------------------------------------------------------------------
    def cache_requests(self) -> Dict[Tuple, Any]:
        """cache id → what its part keeps between steps.  A cache id is (index of the schedule
        entry, index of the branch in its layer) for the branch's part and (entry, branch,
        "shift") for a shift in front of it; a mixer made of several (``sub_mixers``) keeps one for
        each, (entry, branch, its name).  A part may ask for keys and values, for a state of
        fixed size, or for both (a tuple).  An entry that borrows (``ScheduleEntry.cache``) reads
        the owner's keys and values and asks for none; states are always an entry's own."""
        out = {}
        for i, entry in enumerate(self.spec.schedule):
            for k, br in enumerate(self.layers[entry.layer].branches):
                for cid, part in self._keepers(i, k, br.part):
                    if not hasattr(part, "cache_request"):
                        continue
                    reqs = part.cache_request()
                    reqs = list(reqs) if isinstance(reqs, (tuple, list)) else [reqs]
                    reqs = [r for r in reqs if r is not None
                            and not (entry.cache is not None and isinstance(r, KVRequest))]
                    if reqs:
                        out[cid] = reqs[0] if len(reqs) == 1 else tuple(reqs)
                if br.shift is not None:
                    out[(i, k, "shift")] = br.shift.cache_request()
        return out

    @staticmethod
    def _keepers(i: int, k: int, part):
        """(cache id, part) of everything that keeps something in branch k of entry i."""
        if hasattr(part, "sub_mixers"):
            return [((i, k, name), sub) for name, sub in part.sub_mixers()]
        return [((i, k), part)]

    def layer_caches(self, i: int, cache) -> List[Optional[LayerCache]]:
        """What each branch of schedule entry ``i`` is handed: its own keys/values or those of
        the entry it borrows from (read-only), its own states, or None for a branch that keeps
        nothing."""
        entry = self.spec.schedule[i]
        owner = i if entry.cache is None else entry.cache
        views: List[Optional[LayerCache]] = []
        for k, br in enumerate(self.layers[entry.layer].branches):
            cid = (owner, k)
            if entry.cache is not None and br.role == "mixer":
                # the k-th mixer of this layer reads the k-th mixer's cache of the owner's layer
                mine = [j for j, b in enumerate(self.layers[entry.layer].branches)
                        if b.role == "mixer"]
                theirs = [j for j, b in enumerate(
                    self.layers[self.spec.schedule[owner].layer].branches) if b.role == "mixer"]
                cid = (owner, theirs[mine.index(k)])
            shift = cache.state_view((i, k, "shift")) if cache.has_state((i, k, "shift")) else None

            def view(tail=(), shift=None):
                kv = cache.kv_view(cid + tail) if cache.has_kv(cid + tail) else None
                own = (i, k) + tail
                state = cache.state_view(own) if cache.has_state(own) else None
                return None if kv is None and state is None and shift is None else LayerCache(
                    kv=kv, state=state, writes=entry.cache is None, shift_state=shift)
            if hasattr(br.part, "sub_mixers"):
                views.append(LayerCache(writes=entry.cache is None, shift_state=shift, subs={
                    name: view((name,)) for name, _ in br.part.sub_mixers()}))
            else:
                views.append(view(shift=shift))
        return views

    def _reads_stream(self, i: int) -> bool:
        """Whether schedule entry ``i`` begins with a branch that reads the stream itself (no norm in
        front of it), so that a copy in the compute type is worth leaving."""
        if i >= len(self.spec.schedule):
            return False
        entry = self.spec.schedule[i]
        first = self.layers[entry.layer].branches[0]
        return first.norm is None and first.shift is None and not (entry.add_input
                                                                   or entry.merge_input)

    # -- one step ------------------------------------------------------------------
    def forward(self, ctx: StepContext, cache, want_rows: Optional[torch.Tensor]) -> torch.Tensor:
        """Run the scheduled layers on the step's tokens; logits [rows, vocab] float32
        at ``want_rows`` (token indices), or at every token when it is None."""
        from ..csrc import ops
        h = self.embedding.forward(ctx.tok_ids, ctx)
        # a schedule entry may ask for the model's input to be added again (a further pass
        # over a span of layers): the embedding's output is kept for it
        h_in = h.clone() if any(e.add_input for e in self.spec.schedule) else None
        merging = any(e.merge_input for e in self.spec.schedule)
        merge_rows = self.merge.begin(h) if merging else None
        streams = ctx.extras.get("streams")      # a list: the stream after every layer run
        pending = None
        for i, entry in enumerate(self.spec.schedule):
            layer = self.layers[entry.layer]
            if entry.add_input or entry.merge_input:
                if pending is not None:
                    ops.axpy_rows(h, pending.contiguous(), 1.0)
                    pending = None
                ctx.extras.pop("stream_copy", None)
                if entry.add_input:
                    ops.axpy_rows(h, h_in, 1.0)
                if entry.merge_input:
                    self.merge.forward(h, merge_rows)
            ctx.extras["copy_wanted"] = self._reads_stream(i + 1)
            pending = layer.run(layer, h, pending, ctx, self.layer_caches(i, cache))
            if streams is not None:
                streams.append(h.clone() if pending is None else h + pending.to(h.dtype))
        if want_rows is not None and want_rows.numel() == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=h.device)
        if hasattr(self.head, "forward_from_residual"):
            logits = self.head.forward_from_residual(h, pending, self.final_norm, want_rows, ctx)
            if logits is not None:
                return logits
        n = self.final_norm.forward(h, pending, rows=want_rows, write_h=False)
        return self.head.forward(n, ctx)

    def weight_bytes(self) -> int:
        return sum(p.weight_bytes() for p in self._parts)
