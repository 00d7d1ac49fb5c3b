"""Mixers side by side: several mixers read the same input and their outputs are summed, each with a
factor, ``y = sum_s scale_s * mixer_s(x)``.

Where every side offers ``mix`` (what lies between its input and its output product) the sides share
both products: one input product whose columns are the sides' one after the other, then each side's
``mix`` on its columns, leaving its result in its columns of one matrix, then ONE output product over
all of them, which sums the sides in its 32-bit accumulator.  In a step of few tokens the last
side's kernels run on a stream of their own beside the others'.  The factors cost nothing: a side
takes its own as ``out_scale`` and applies it where it writes in 32-bit anyway.  Other mixers run one
after the other and their outputs are scaled and added.

What a side keeps between steps is its own: its cache id is the branch's with the side's name.
"""
from __future__ import annotations

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from .base import Part, build_part, lookup_part, register_part
from .linear import linear_few
from .side_stream import Fork, forks

_apart = False


def sides_apart(on: bool) -> None:
    """Run the sides one after the other through their own ``forward`` (tests compare both ways)."""
    global _apart
    _apart = bool(on)


@register_part("mixer", "parallel")
class ParallelMixers(Part):
    """params: ``sides``, a list of ``{"name", "kind", "params", "scale"}`` (``kind`` and ``params``
    of a registered mixer)."""

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.names = [s["name"] for s in params["sides"]]
        if not self.names or len(set(self.names)) != len(self.names):
            raise ValueError("parallel: every side needs a name of its own")
        self.scales = [float(s.get("scale", 1.0)) for s in params["sides"]]
        self.sides = [build_part("mixer", PartSpec(s["kind"], s["params"]), hidden_size, dtype, device)
                      for s in params["sides"]]
        self.together = all(getattr(p, "can_mix", False) for p in self.sides)
        if self.together:                       # a side that can mix takes its factor itself
            self.sides = [build_part("mixer", PartSpec(s["kind"], {**s["params"],
                                                                   "out_scale": scale}),
                                     hidden_size, dtype, device)
                          for s, scale in zip(params["sides"], self.scales)]
        self.graph_safe = all(getattr(p, "graph_safe", False) for p in self.sides)

    @classmethod
    def weight_specs(cls, params, hidden_size):
        out = {}
        for s in params["sides"]:
            specs = lookup_part("mixer", s["kind"]).weight_specs(s["params"], hidden_size)
            for key, spec in specs.items():
                out[f"{s['name']}.{key}"] = spec
        return out

    def load(self, tensors):
        for name, side in zip(self.names, self.sides):
            side.load({k[len(name) + 1:]: v for k, v in tensors.items()
                       if k.startswith(name + ".")})
        if not self.together:
            return
        # the stacked matrices; each side keeps its part of them as a view.  The sides' rows of the
        # input matrix are multiples of eight already, their columns of the output matrix are
        # brought to multiples of eight with zeros.
        self.w_in = torch.cat([side.w_in for side in self.sides], dim=0)
        self.rows, self.cols = [], []
        at = col = 0
        for side in self.sides:
            n = side.w_in.shape[0]
            self.rows.append((at, at + n))
            at += n
            self.cols.append((col, col + side.w_out.shape[1]))
            col += -(-side.w_out.shape[1] // 8) * 8
        self.o_dim = col
        self.padded = any(b - a != -(-(b - a) // 8) * 8 for a, b in self.cols)
        w_out = torch.zeros((self.hidden_size, col), dtype=self.dtype, device=self.device)
        for side, (a, b), (r0, r1) in zip(self.sides, self.cols, self.rows):
            w_out[:, a:b] = side.w_out
            side.w_in = self.w_in[r0:r1]
            side.w_out = w_out[:, a:b]
        self.w_out = w_out

    def prepare(self, max_positions: int) -> None:
        for side in self.sides:
            if hasattr(side, "prepare"):
                side.prepare(max_positions)

    def sub_mixers(self):
        """(name, part) of the sides, for the cache: each keeps what it asks for itself."""
        return list(zip(self.names, self.sides))

    def forward(self, x, ctx, cache):
        caches = [None if cache is None else cache.subs.get(n) for n in self.names]
        if not self.together or _apart:
            y = torch.zeros((ctx.T, self.hidden_size), dtype=torch.float32, device=x.device)
            for side, c, scale in zip(self.sides, caches, self.scales):
                ops.axpy_rows(y, side.forward(x, ctx, c).contiguous(), 1.0 if self.together else scale)
            return y
        proj = linear_few(x, self.w_in, out_dtype=torch.float32)
        make = torch.zeros if self.padded else torch.empty     # (columns of zeros stay zero)
        o = make((ctx.T, self.o_dim), dtype=self.dtype, device=x.device)
        run = [lambda s=side, c=c, r=r, k=k: s.mix(proj[:, r[0]:r[1]], ctx, c, o[:, k[0]:k[1]])
               for side, c, r, k in zip(self.sides, caches, self.rows, self.cols)]
        if forks(ctx.T):                        # few tokens: the last side beside the others
            fork = Fork(x.device)
            with fork:
                run.pop()()
            for mix in run:
                mix()
            fork.join()
        else:
            for mix in run:
                mix()
        return linear_few(o, self.w_out, out_dtype=torch.float32)

    def weight_bytes(self):
        return sum(side.weight_bytes() for side in self.sides)
