"""Two mixers side by side on the same input (spec: ``ParallelMixersSpec``):

    y = factor (RMSnorm(left(h)) w_left + RMSnorm(right(h)) w_right)

or, with ``branch_norms`` False,

    y = left_factor left(h) + right_factor right(h).

Both branches are mixers of the registry, built from their own specs under
``<prefix>.<left_name>`` and ``<prefix>.<right_name>``.  With norms each returns its projected result in
float32 and one kernel norms both over the model width and adds them.  Without norms the sum is linear in
what the branches' last products read, so both first products are one product and both last products are
one: the matrices are concatenated at load, each branch works on its columns of the two rows and
multiplies its own by its factor (``splits_projections``, see ``parts/base.py``).  Between the two products
the branches have nothing to do with one another: in a captured step the right one runs on a stream of
its own, so that two chains of short kernels run side by side.

What the branches ask of the cache is merged into one request of this mixer: pages from the one
branch that wants pages (two paged branches would need two block tables a layer, which is not
built), and ONE per-request state record that holds the branches' records side by side.  Each
branch sees its own slice of the record through a ``LayerCache`` of its own (the rows of a slice
are the whole record's length apart, which the kernels that index state take as a stride).
"""

from __future__ import annotations

import torch

from ..cache.manager import FixedStateRequest, paged_part, record_floats
from ..ops import kernels as K
from ..ops.linear import linear
from ..weights.source import NORM, TensorDecl
from .base import LayerCache, Mixer
from .registry import MIXERS, build_part, part_class, register_mixer


overlap_branches = True       # (captured steps; off: one after the other, as in steps launched one by one)
_side_streams = {}


def _side_stream(device) -> torch.cuda.Stream:
    key = torch.device(device)
    if key not in _side_streams:
        _side_streams[key] = torch.cuda.Stream(device=key)
    return _side_streams[key]


def _record_sizes(spec):
    """Floats of each branch's state record, rounded up to 4 (16-byte aligned slices)."""
    return [record_floats(part_class(MIXERS, b).cache_request(b)) for b in (spec.left, spec.right)]


@register_mixer("parallel_mixers")
class ParallelMixers(Mixer):
    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        self.left = build_part(MIXERS, spec.left, f"{prefix}.{spec.left_name}", env)
        self.right = build_part(MIXERS, spec.right, f"{prefix}.{spec.right_name}", env)
        for branch in (self.left, self.right):
            if spec.branch_norms:
                if not hasattr(branch, "out_dtype"):
                    raise ValueError(f"parallel_mixers: the mixer {branch.spec.kind!r} cannot return float32 results")
                branch.out_dtype = torch.float32
            elif not getattr(branch, "splits_projections", False):
                raise ValueError(f"parallel_mixers: without norms on the branches the mixer {branch.spec.kind!r} "
                                 "would have to split off its projections")
        self.graph_safe = all(getattr(b, "graph_safe", False) for b in (self.left, self.right))
        self.padded_steps_safe = all(getattr(b, "padded_steps_safe", False) for b in (self.left, self.right))
        self.sizes = _record_sizes(spec)

    @classmethod
    def _norm_names(cls, spec, prefix):
        return (f"{prefix}.{spec.left_name}{spec.out_suffix}", f"{prefix}.{spec.right_name}{spec.out_suffix}")

    @classmethod
    def declare(cls, spec, prefix):
        out = []
        for branch, name in ((spec.left, spec.left_name), (spec.right, spec.right_name)):
            out += part_class(MIXERS, branch).declare(branch, f"{prefix}.{name}")
        if not spec.branch_norms:
            return out
        return out + [TensorDecl(n, (spec.hidden_size,), NORM) for n in cls._norm_names(spec, prefix)]

    @classmethod
    def cache_request(cls, spec):
        requests = [part_class(MIXERS, b).cache_request(b) for b in (spec.left, spec.right)]
        pages = [p for p in (paged_part(r) for r in requests) if p is not None]
        if len(pages) > 1:
            raise ValueError("parallel_mixers: only one branch may keep pages of keys")
        total = sum(_record_sizes(spec))
        out = tuple(pages) + ((FixedStateRequest((total,)),) if total else ())
        return out[0] if len(out) == 1 else (out or None)

    def load(self, store):
        self.left.load(store)
        self.right.load(store)
        if self.spec.branch_norms:
            self.w_left, self.w_right = (store.get(n) for n in self._norm_names(self.spec, self.prefix))
        else:
            self._merge()

    def _merge(self):
        """One matrix for both first products and one for both last ones; a branch's columns of the last
        product's rows begin at a multiple of 8 (zero columns of the matrix between)."""
        left, right = self.left, self.right
        self.w_in = torch.cat([left.w_in, right.w_in]).contiguous()
        self.right_rows = left.w_in.shape[0]
        wide = [-(-b.out_width // 8) * 8 for b in (left, right)]
        self.right_at, self.row_width = wide[0], sum(wide)
        self.row_padding = self.row_width != left.out_width + right.out_width
        hidden = left.w_o.shape[0]
        w_o = torch.zeros((hidden, self.row_width), dtype=left.w_o.dtype, device=left.w_o.device)
        w_o[:, :left.out_width] = left.w_o
        w_o[:, self.right_at:self.right_at + right.out_width] = right.w_o
        self.w_o, self.o_bias = w_o, None
        for branch, factor in ((left, self.spec.left_factor), (right, self.spec.right_factor)):
            if branch.o_bias is not None:
                term = factor * branch.o_bias
                self.o_bias = term if self.o_bias is None else self.o_bias + term
            branch.w_in = branch.w_o = None
        self.o_bias_cast = None if self.o_bias is None else self.o_bias.to(self.env.dtype)
        if self.w_in.is_cuda:
            _side_stream(self.w_in.device)                 # (made now, not in a capture)

    def _branch_cache(self, cache: LayerCache, index: int) -> LayerCache:
        return cache.with_state_slice(sum(self.sizes[:index]), self.sizes[index])

    def forward(self, ctx, x, cache, owns_cache):
        if not self.spec.branch_norms:
            return self._forward_merged(ctx, x, cache, owns_cache)
        a = K.plain_unless(None, self.left.forward(ctx, x, self._branch_cache(cache, 0), owns_cache))
        b = K.plain_unless(None, self.right.forward(ctx, x, self._branch_cache(cache, 1), owns_cache))
        out = torch.empty((x.shape[0], self.spec.hidden_size), dtype=x.dtype, device=x.device)
        K.norm_sum2(a, b, self.w_left, self.w_right, self.spec.eps, self.spec.factor, out)
        return out

    def _forward_merged(self, ctx, x, cache, owns_cache):
        proj = K.plain_unless(None, linear(x, self.w_in))
        make = torch.zeros if self.row_padding else torch.empty
        row = make((x.shape[0], self.row_width), dtype=x.dtype, device=x.device)
        early = self.right.early(ctx, x)

        def left():
            self.left.core(ctx, x, proj[:, :self.right_rows], self._branch_cache(cache, 0), owns_cache,
                           row[:, :self.left.out_width], self.spec.left_factor, self.left.early(ctx, x))

        def right():
            self.right.core(ctx, x, proj[:, self.right_rows:], self._branch_cache(cache, 1), owns_cache,
                            row[:, self.right_at:self.right_at + self.right.out_width], self.spec.right_factor, early)
        if overlap_branches and torch.cuda.is_current_stream_capturing():
            main, side = torch.cuda.current_stream(), _side_stream(x.device)
            side.wait_stream(main)
            with torch.cuda.stream(side):
                right()
            left()
            main.wait_stream(side)
        else:
            left()
            right()
        return linear(row, self.w_o, self.o_bias, consumer="norm", bias_cast=self.o_bias_cast)
