"""A mixer made of several mixers that read the same input side by side; its output is their weighted sum.

Spec parameters: `members`, a list of dicts with `kind` (a registered mixer kind), `params` (that mixer's own
parameters), `prefix` (added to the part's prefix for the member's tensors), `weight` (the factor on the
member's output, default 1) and `out_norm` {tensor, size, eps} (optional: the member's output is divided by its root mean
square over the row and multiplied by that stored vector, named under the member's prefix, before it is added).  Each
member keeps a cache or state of its own: the part's cache request is the tuple
of its members' requests and it is handed the tuple of their views.  A member that takes its factor into its own
last step (`scale_output(w) -> bool`) adds straight into the output; any other member writes into a zeroed buffer
that is added with its factor.  Members with a norm write into buffers side by side, zeroed unless the member says
(`overwrites`) that it stores its output where ctx.shared["output_empty"] is set; one kernel norms, weighs and adds
them, and leaves the rows behind the block's next norm where that works element by element (`NormedRows`).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..config.spec import PartSpec
from ..csrc import kernels as K
from ..weights.loader import TensorDecl
from .base import NormedRows, Runtime, StepContext
from .registry import MIXERS, lookup, register_mixer


def _members(spec: PartSpec) -> List[Tuple[PartSpec, type, float, Optional[dict]]]:
    out = []
    for m in spec["members"]:
        ps = PartSpec(kind=m["kind"], params=dict(m.get("params") or {}), prefix=m.get("prefix", ""))
        out.append((ps, lookup(MIXERS, ps.kind, "mixer"), float(m.get("weight", 1.0)), m.get("out_norm")))
    if not out:
        raise ValueError("side_by_side: no members")
    return out


@register_mixer("side_by_side")
class SideBySideMixer:
    ZEROED = "side_by_side_normed_zeroed"      # ctx.shared: the normed members' buffers while they are known to hold zeros

    @classmethod
    def tensors(cls, spec: PartSpec) -> Dict[str, TensorDecl]:
        t: Dict[str, TensorDecl] = {}
        for ps, mcls, _, norm in _members(spec):
            own = dict(mcls.tensors(ps))
            if norm is not None:
                if norm["tensor"] in own:
                    raise ValueError(f"side_by_side: the member also declares the tensor {norm['tensor']!r}")
                own[norm["tensor"]] = TensorDecl(shape=(int(norm["size"]),), init="ones_normal")
            for local, decl in own.items():
                if ps.prefix + local in t:
                    raise ValueError(f"side_by_side: two members declare the tensor {ps.prefix + local!r}")
                t[ps.prefix + local] = decl
        return t

    @classmethod
    def cache_request(cls, spec: PartSpec):
        return tuple(mcls.cache_request(ps) for ps, mcls, _, _ in _members(spec))

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], rt: Runtime):
        self.rt = rt
        self.members = []
        weights_n, self.norm_eps = [], []          # of the members with a norm, their factors multiplied in
        for ps, mcls, w, norm in _members(spec):
            own = {local: weights[ps.prefix + local] for local in mcls.tensors(ps) if ps.prefix + local in weights}
            part = mcls(ps, own, rt)
            if norm is not None:
                weights_n.append(rt.vector(weights[ps.prefix + norm["tensor"]]) * w)
                self.norm_eps.append(float(norm["eps"]))
                self.members.append((part, w, None))
                continue
            take = getattr(part, "scale_output", None)
            direct = w == 1.0 or (take is not None and bool(take(w)))
            self.members.append((part, w, direct))
        if len(weights_n) > K.NORMED_MAX:
            raise ValueError(f"side_by_side: at most {K.NORMED_MAX} members have a norm")
        # do all members with a norm store their outputs, so that nobody has to clear the buffers?
        self.overwrites = all(getattr(p, "overwrites", False) for p, _, direct in self.members if direct is None)
        self.norm_weight = torch.stack(weights_n).contiguous() if weights_n else None

    def absorb_norm(self, norm) -> bool:
        """The norm before this mixer goes into every member's first projection, or into none: all members read
        the same input."""
        parts = [p for p, _, _ in self.members]
        if not all(getattr(p, "can_absorb_norm", None) is not None and p.can_absorb_norm(norm) for p in parts):
            return False
        return all([bool(p.absorb_norm(norm)) for p in parts])

    @property
    def capturable(self) -> bool:
        return all(getattr(p, "capturable", True) for p, _, _ in self.members)

    def prepare(self, ctx: StepContext) -> None:
        for part, _, _ in self.members:
            prep = getattr(part, "prepare", None)
            if prep is not None:
                prep(ctx)

    def forward(self, h: torch.Tensor, residual: torch.Tensor, ctx: StepContext, cache, writes_cache: bool = True) -> None:
        if not isinstance(cache, tuple) or len(cache) != len(self.members):
            raise ValueError("side_by_side: one cache view per member is expected")
        # no member's last product is the last add into the stream: none of them is offered the stream's rows
        ahead = ctx.shared.pop("row_stats", None)
        parts_out = None
        if self.norm_weight is not None:
            parts_out = ctx.ws.get("side_by_side_normed", (len(self.norm_eps),) + tuple(residual.shape), torch.float32)
            if not self.overwrites and ctx.shared.get(self.ZEROED) != (parts_out.data_ptr(), parts_out.numel()):
                parts_out.zero_()
        k = 0
        for (part, w, direct), view in zip(self.members, cache):
            if direct is None:
                if self.overwrites:
                    ctx.shared["output_empty"] = True
                part.forward(h, parts_out[k], ctx, view, writes_cache)
                ctx.shared.pop("output_empty", None)
                k += 1
                continue
            if direct:
                part.forward(h, residual, ctx, view, writes_cache)
                continue
            buf = ctx.ws.get("side_by_side_out", tuple(residual.shape), torch.float32)
            buf.zero_()
            part.forward(h, buf, ctx, view, writes_cache)
            K.residual_axpy(residual, buf, w)
        if ahead is not None:
            ctx.shared["row_stats"] = ahead
        if parts_out is not None:
            emit = isinstance(ahead, NormedRows) and ahead.norm is not None and ahead.rows.shape == residual.shape
            K.normed_sum(residual, parts_out, self.norm_weight, self.norm_eps, ahead.rows if emit else None,
                         ahead.norm.emit if emit else None, zero_y=not self.overwrites)
            if emit:
                ahead.fresh = True
            if self.overwrites:
                ctx.shared.pop(self.ZEROED, None)
            else:
                ctx.shared[self.ZEROED] = (parts_out.data_ptr(), parts_out.numel())
