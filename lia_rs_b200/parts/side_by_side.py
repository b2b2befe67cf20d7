"""Several mixers side by side: all read the same input, and the result is the weighted sum of theirs,

    mixer(x) = sum_i scale_i * norm_i(mixer_i(x)),    norm_i an RMS norm with a weight over the model's width, or nothing.

Each member is a registered mixer with its own parameters and checkpoint prefix.  Without norms every member adds its share
into the residual stream itself (a mixer's `forward` does `residual += scale * f(x)`, so the weights ride on the members'
last products and no sum is formed anywhere else).  With norms every member stores into rows of its own, and the sum is
left to the arrangement as terms (`Mixer.output_terms`), which norms, adds and joins the stream in one kernel; an output
bias of such a member is added there too.  Members that read their input through one product each (`projects_input`) then
share one product.  At most one member may ask for a paged cache and at most one for per-request
state: the layer's cache and state are handed to those.

Parameters: `members`: a list of {"kind", "params", "prefix", "scale", "norm": {"tensor", "hidden", "eps"} (absent: none; the
weight's checkpoint name behind the mixer's prefix)}; either all members have a norm or none has."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import TensorSpec
from .base import MIXERS, Mixer, lookup, register_mixer
from .linear import STORE, linear


@register_mixer("side_by_side")
class SideBySide(Mixer):
    can_store = False

    @staticmethod
    def _members(params):
        return [(lookup(MIXERS, m["kind"], "mixer"), m["params"], m.get("prefix", ""), float(m.get("scale", 1.0)))
                for m in params["members"]]

    @staticmethod
    def check_params(params):
        members = SideBySide._members(params)
        if not members:
            raise ValueError("mixers side by side: at least one member")
        for cls, member_params, _, _ in members:
            cls.check_params(member_params)
        if sum(cls.cache_request(p) is not None for cls, p, _, _ in members) > 1 or \
                sum(cls.state_request(p) is not None for cls, p, _, _ in members) > 1:
            raise ValueError("mixers side by side: at most one member with a paged cache and one with per-request state")
        normed = [m.get("norm") is not None for m in params["members"]]
        if any(normed) and (not all(normed) or len(normed) > 2 or not all(cls.can_store for cls, _, _, _ in members)):
            raise ValueError("mixers side by side: norms for all members or for none, of at most two members that can store")

    @staticmethod
    def tensor_specs(params, prefix):
        specs = [spec for cls, p, member_prefix, _ in SideBySide._members(params) for spec in cls.tensor_specs(p, prefix + member_prefix)]
        return specs + [TensorSpec(prefix + m["norm"]["tensor"], (int(m["norm"]["hidden"]),), kind="norm")
                        for m in params["members"] if m.get("norm")]

    @staticmethod
    def cache_request(params):
        for cls, p, _, _ in SideBySide._members(params):
            if cls.cache_request(p) is not None:
                return cls.cache_request(p)
        return None

    @staticmethod
    def state_request(params):
        for cls, p, _, _ in SideBySide._members(params):
            if cls.state_request(p) is not None:
                return cls.state_request(p)
        return None

    def __init__(self, params, tensors, prefix, runtime):
        super().__init__(params, tensors, prefix, runtime)
        self.check_params(params)
        self.members = []
        for cls, p, member_prefix, scale in self._members(params):
            part = cls(p, tensors, prefix + member_prefix, runtime)
            if part.output_bias is not None and not params["members"][0].get("norm"):
                raise ValueError("mixers side by side: a member's output bias is not added")
            self.members.append((part, scale, cls.cache_request(p) is not None, cls.state_request(p) is not None))
        # per member (weight, eps) of its norm: the sum is then the arrangement's
        self.norms = [(tensors[prefix + m["norm"]["tensor"]].to(torch.float32).contiguous(), float(m["norm"]["eps"]))
                      for m in params["members"] if m.get("norm")]
        self.gives_terms = bool(self.norms)
        # members whose input products can be one product over the same rows
        self.runtime, self.w_in, self.columns = runtime, None, []
        if self.gives_terms and all(part.projects_input for part, _, _, _ in self.members):
            at = 0
            for part, _, _, _ in self.members:
                self.columns.append((at, at + part.w_in.shape[0]))
                at += part.w_in.shape[0]
            self.w_in = torch.cat([part.w_in for part, _, _, _ in self.members], dim=0)
            for part, _, _, _ in self.members:
                part.w_in = None
        self.graph_safe = all(part.graph_safe for part, _, _, _ in self.members)
        self.takes_deferred_norm = all(part.takes_deferred_norm for part, _, _, _ in self.members)

    def graph_key(self, ctx) -> tuple:
        key = ()
        for part, _, _, _ in self.members:
            key += part.graph_key(ctx)
        return key

    def output_terms(self, ctx, x, kv=None, state=None):
        n, terms, projected = x.shape[0], [], [{} for _ in self.members]
        if self.w_in is not None:
            shared = ctx.buffer("side_by_side.in", (n, self.w_in.shape[0]), torch.float32)
            linear(self.runtime, STORE, x, self.w_in, shared, error_flag=ctx.error_flag, name="mixers_in")
            projected = [{"projected": shared[:, begin:end]} for begin, end in self.columns]
        for i, ((part, weight, wants_cache, wants_state), (norm, eps)) in enumerate(zip(self.members, self.norms)):
            rows = ctx.buffer(f"side_by_side.{i}", (n, norm.numel()), torch.float32)
            part.forward(ctx, x, rows, 1.0, kv=kv if wants_cache else None, state=state if wants_state else None, store=True,
                         **projected[i])
            terms.append(ops.NormTerm(rows, bias=part.output_bias, weight=norm, scale=weight, eps=eps))
        return terms

    def forward(self, ctx, x, residual, scale, kv=None, state=None):
        if self.gives_terms:
            raise ValueError("mixers side by side with norms leave their sum to the arrangement")
        for part, weight, wants_cache, wants_state in self.members:
            part.forward(ctx, x, residual, scale * weight, kv=kv if wants_cache else None, state=state if wants_state else None)
