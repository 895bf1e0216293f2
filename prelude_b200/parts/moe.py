"""Routed experts: a mixture of feed-forwards (SiLU-gated, gated by the clamped unit, or plain with squared ReLU), a few per token.

The router's logits are a 32-bit product of the feed-forward's input with the
router matrix (float32 sums of exact products on the float32 units, whatever
the run's type: ``kernels.router_logits``), plus a bias where the design has one.  Scores are their sigmoids or their softmax,
or the logits themselves with the softmax over the chosen ones as weights; experts form equal groups of
neighbours, a group scores the sum of its largest scores, and only experts of
the best groups can be chosen; the chosen scores weigh the experts' outputs
(``RoutedExpertsSpec`` has the constants).  A learned correction per expert may
join the scores for the choice alone, and one more expert may run for every token.

All experts' gate and up rows live in one tensor [experts, 2 * expert_size,
hidden] and their down rows in another [experts, hidden, expert_size].  A step
groups its (token, choice) pairs by expert on the device and runs two grouped
products over them (gate/up with the activation in the epilogue, then down)
and a weighted sum per token: five launches after the router's product, none
of whose shapes depends on what the router chose, so the part can be recorded.
A decode step's few tokens take a shorter way: router product and choice in one
kernel, no grouping (the products look an expert's rows up in the choices).
The weighted sum runs together with what stands behind it where the block hands it
on (``defer_output``): the residual add and a squashing, or the norm of the
output, the add and the norm that follows.  Plain experts have up rows only in the
first tensor.
"""
from __future__ import annotations

import os
from typing import Dict

import torch

from ..config.spec import RoutedExpertsSpec
from ..ops import kernels as K
from ..ops import linear as L
from ..weights.loader import TensorReq
from .registry import RunContext, register_part


# average rows per expert up to which a step's products run on the kernel that only streams the experts' weights
MOE_FEW_ROWS = int(os.environ.get("PRELUDE_MOE_FEW_ROWS", "6"))
# tokens up to which the router's product and choice run in one kernel
ROUTE_FEW_TOKENS = int(os.environ.get("PRELUDE_MOE_ROUTE_FEW_TOKENS", "32"))
# average rows per expert from which a step's products run on the paired-block tcgen05 kernel
MOE_PAIR_MIN_ROWS = int(os.environ.get("PRELUDE_MOE_PAIR_MIN_ROWS", "192"))

# an activation's name: (two matrices on the way up or one, its number in the products' epilogues)
_ACTS = {"silu_gated": (True, K.ACT_NONE), "clamped_glu": (True, K.ACT_CLAMPED), "relu2": (False, K.ACT_RELU2)}


@register_part("feed_forward", "routed_experts")
class RoutedExperts:
    defer_output = False        # True: the weighted sum is handed on as a kernel still to run (``PendingExperts``)

    def __init__(self, spec: RoutedExpertsSpec, prefix: str):
        s = spec
        if s.activation not in _ACTS or s.scoring not in ("sigmoid", "softmax", "softmax_chosen"):
            raise ValueError(f"routed experts with activation {s.activation!r} and scores by {s.scoring!r} are not known")
        if s.scoring == "softmax_chosen" and s.renormalize:
            raise ValueError("weights that are a softmax over the chosen experts add up to one: nothing to renormalize")
        self.gated, act = _ACTS[s.activation]
        self.clamped = act == K.ACT_CLAMPED
        if self.clamped and (s.limit <= 0 or (s.shared_size is not None and s.shared_limit <= 0)):
            raise ValueError(f"the clamped unit needs a positive limit, got {s.limit} and {s.shared_limit} for the shared expert")
        self.act = dict(act=act, limit=s.limit, alpha=s.alpha) if self.clamped else dict(act=act)
        if s.n_experts % s.n_groups or not 0 < s.keep_groups <= s.n_groups:
            raise ValueError(f"{s.n_experts} experts do not form {s.n_groups} equal groups of which {s.keep_groups} are kept")
        if not 0 < s.top_k <= s.keep_groups * (s.n_experts // s.n_groups):
            raise ValueError(f"top_k={s.top_k} experts cannot come from {s.keep_groups} groups of {s.n_experts // s.n_groups}")
        self.spec, self.prefix = spec, prefix
        self.w_router = self.w_gate_up = self.w_down = self.correction = self.router_bias = None
        self.w_shared_up = self.w_shared_down = None

    def _expert(self, e: int, name: str) -> str:
        return f"{self.prefix}.{self.spec.expert_prefix}{e}.{name}"

    def tensors(self) -> Dict[str, TensorReq]:
        s = self.spec
        req = {f"{self.prefix}.{s.router_name}": TensorReq((s.n_experts, s.hidden_size))}
        if s.correction_name is not None:
            req[f"{self.prefix}.{s.correction_name}"] = TensorReq((s.n_experts,), "bias")
        if s.router_bias_name is not None:
            req[f"{self.prefix}.{s.router_bias_name}"] = TensorReq((s.n_experts,), "bias")
        every = [(f"{self.prefix}.{s.expert_prefix}{e}", s.expert_size) for e in range(s.n_experts)]
        if s.shared_size is not None:
            every.append((f"{self.prefix}.{s.shared_prefix}", s.shared_size))
        for name, size in every:
            if self.gated:
                req[f"{name}.{s.gate_name}"] = TensorReq((size, s.hidden_size))
            req[f"{name}.{s.up_name}"] = TensorReq((size, s.hidden_size))
            req[f"{name}.{s.down_name}"] = TensorReq((s.hidden_size, size))
        return req

    def load(self, get, ctx: RunContext) -> None:
        s = self.spec

        def mat(name):
            return get(name).to(device=ctx.device, dtype=ctx.dtype)

        self.w_router = mat(f"{self.prefix}.{s.router_name}").contiguous()

        def vec(name):
            return get(f"{self.prefix}.{name}").to(device=ctx.device, dtype=torch.float32).contiguous()

        if s.correction_name is not None:
            self.correction = vec(s.correction_name)
        if s.router_bias_name is not None:
            self.router_bias = vec(s.router_bias_name)

        def up(name):
            rows = [mat(f"{name}.{s.gate_name}"), mat(f"{name}.{s.up_name}")] if self.gated else [mat(f"{name}.{s.up_name}")]
            return torch.cat(rows, dim=0).contiguous()

        self.w_gate_up = torch.stack([up(f"{self.prefix}.{s.expert_prefix}{e}") for e in range(s.n_experts)]).contiguous()
        self.w_down = torch.stack([mat(self._expert(e, s.down_name)) for e in range(s.n_experts)]).contiguous()
        if s.shared_size is not None:
            self.w_shared_up = up(f"{self.prefix}.{s.shared_prefix}")
            self.w_shared_down = mat(f"{self.prefix}.{s.shared_prefix}.{s.down_name}").contiguous()

    def activation_bytes_per_token(self, elem: int) -> int:
        s = self.spec
        shared = 0 if s.shared_size is None else 2 * s.shared_size * elem + s.hidden_size * 4
        return s.top_k * (s.expert_size * elem + s.hidden_size * 4) + s.n_experts * 4 + s.hidden_size * elem + shared

    def pair_takes(self, x: torch.Tensor) -> bool:
        """Whether a step's products run on the paired-block kernel: bfloat16, aligned sizes, and rows enough that an
        expert's 256-row tiles are mostly full (PRELUDE_MOE_PAIR_MIN_ROWS rows per expert on average, default 192)."""
        s = self.spec
        return (x.dtype == torch.bfloat16 and L.PREFILL_GEMM != "cublas" and s.hidden_size % 8 == 0 and s.expert_size % 8 == 0
                and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and x.shape[0] * s.top_k >= MOE_PAIR_MIN_ROWS * s.n_experts
                # operands no smaller than one copy box of the kernel (128 rows of 64 elements)
                and s.hidden_size >= 64 and s.expert_size >= 64 and s.n_experts * min(s.hidden_size, self.w_gate_up.shape[1]) >= 128)

    def _router_args(self):
        s = self.spec
        return (s.top_k, s.n_groups, s.keep_groups, s.group_score_top, s.renormalize, self.correction, s.scoring == "softmax",
                s.renormalize_eps, s.weight_scale, self.router_bias, s.scoring == "softmax_chosen")

    def route(self, x: torch.Tensor):
        """(experts int32 [T, top_k], weights float32 [T, top_k]) for the rows of x."""
        if x.shape[0] <= ROUTE_FEW_TOKENS and K.moe_route_few_takes(x, self.w_router):
            return K.moe_route_few(x, self.w_router, *self._router_args())
        return K.moe_route(K.router_logits(x, self.w_router), *self._router_args())

    def shared(self, x: torch.Tensor):
        """What every token adds beside its experts, or None."""
        if self.w_shared_up is None:
            return None
        s = self.spec
        if self.clamped:
            h = L.gated_linear_clamped(x, self.w_shared_up, s.shared_limit, s.alpha)
            if h is None:
                h = K.clamped_glu(L.linear(x, self.w_shared_up), s.shared_limit, s.alpha)
        elif self.gated:
            h = L.gated_linear_silu(x, self.w_shared_up)
            if h is None:
                h = K.silu_mul(L.linear(x, self.w_shared_up))
        else:
            h = L.linear_relu2(x, self.w_shared_up)
        return L.linear(h, self.w_shared_down, partial_sums_ok=True)

    def _sum(self, y: torch.Tensor, place_of, weights: torch.Tensor, shared, dtype: torch.dtype):
        out = K.PendingExperts(y, place_of, weights, shared, dtype)
        return out if self.defer_output else out.resolve()

    def forward(self, x: torch.Tensor):
        s = self.spec
        ids, weights = self.route(x)
        shared = self.shared(x)
        if self.pair_takes(x):
            # a long prompt step: rows sorted by expert, both products on the paired-block tcgen05 kernel (tiles of 256 rows)
            plan = K.moe_sort(ids, s.n_experts, 256)
            status = L.tc_status(x.device)
            h = K.moe_gemm_pair(K.moe_gather_rows(x, plan, s.top_k), self.w_gate_up, plan, self.gated, status, **self.act)
            return self._sum(K.moe_gemm_pair(h, self.w_down, plan, False, status), plan.place_of, weights, shared, x.dtype)
        # tiles of 128 rows where the experts have many rows each and the tensor-core kernel takes the shapes, else of 64
        small = x.dtype != torch.bfloat16 or s.hidden_size % 8 or s.expert_size % 8
        few = not small and x.shape[0] * s.top_k <= MOE_FEW_ROWS * s.n_experts       # a decode step: stream the weights
        if few and K.moe_gemv_takes(x, self.w_gate_up, ids.numel()):
            h = K.moe_gemv(x, self.w_gate_up, ids, False, x.dtype, gated=self.gated, **self.act)
            y = K.moe_gemv(h, self.w_down, ids, True, torch.float32)
            return self._sum(y, None, weights, shared, x.dtype)
        plan = K.moe_sort(ids, s.n_experts, 64 if (small or few) else None)
        h = K.moe_gemm(x, self.w_gate_up, plan, gated=self.gated, gather_div=s.top_k, few_rows=few, **self.act)
        y = K.moe_gemm(h, self.w_down, plan, gated=False, out_dtype=torch.float32, few_rows=few)
        return self._sum(y, plan.place_of, weights, shared, x.dtype)
