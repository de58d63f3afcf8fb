"""Mixture-of-experts ops: router top-k and the routed-expert FFN.

CPU path (oracle): route with the reference formulas, then loop over experts.
CUDA path: ``csrc/moe.cu`` — one block per token for routing (softmax top-k, or sigmoid +
selection bias + group-limited top-k), a counting sort of (token, expert) pairs into
expert-contiguous rows with a tile work-list, then the tcgen05 grouped GEMMs over
``[experts * N, K]`` stacked weights, and a weighted un-permute that also blends the shared
expert. Reference behaviour: ``kernels/gb10/common/moe_topk.cu``, ``moe_topk_sigmoid.cu``,
``moe_permute.cu``, ``moe_w8a8_grouped_gemm.cu``, ``moe_unpermute_blend.cu``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from . import _native, reference as ref


@dataclass
class GroupedExperts:
    """Experts stacked along N for the grouped GEMM: gate_up [E * 2I, K], down [E * H, I]."""
    gate_up: object
    down: object
    num: int
    n_gate_up: int
    n_down: int
    interleaved: bool
    shared_slot: Optional[int] = None     # local expert index of a folded-in shared expert (every token routes to it)
    clamp_glu: Optional[tuple] = None     # (alpha, limit): clamped GLU instead of SwiGLU (interleaved rows)


@dataclass
class RouterSpec:
    """Routing of one layer, where layers differ; the names are the model configuration's."""
    num_experts: int
    experts_per_token: int
    router: str = "softmax_topk"          # softmax over the chosen ones of the biased logits; "softmax_grouped": softmax over
                                          # all, chosen from the groups with the largest scores, times router_scaling
    router_n_group: int = 1
    router_topk_group: int = 1
    router_renormalize: bool = True
    router_scaling: float = 1.0
    ffn_act: str = "swiglu"


def stack_experts(experts) -> Optional[GroupedExperts]:
    if not experts:
        return None
    from . import concat_weights
    nvfp4 = experts[0].gate_up.fmt == "nvfp4"
    if nvfp4 and (experts[0].gate_up.N % 128 or experts[0].down.N % 128):
        # the scale factors of an NVFP4 operand are tiled by 128 rows: an expert whose row count is not a
        # multiple of that shares a tile with its neighbour, and such experts run one GEMM per active expert
        # (models/moe.py::routed_experts) instead of the grouped path
        return None
    gu = concat_weights([e.gate_up for e in experts])
    dn = concat_weights([e.down for e in experts])
    if nvfp4 and gu.data.is_cuda:
        gu.prepare_cuda()                                  # tiled scale factors, built once at load
        dn.prepare_cuda()
    return GroupedExperts(gu, dn, len(experts), experts[0].gate_up.N, experts[0].down.N,
                          experts[0].interleaved)


def route(logits: torch.Tensor, cfg, bias=None):
    """Router logits [T, E] fp32 -> (weights [T, k] fp32, expert ids [T, k] int32)."""
    k = cfg.experts_per_token
    if logits.is_cuda and _native.available() and hasattr(_native.lib(), "mb_moe_route"):
        from .moe_cuda import route_cuda
        return route_cuda(logits, cfg, bias)
    if cfg.router == "softmax_topk":
        z = logits.float() if bias is None else logits.float() + bias
        top, idx = ref.topk_stable(z, k)
        w = torch.softmax(top, -1)
    elif cfg.router == "softmax_grouped":
        w, idx = ref.route_softmax_grouped(logits, k, cfg.router_n_group, cfg.router_topk_group, cfg.router_renormalize, cfg.router_scaling)
    elif cfg.router == "softmax":
        w, idx = ref.route_softmax_topk(logits, k, cfg.router_renormalize)
    else:
        w, idx = ref.route_sigmoid_grouped(logits, bias, k, cfg.router_n_group, cfg.router_topk_group,
                                           cfg.router_renormalize, cfg.router_scaling)
    return w.float(), idx.to(torch.int32)


def expert_sum_ref(act, weights: torch.Tensor, idx: torch.Tensor, ge: GroupedExperts, width: int, ffn_act: str = "swiglu") -> torch.Tensor:
    """CPU: sum_j weights[t, j] * expert idx[t, j] of row t over stacked (padded) experts; fp32 [T, width]."""
    from . import Act, QuantWeight, linear
    out = torch.zeros(act.M, width)
    part = lambda w, e, n: QuantWeight(w.fmt, n, w.K, w.data[e * n:(e + 1) * n])
    epi = dict(relu2=True) if ffn_act == "relu2" else dict(swiglu=ge.clamp_glu is None, clamp_glu=ge.clamp_glu)
    for e in range(ge.num):
        tok, slot = torch.nonzero(idx == e, as_tuple=True)
        if tok.numel() == 0:
            continue
        h = linear(Act(act.fmt, tok.numel(), act.K, act.data[tok]), part(ge.gate_up, e, ge.n_gate_up), **epi)
        y = linear(Act(act.fmt, tok.numel(), h.shape[1], h.float()), part(ge.down, e, ge.n_down), out_f32=True)
        out.index_add_(0, tok, y[:, :width] * weights[tok, slot][:, None])
    return out
