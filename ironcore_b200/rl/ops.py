"""Ops of the rollout and GRPO paths: native kernels on CUDA, PyTorch restatements elsewhere (oracle / CPU path)."""

from __future__ import annotations

import torch

from ..ops import native
from ..ops.native import call, ptr, stream_ptr
from ..ops.paged import kv_append, paged_decode, paged_decode_reference  # noqa: F401

P, L, F = native.P, native.L, native.F
native.register("icb_grpo_loss", [P, P, P, P, P, P, P, P, P, L, F, F, P])


class _GrpoLoss(torch.autograd.Function):
    @staticmethod
    def forward(ctx, logp, logp_old, logp_ref, adv, mask, eps, beta):
        n = logp.numel()
        loss = torch.empty_like(logp)
        dlogp = torch.empty_like(logp)
        ratio = torch.empty_like(logp)
        kl = torch.empty_like(logp)
        call("icb_grpo_loss", ptr(logp), ptr(logp_old), ptr(logp_ref), ptr(adv), ptr(mask), ptr(loss), ptr(dlogp),
             ptr(ratio), ptr(kl), n, float(eps), float(beta), stream_ptr())
        ctx.save_for_backward(dlogp)
        ctx.mark_non_differentiable(ratio, kl)
        return loss, ratio, kl

    @staticmethod
    def backward(ctx, gloss, _gr, _gk):
        (dlogp,) = ctx.saved_tensors
        return gloss * dlogp, None, None, None, None, None, None


def grpo_token_loss(logp, logp_old, logp_ref, adv, mask, eps: float, beta: float):
    """Per-token GRPO loss (PPO-clip + beta * k3 KL). All inputs fp32 [N]; returns (loss, ratio, kl)."""
    if logp.is_cuda:
        f = lambda t: None if t is None else t.contiguous().float()
        return _GrpoLoss.apply(f(logp), f(logp_old), f(logp_ref), f(adv), f(mask), eps, beta)
    ratio = torch.exp(logp - logp_old)
    pg = -torch.minimum(ratio * adv, ratio.clamp(1 - eps, 1 + eps) * adv)
    if logp_ref is not None:
        delta = logp_ref - logp
        kl = torch.exp(delta) - delta - 1
    else:
        kl = torch.zeros_like(logp)
    return mask * (pg + beta * kl), ratio.detach(), kl.detach()
