"""A gated linear recurrence per channel inside a two-branch block, as a mixer part: the channels' states
and the short convolution's kept inputs per request live in a float32 state slot of the cache."""

from __future__ import annotations

from typing import Mapping, Optional

import torch

from tokensprint_b200 import ops
from tokensprint_b200.parts.base import BuildContext, CacheNeed, LayerCache, Mixer, ResidualNorm, StepContext, TensorSpec, register_part
from tokensprint_b200.parts.linear import folding_possible, linear, linear_into_residual, linear_scaled


@register_part("mixer", "gated_recurrence")
class GatedRecurrence(Mixer):
    """Two branches of `width` channels:

        y = gelu_tanh(W_y x + y_bias)
        u = conv(W_x x + x_bias) + conv_bias             causal, per channel, `taps` wide, no activation
        r = sigmoid(R_b u_b + r_bias),  i = sigmoid(I_b u_b + i_bias)     u in `blocks` equal parts u_b, square matrices
        log a = -decay_scale r softplus(lam),  a = exp(log a)
        S_t = a S_(t-1) + sqrt(1 - a^2) i u,  S = 0 before the first token
        out = W_o (S * y)

    One product gives [y | x]; the convolution adds x's bias as it reads its inputs (the zeros before a
    sequence get none); the block products leave float32 sums; one kernel does gates, recurrence and the
    second branch's gelu, and the block products too in a bfloat16 step of one token per sequence.  Gates, decays, the state and the recurrence are float32 whatever the compute
    dtype.  The state slot holds [width] states followed by the last taps - 1 inputs of the convolution
    [taps - 1, width], oldest first; zeros before the first token, so prompts may be cut anywhere.

    Parameters: `hidden_size`, `width`, `blocks`, `taps`, `decay_scale` and the tensors' names."""

    graph_safe = True
    reads_through_ops = False  # the block products may be the library's
    folds_norms = True

    def __init__(self, ctx: BuildContext, *, hidden_size: int, width: int, blocks: int, taps: int, decay_scale: float, y: str, y_bias: str,
                 x: str, x_bias: str, conv: str, conv_bias: str, r: str, r_bias: str, i: str, i_bias: str, lam: str, o: str) -> None:
        self.hidden_size, self.width, self.blocks, self.taps = int(hidden_size), int(width), int(blocks), int(taps)
        self.decay_scale = float(decay_scale)
        if min(self.width, self.blocks, self.taps) < 1 or self.width % self.blocks:
            raise ValueError("gated recurrence: sizes must be positive and the width a multiple of the blocks")
        self.block_width = self.width // self.blocks
        self.names = {"y": y, "y_bias": y_bias, "x": x, "x_bias": x_bias, "conv": conv, "conv_bias": conv_bias, "r": r, "r_bias": r_bias,
                      "i": i, "i_bias": i_bias, "lam": lam, "o": o}
        self.in_weight: Optional[torch.Tensor] = None    # [y | x] stacked
        self.gate_weight: Optional[torch.Tensor] = None  # [blocks, 2 block_width, block_width]: per block R_b, then I_b
        self.o_weight: Optional[torch.Tensor] = None

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.in_weight

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="none", state_shape=(self.width * self.taps,), state_dtype=torch.float32)

    def tensor_specs(self) -> list[TensorSpec]:
        W, w, n, B, k = self.hidden_size, self.width, self.names, self.blocks, self.block_width
        vectors = [TensorSpec(n[name], (w,), "vector") for name in ("y_bias", "x_bias", "conv_bias", "lam")]
        return [TensorSpec(n["y"], (w, W)), TensorSpec(n["x"], (w, W)), TensorSpec(n["conv"], (w, self.taps), "vector"),
                TensorSpec(n["r"], (B, k, k)), TensorSpec(n["r_bias"], (B, k), "vector"), TensorSpec(n["i"], (B, k, k)),
                TensorSpec(n["i_bias"], (B, k), "vector"), TensorSpec(n["o"], (W, w))] + vectors

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        self.in_weight = torch.cat([tensors[n["y"]], tensors[n["x"]]], dim=0).contiguous()
        self.y_bias, self.x_bias, self.conv_bias, self.lam = (tensors[n[name]] for name in ("y_bias", "x_bias", "conv_bias", "lam"))
        self.conv_weight = tensors[n["conv"]].t().contiguous()  # tap by tap, as the kernel reads them
        self.gate_weight = torch.cat([tensors[n["r"]], tensors[n["i"]]], dim=1).contiguous()
        self.r_bias, self.i_bias = tensors[n["r_bias"]].reshape(-1), tensors[n["i_bias"]].reshape(-1)
        self.o_weight = tensors[n["o"]]

    def can_fold(self, num_tokens: int, dtype: torch.dtype) -> bool:
        return folding_possible(num_tokens, dtype, self.in_weight, self.o_weight)

    def forward(self, x, step: StepContext, cache: LayerCache, fold: Optional[ResidualNorm] = None):
        """x: [T, hidden], or a PreNormed (its missing 1/rms is applied by the first product).  With `fold` the
        output product adds its result into fold.hidden and the PreNormed of the norm that follows is returned."""
        if cache.state is None:
            raise ops.KernelError("gated recurrence: this mixer needs a state slot per request (none was bound to its run)")
        if not cache.writes:
            raise ops.KernelError("gated recurrence: a run cannot read another run's state")
        w, k, B = self.width, self.block_width, self.blocks
        state = cache.state.view(cache.state.shape[0], -1)
        proj = linear_scaled(x, self.in_weight, next_weight=self.o_weight)
        T, dev, dtype = proj.shape[0], proj.device, proj.dtype
        u = torch.empty((T, w), device=dev, dtype=dtype)
        ops.causal_conv(proj[:, w:], self.conv_weight, self.conv_bias, state[:, w:] if self.taps > 1 else None, step.state_slots,
                        step.cu_seqlens_q, step.seq_index, step.num_seqs, u, in_bias=self.x_bias)
        out = torch.empty((T, w), device=dev, dtype=dtype)
        if step.max_seqlen_q == 1 and ops.rglru_step_supported(u, self.gate_weight):
            ops.rglru_step(u, self.gate_weight, self.r_bias, self.i_bias, self.lam, self.decay_scale, proj[:, :w], self.y_bias, state,
                           step.state_slots, step.seq_index, out)
        else:
            pre = torch.empty((T, B, 2 * k), device=dev, dtype=torch.float32)
            batched = ops.sgemm_nt_batched if dtype == torch.float32 else ops.library_bmm_float32
            batched(u.view(T, B, k).transpose(0, 1), self.gate_weight, pre.transpose(0, 1))
            ops.rglru_scan(u, pre, self.r_bias, self.i_bias, self.lam, self.decay_scale, proj[:, :w], self.y_bias, state, step.state_slots,
                           step.cu_seqlens_q, step.seq_index, out, step.num_seqs, B, step.max_seqlen_q, step.decode_seqs)
        if fold is not None:
            return linear_into_residual(out, self.o_weight, fold, next_weight=step.weight_after)
        return linear(out, self.o_weight, next_weight=step.weight_after)
