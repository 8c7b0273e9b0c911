"""The gated delta rule as a mixer part: a recurrence whose state is corrected, token by token, by
what it already returns for the new key; state and the short convolutions' kept inputs per request
live in a float32 state slot of the cache."""

from __future__ import annotations

from typing import Mapping, Optional, Sequence

import torch

from tokensprint_b200 import ops
from tokensprint_b200.parts.base import BuildContext, CacheNeed, LayerCache, Mixer, StepContext, TensorSpec, register_part
from tokensprint_b200.parts.linear import linear, linear_float32_out

DECAY_AHEAD_TOKENS = 64  # steps of more tokens work the decays per key channel out in a kernel of their own


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    """With H heads of value width e, G <= H heads of q and k of width d (head h reads q/k head
    h // (H / G)), for the tokens of a sequence in order:

        q = silu(conv(W_q x)),  k = silu(conv(W_k x)),  v = silu(conv(W_v x))     short causal convolutions per
                                                                                channel, `taps` wide, no bias
        q <- q / sqrt(sum q^2 + unit_eps) * q_scale,   k <- k / sqrt(sum k^2 + unit_eps)     per head
        beta = sigmoid(W_b x),   g = exp(-exp(A_log_h) * softplus(W_a x + dt_bias_h))         per head
        S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q                      S [d, e], zero at first
        y = W_o ( concat over heads of  o * rsqrt(mean(o^2) + norm_eps) * w_norm * silu(W_g x) )

    `decay_pair` = (a1, a2) in place of `decay`: a decay per head and key channel, through a narrow pair of matrices,
        g = exp(-exp(A_log_h) * softplus(W_a2 (W_a1 x) + dt_bias))       laid out H x d, dt_bias [H d]
        S <- diag(g) S
    `gate_pair` = (g1, g2) in place of `gate` (the two pairs come together): the output gate through a narrow pair as
    well; `gate_activation` "silu" (the default) or "sigmoid" is what the gate passes through.

    Parameters: `hidden_size`, `num_heads`, `num_qk_heads`, `key_dim`, `value_dim`, `taps`, `norm_eps`,
    `unit_eps` (default 1e-6), `q_scale` (default key_dim^-0.5), `decay_rank` / `gate_rank` (inner widths of
    the pairs; None: the checkpoint's own) and the tensors' names.  One product
    gives [q | k | v | output gate] in the compute dtype, a second one the raw write-strength and
    decay rows, whose sums leave in float32.  With the pairs, one product gives [q | k | v | a1 | g1 | write
    strength] and a second one, whose matrix holds W_a2 and W_g2 as two blocks, the raw decay and gate rows in
    float32.  The convolutions with their silu, unit lengths, beta,
    the decay, the state, the recurrence and the head norm are float32 whatever the compute dtype.
    The state slot holds the state [H, e, d] (value column by value column) followed by the last
    taps - 1 inputs of the convolutions [taps - 1, 2 G d + H e], oldest first; zeros before the first
    token, so prompts may be cut anywhere."""

    graph_safe = True
    reads_through_ops = True

    def __init__(self, ctx: BuildContext, *, hidden_size: int, num_heads: int, num_qk_heads: int, key_dim: int, value_dim: int, taps: int,
                 norm_eps: float, q: str, k: str, v: str, q_conv: str, k_conv: str, v_conv: str, beta: str, a_log: str,
                 dt_bias: str, norm: str, o: str, decay: Optional[str] = None, gate: Optional[str] = None,
                 decay_pair: Optional[Sequence[str]] = None, gate_pair: Optional[Sequence[str]] = None, decay_rank: Optional[int] = None,
                 gate_rank: Optional[int] = None, gate_activation: str = "silu", unit_eps: float = 1e-6,
                 q_scale: Optional[float] = None) -> None:
        self.hidden_size, self.num_heads, self.num_qk_heads = int(hidden_size), int(num_heads), int(num_qk_heads)
        self.key_dim, self.value_dim, self.taps = int(key_dim), int(value_dim), int(taps)
        self.norm_eps, self.unit_eps = float(norm_eps), float(unit_eps)
        if min(self.num_heads, self.num_qk_heads, self.key_dim, self.value_dim, self.taps) < 1 or self.num_heads % self.num_qk_heads:
            raise ValueError("gated delta rule: sizes must be positive and heads a multiple of the q/k heads")
        if self.key_dim > ops.DELTA_MAX_KEY_DIM:
            raise ValueError(f"gated delta rule: key_dim {key_dim} exceeds the kernel's {ops.DELTA_MAX_KEY_DIM}")
        self.per_channel = decay_pair is not None
        if (decay_pair is None) != (gate_pair is None) or self.per_channel == (decay is not None) or self.per_channel == (gate is not None):
            raise ValueError("gated delta rule: either a decay and a gate matrix, or a narrow pair of matrices for each of the two")
        if gate_activation not in ("silu", "sigmoid"):
            raise ValueError(f"gated delta rule: gate_activation must be 'silu' or 'sigmoid', got {gate_activation!r}")
        self.gate_activation = gate_activation
        self.ranks = (-1 if decay_rank is None else int(decay_rank), -1 if gate_rank is None else int(gate_rank))
        self.q_scale = float(q_scale) if q_scale is not None else float(self.key_dim) ** -0.5
        self.qk_width, self.v_width = self.num_qk_heads * self.key_dim, self.num_heads * self.value_dim
        self.channels = 2 * self.qk_width + self.v_width
        self.memory_floats = self.num_heads * self.key_dim * self.value_dim
        self.names = {"q": q, "k": k, "v": v, "q_conv": q_conv, "k_conv": k_conv, "v_conv": v_conv, "beta": beta, "decay": decay,
                      "a_log": a_log, "dt_bias": dt_bias, "gate": gate, "norm": norm, "o": o}
        if self.per_channel:
            self.names.update(a1=decay_pair[0], a2=decay_pair[1], g1=gate_pair[0], g2=gate_pair[1])
        self.in_weight: Optional[torch.Tensor] = None    # [q | k | v | gate] stacked, or [q | k | v | a1 | g1 | beta]
        self.gate_rows: Optional[torch.Tensor] = None    # [beta | decay] stacked
        self.pair_out: Optional[torch.Tensor] = None     # a2 and g2 as the two blocks of one matrix
        self.o_weight: Optional[torch.Tensor] = None

    def first_weight(self) -> Optional[torch.Tensor]:
        return self.in_weight

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="none", state_shape=(self.memory_floats + (self.taps - 1) * self.channels,), state_dtype=torch.float32)

    def tensor_specs(self) -> list[TensorSpec]:
        W, n, H = self.hidden_size, self.names, self.num_heads
        specs = [TensorSpec(n["q"], (self.qk_width, W)), TensorSpec(n["k"], (self.qk_width, W)), TensorSpec(n["v"], (self.v_width, W)),
                 TensorSpec(n["q_conv"], (self.qk_width, self.taps), "vector"), TensorSpec(n["k_conv"], (self.qk_width, self.taps), "vector"),
                 TensorSpec(n["v_conv"], (self.v_width, self.taps), "vector"), TensorSpec(n["beta"], (H, W)), TensorSpec(n["a_log"], (H,), "vector"),
                 TensorSpec(n["norm"], (self.value_dim,), "vector"), TensorSpec(n["o"], (W, self.v_width))]
        if not self.per_channel:
            return specs + [TensorSpec(n["decay"], (H, W)), TensorSpec(n["dt_bias"], (H,), "vector"), TensorSpec(n["gate"], (self.v_width, W))]
        ra, rg, Hd = *self.ranks, H * self.key_dim
        return specs + [TensorSpec(n["a1"], (ra, W)), TensorSpec(n["a2"], (Hd, ra)), TensorSpec(n["dt_bias"], (Hd,), "vector"),
                        TensorSpec(n["g1"], (rg, W)), TensorSpec(n["g2"], (self.v_width, rg))]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        qkv = [tensors[n["q"]], tensors[n["k"]], tensors[n["v"]]]
        if self.per_channel:
            self._load_pairs(qkv, tensors)
        else:
            self.in_weight = torch.cat(qkv + [tensors[n["gate"]]], dim=0).contiguous()
            self.gate_rows = torch.cat([tensors[n["beta"]], tensors[n["decay"]]], dim=0).contiguous()
        # the three convolutions as one, tap by tap [taps, channels], as the kernel reads them
        self.conv_weight = torch.cat([tensors[n["q_conv"]], tensors[n["k_conv"]], tensors[n["v_conv"]]], dim=0).t().contiguous()
        self.a_log, self.dt_bias = tensors[n["a_log"]], tensors[n["dt_bias"]]
        self.norm_weight, self.o_weight = tensors[n["norm"]], tensors[n["o"]]

    def _load_pairs(self, qkv: list[torch.Tensor], tensors: Mapping[str, torch.Tensor]) -> None:
        """Stacks [q | k | v | a1 | g1 | beta] and puts a2 and g2 into one matrix.  Zero rows bring the inner rows
        to a multiple of eight columns of the product, at a multiple of eight, and the whole row to one."""
        n = self.names
        a1, a2, g1, g2, beta = (tensors[n[k]] for k in ("a1", "a2", "g1", "g2", "beta"))
        for narrow, wide in (("a1", "a2"), ("g1", "g2")):
            if tensors[n[narrow]].shape[0] != tensors[n[wide]].shape[1]:
                raise ValueError(f"gated delta rule: {n[narrow]} has {tensors[n[narrow]].shape[0]} rows, {n[wide]} {tensors[n[wide]].shape[1]} columns")
        ra, rg = int(a1.shape[0]), int(g1.shape[0])

        def fill(rows: int) -> torch.Tensor:
            return torch.zeros((-rows % 8, self.hidden_size), device=a1.device, dtype=a1.dtype)

        self.low_at = self.channels + (-self.channels % 8)
        self.low_width = ra + rg + (-(ra + rg) % 8)
        self.beta_at = self.low_at + self.low_width
        self.in_weight = torch.cat(qkv + [fill(self.channels), a1, g1, fill(ra + rg), beta, fill(self.num_heads)], dim=0).contiguous()
        Hd = self.num_heads * self.key_dim
        self.pair_out = torch.zeros((Hd + self.v_width, self.low_width), device=a2.device, dtype=a2.dtype)
        self.pair_out[:Hd, :ra] = a2
        self.pair_out[Hd:, ra:ra + rg] = g2

    def forward(self, x: torch.Tensor, step: StepContext, cache: LayerCache) -> torch.Tensor:
        if cache.state is None:
            raise ops.KernelError("gated delta rule: this mixer needs a state slot per request (none was bound to its run)")
        if not cache.writes:
            raise ops.KernelError("gated delta rule: a run cannot read another run's state")
        T, H, G, d, e = x.shape[0], self.num_heads, self.num_qk_heads, self.key_dim, self.value_dim
        C = self.channels
        state = cache.state.view(cache.state.shape[0], -1)
        if self.per_channel:
            proj = linear(x, self.in_weight, next_weight=self.pair_out)
            rows = linear_float32_out(proj[:, self.low_at:self.low_at + self.low_width], self.pair_out)
            beta, decay, gate = proj[:, self.beta_at:self.beta_at + H], rows[:, :H * d], rows[:, H * d:]
        else:
            rows = linear_float32_out(x, self.gate_rows)
            proj = linear(x, self.in_weight, next_weight=self.o_weight)
            beta, decay, gate = rows[:, :H], rows[:, H:], proj[:, C:]
        conv = torch.empty((T, C), device=x.device, dtype=torch.float32)
        ops.causal_conv(proj[:, :C], self.conv_weight, None, state[:, self.memory_floats:] if self.taps > 1 else None, step.state_slots,
                        step.cu_seqlens_q, step.seq_index, step.num_seqs, conv, activation="silu")
        a_log, dt_bias = self.a_log, self.dt_bias
        if self.per_channel and T > DECAY_AHEAD_TOKENS:
            # the scan's CTAs that share a head would all work these out
            ops.channel_decay(decay, a_log, dt_bias, H, d)
            a_log = dt_bias = None
        o = torch.empty((T, self.v_width), device=x.device, dtype=torch.float32)
        ops.delta_scan(conv, 0, self.qk_width, 2 * self.qk_width, beta, decay, a_log, dt_bias, state, step.state_slots, step.cu_seqlens_q, o,
                       step.num_seqs, H, G, d, e, self.q_scale, self.unit_eps, max_seqlen=step.max_seqlen_q)
        y = torch.empty((T, self.v_width), device=x.device, dtype=x.dtype)
        ops.gla_norm_gate(o, gate, self.norm_weight, y, H, e, self.norm_eps, activation=self.gate_activation)
        return linear(y, self.o_weight, next_weight=step.weight_after)
