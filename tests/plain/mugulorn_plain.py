"""Plain, slow Mugulorn: whole sequences, no cache, one function per mechanism.

Mugulorn is a decoder-only model with a norm in front of every sublayer and one constant that
multiplies what every sublayer adds:

    x <- x + m mixer(N1(x));   x <- x + m ff(N2(x))      (the second half where a layer has one)

A layer's mixer is one of two.  A latent attention inside a sliding window: queries through a normed
latent, keys and values rebuilt from a normed latent plus one rotated key part for all heads (entry i
turns with entry i + half; frequencies stretched between two wavelengths), a learned score per head
that joins the softmax's denominator only, and the heads' outputs multiplied entry by entry by the
sigmoid of a projection of the input; a layer may read the latents another layer made.  A gated linear
recurrence per channel (two branches, one through gelu, the other through a short convolution; the
decay and the input gate come from products of that branch in blocks).  The feed-forward is a gated
one with the tanh form of gelu.  The embedding table, without its multiplier, is the output matrix.

Everything here runs on whole sequences in one dtype (float64 by default) on the CPU and shares
no code with the engine under test.  `config` is the content of a config.json as a dict,
`weights` a dict of tensors under the checkpoint's names.
"""

from __future__ import annotations

import math
from typing import Callable, Mapping, Optional, Sequence

import torch

Weights = Mapping[str, torch.Tensor]


# ---------------------------------------------------------------------------
# small functions


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """Rows divided by their root mean square (eps under the root), channel by channel times w."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(z, torch.zeros_like(z))


def causal_conv(h: torch.Tensor, w: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """h [T, C], w [C, taps]: out_t = bias + sum_j w[:, j] h_(t - taps + 1 + j); rows before the start are
    zeros (the last column weighs the current token)."""
    T, taps = h.shape[0], w.shape[1]
    out = bias.to(h.dtype)[None, :].expand(T, -1).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j].to(h.dtype)[None, :] * h[: T - back]
    return out


# ---------------------------------------------------------------------------
# embedding and output


def embed(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64) -> torch.Tensor:
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    return weights["embed"].to(dtype)[ids] * float(config["embedding"]["scale"])


def output_logits(x: torch.Tensor, weights: Weights, config: dict) -> torch.Tensor:
    return rms_norm(x, weights["final.norm"], float(config["norm"]["eps"])) @ weights["embed"].to(x.dtype).T


# ---------------------------------------------------------------------------
# latent attention


def stretched_frequencies(base: float, dims: int, s: Optional[dict]) -> tuple[torch.Tensor, float]:
    """Turns per position of every pair, and the factor on cosines and sines."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.as_tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims)
    if s is None:
        return f, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(s["fast"]))), 0)
    hi = min(math.ceil(index_of(float(s["slow"]))), dims - 1)
    ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_halves(x: torch.Tensor, positions: Sequence[int], freq: torch.Tensor, magnitude: float) -> torch.Tensor:
    """x [T, ..., n]: entries i and i + len(freq) turn together by position * freq[i]; cosine and sine
    carry `magnitude`; entries behind the first 2 len(freq) stay."""
    half = freq.numel()
    if half == 0:
        return x
    ang = torch.as_tensor(list(positions), dtype=torch.float64)[:, None] * freq[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c = (torch.cos(ang) * magnitude).to(x.dtype).view(shape)
    s = (torch.sin(ang) * magnitude).to(x.dtype).view(shape)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def _rotation(m: dict) -> tuple[torch.Tensor, float]:
    return stretched_frequencies(float(m["rot"]["base"]), int(m["rot"]["dims"]), m["rot"].get("scaling"))


def latent_rows(h: torch.Tensor, positions: Sequence[int], m: dict, w: Weights, p: str, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """What a latent attention layer caches per token: the normed latent and the rotated key part."""
    R = int(m["kv_rank"])
    rows = h @ w[p + "dkv"].to(h.dtype).T
    return rms_norm(rows[:, :R], w[p + "dkv.norm"], eps), rotate_halves(rows[:, R:], positions, *_rotation(m))


def softmax_with_sink(scores: torch.Tensor, visible: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Rows of weights exp(s_j) / (exp(sink) + sum over the visible of exp(s)); they sum to less than one."""
    s = scores.masked_fill(~visible, float("-inf"))
    top = torch.maximum(s.amax(-1, keepdim=True), sink.to(s.dtype))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.to(s.dtype) - top))


def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (dist >= 0) if size is None else (dist >= 0) & (dist < size)


def latent_attention(h: torch.Tensor, positions: Sequence[int], m: dict, w: Weights, p: str, eps: float,
                     c: torch.Tensor, k_rot: torch.Tensor) -> torch.Tensor:
    """The mixer on the latents c and rotated key parts k_rot (its own, or another layer's)."""
    dt = h.dtype
    T, H, d, r, e = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    cq = rms_norm(h @ w[p + "dq"].to(dt).T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].to(dt).T).view(T, H, d + r)
    q_plain, q_rot = q[..., :d], rotate_halves(q[..., d:], positions, *_rotation(m))
    k_plain = (c @ w[p + "uk"].to(dt).T).view(T, H, d)
    v = (c @ w[p + "uv"].to(dt).T).view(T, H, e)
    visible = window_mask(T, None if m.get("mask") is None else int(m["mask"]["size"]))
    heads = []
    for a in range(H):
        s = (q_plain[:, a] @ k_plain[:, a].T + q_rot[:, a] @ k_rot.T) * float(m["scale"])
        heads.append(softmax_with_sink(s, visible, w[p + "sink"][a]) @ v[:, a])
    gate = torch.sigmoid(h @ w[p + "g"].to(dt).T)
    return (torch.cat(heads, dim=-1) * gate) @ w[p + "o"].to(dt).T


# ---------------------------------------------------------------------------
# gated linear recurrence


def block_gate(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """sigmoid(w[j] u_j + b[j]) on the equal parts u_j of every row; w [blocks, out, in], b [blocks, out]."""
    T, n = u.shape[0], w.shape[0]
    parts = u.view(T, n, -1)
    return torch.sigmoid(torch.stack([parts[:, j] @ w[j].to(u.dtype).T + b[j].to(u.dtype) for j in range(n)], dim=1)).reshape(T, -1)


def gated_recurrence(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """Per channel, from zero: a = exp(-8 r softplus(lam)), S <- a S + sqrt(1 - a^2) i u."""
    log_a = -8.0 * r * softplus(lam.to(u.dtype))
    a, inp = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + inp[t]
        out[t] = S
    return out


def recurrent_mixer(h: torch.Tensor, w: Weights, p: str) -> torch.Tensor:
    dt = h.dtype
    y = gelu_tanh(h @ w[p + "y"].to(dt).T + w[p + "y.b"].to(dt))
    u = causal_conv(h @ w[p + "x"].to(dt).T + w[p + "x.b"].to(dt), w[p + "conv"], w[p + "conv.b"])
    r, i = block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"])
    return (gated_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].to(dt).T


# ---------------------------------------------------------------------------
# feed-forward


def gelu_ff(h: torch.Tensor, w: Weights, p: str) -> torch.Tensor:
    dt = h.dtype
    return (gelu_tanh(h @ w[p + "gate"].to(dt).T) * (h @ w[p + "up"].to(dt).T)) @ w[p + "down"].to(dt).T


# ---------------------------------------------------------------------------
# the model


def forward_stream(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64,
                   rounding: Optional[Callable[[torch.Tensor], torch.Tensor]] = None) -> list[torch.Tensor]:
    """The residual stream [T, width] after the embedding and after every layer.  `rounding`, if
    given, is applied to what every sublayer reads (to see what a narrower number format does)."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    rd = rounding if rounding is not None else (lambda t: t)
    positions = list(range(len(tokens)))
    x = embed(tokens, weights, config, dtype)
    streams = [x]
    latents: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}
    for i, layer in enumerate(config["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = rd(rms_norm(x, weights[p + "norm1"], eps))
        if kind == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_rows(h, positions, m, weights, p + "mix.", eps)
                src = i
            y = latent_attention(h, positions, m, weights, p + "mix.", eps, *latents[int(src)])
        elif kind == "rglru":
            y = recurrent_mixer(h, weights, p + "mix.")
        else:
            raise ValueError(f"unknown mixer {kind!r}")
        x = x + mult * y
        if layer.get("mlp") is not None:
            x = x + mult * gelu_ff(rd(rms_norm(x, weights[p + "norm2"], eps)), weights, p + "mlp.")
        streams.append(x)
    return streams


def forward_logits(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64,
                   rounding: Optional[Callable[[torch.Tensor], torch.Tensor]] = None) -> torch.Tensor:
    return output_logits(forward_stream(tokens, weights, config, dtype, rounding)[-1], weights, config)
