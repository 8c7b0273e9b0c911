"""Plain, slow Vepevik: whole sequences, no cache, one function per mechanism.

Vepevik is a decoder-only model of pre-normed layers over a normed embedding, with tied logits:

    x = N_embed(embed[token]);   x <- x + mixer(N1(x));   x <- x + ff(N2(x))     (the last where a layer has one)
    logits = embed . N_final(x)

A layer's mixer is one of three.  "attention": grouped-query softmax attention inside chunks of
positions, normed and partly rotated q and k, values that blend with those of the first blending
layer, a sigmoid gate per head.  "retention": a linear recurrence over rotated q and k with one
constant decay per head, a norm per head without weight and a silu gate.  "channel_delta": the gated
delta rule with a decay per head and key channel that passes a narrow pair of matrices, as does the
sigmoid output gate.  The feed-forward is a dense gated one with capped operands or a set of routed
SwiGLU experts, chosen inside the best groups of experts by softmax scores.

Everything here runs on whole sequences in one dtype (float64 by default) on the CPU and shares
no code with the engine under test.  `config` is the content of a config.json as a dict,
`weights` a dict of tensors under the checkpoint's names.
"""

from __future__ import annotations

from typing import Callable, Mapping, Optional, Sequence

import torch

Weights = Mapping[str, torch.Tensor]


# ---------------------------------------------------------------------------
# small functions


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Rows divided by their root mean square, eps under the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w.to(x.dtype)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(z, torch.zeros_like(z))


def project(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h @ w.to(h.dtype).T


def causal_conv(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h [T, C], w [C, taps]: out_t = sum_j w[:, j] h_(t - taps + 1 + j); rows before the start are zeros
    (the last column weighs the current token)."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j].to(h.dtype)[None, :] * h[: T - back]
    return out


def rotate_half(x: torch.Tensor, positions: Sequence[int], base: float, dims: int) -> torch.Tensor:
    """x [T, heads, n]: entries i and i + dims/2 (i < dims/2) turn together by position * base^(-2i/dims);
    the entries from `dims` on stay."""
    if dims == 0:
        return x
    half = dims // 2
    freq = torch.as_tensor(float(base), dtype=torch.float64) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    ang = torch.as_tensor(list(positions), dtype=torch.float64)[:, None, None] * freq
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def rotate(x: torch.Tensor, positions: Sequence[int], m: dict) -> torch.Tensor:
    rot = m.get("rot")
    return x if rot is None else rotate_half(x, positions, float(rot["base"]), int(rot["dims"]))


# ---------------------------------------------------------------------------
# embedding and output


def embed(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64) -> torch.Tensor:
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    return rms_norm(weights["embed"].to(dtype)[ids], weights["embed.norm"], float(config["norm"]["eps"]))


def output_logits(x: torch.Tensor, weights: Weights, config: dict) -> torch.Tensor:
    return project(rms_norm(x, weights["final.norm"], float(config["norm"]["eps"])), weights["embed"])


# ---------------------------------------------------------------------------
# attention inside chunks


def visible_in_chunks(positions: Sequence[int], size: Optional[int]) -> torch.Tensor:
    """[query, key]: not later, and (with a size) in the same chunk of `size` positions."""
    pos = torch.as_tensor(list(positions), dtype=torch.long)
    see = pos[None, :] <= pos[:, None]
    if size:
        see = see & (pos[None, :] // size == pos[:, None] // size)
    return see


def blend_values(v: torch.Tensor, first: torch.Tensor, share: torch.Tensor) -> torch.Tensor:
    lam = share.to(v.dtype).reshape(())
    return (1.0 - lam) * v + lam * first


def attention(h: torch.Tensor, positions: Sequence[int], m: dict, w: Weights, p: str, eps: float,
              first_values: Optional[torch.Tensor]) -> tuple[torch.Tensor, torch.Tensor]:
    """Returns the branch and the layer's own values [T, G, e] before any blending."""
    T, H, G, d, e = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(rms_norm(project(h, w[p + "q"]).view(T, H, d), w[p + "q.norm"], eps), positions, m)
    k = rotate(rms_norm(project(h, w[p + "k"]).view(T, G, d), w[p + "k.norm"], eps), positions, m)
    own = project(h, w[p + "v"]).view(T, G, e)
    v = own if first_values is None else blend_values(own, first_values, w[p + "vmix"])
    see = visible_in_chunks(positions, int(m["mask"]["size"]) if m.get("mask") is not None else None)
    gate = torch.sigmoid(project(h, w[p + "g"]))
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(m["scale"])
        heads.append(torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, g] * gate[:, a:a + 1])
    return project(torch.cat(heads, dim=-1), w[p + "o"]), own


# ---------------------------------------------------------------------------
# retention


def retention_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: float) -> torch.Tensor:
    """One head: S <- decay S + k v^T, o = S^T q, S zero before the first token."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def retention(h: torch.Tensor, positions: Sequence[int], m: dict, w: Weights, p: str, eps: float) -> torch.Tensor:
    T, H, d, e = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(project(h, w[p + "q"]).view(T, H, d), positions, m)
    k = rotate(project(h, w[p + "k"]).view(T, H, d), positions, m) * d ** -0.5
    v = project(h, w[p + "v"]).view(T, H, e)
    heads = [unit_rms(retention_recurrence(q[:, a], k[:, a], v[:, a], float(m["decay"][a])), eps) for a in range(H)]
    return project(torch.cat(heads, dim=-1) * silu(project(h, w[p + "g"])), w[p + "o"])


# ---------------------------------------------------------------------------
# delta rule with a decay per key channel


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def channel_delta_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """One head.  q, k, decay [T, d], v [T, e], beta [T].  S [d, e] starts at zero; per token:
    S <- diag(decay) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def channel_decay(h: torch.Tensor, w: Weights, p: str, heads: int, dim: int) -> torch.Tensor:
    """[T, heads, dim]: exp(-exp(A_log) softplus(a2 a1 h + dt_bias))."""
    z = project(project(h, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"].to(h.dtype)
    return torch.exp(-torch.exp(w[p + "A_log"].to(h.dtype))[None, :, None] * softplus(z).view(h.shape[0], heads, dim))


def channel_delta(h: torch.Tensor, m: dict, w: Weights, p: str, eps: float) -> torch.Tensor:
    T, H, G, d, e = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])

    def short(name: str) -> torch.Tensor:
        return silu(causal_conv(project(h, w[p + name]), w[p + name + ".conv"]))

    q = unit_length(short("q").view(T, G, d)) * d ** -0.5
    k = unit_length(short("k").view(T, G, d))
    v = short("v").view(T, H, e)
    beta = torch.sigmoid(project(h, w[p + "b"]))
    decay = channel_decay(h, w, p, H, d)
    gate = torch.sigmoid(project(project(h, w[p + "g1"]), w[p + "g2"])).view(T, H, e)
    heads = []
    for a in range(H):
        g = a // (H // G)
        o = channel_delta_recurrence(q[:, g], k[:, g], v[:, a], decay[:, a], beta[:, a])
        heads.append(rms_norm(o, w[p + "norm"], eps) * gate[:, a])
    return project(torch.cat(heads, dim=-1), w[p + "o"])


# ---------------------------------------------------------------------------
# feed-forwards


def capped_ff(h: torch.Tensor, limit: float, w: Weights, p: str) -> torch.Tensor:
    a = torch.clamp(project(h, w[p + "gate"]), max=limit)
    b = torch.clamp(project(h, w[p + "up"]), -limit, limit)
    return project(a * torch.sigmoid(1.702 * a) * (b + 1.0), w[p + "down"])


def route(h: torch.Tensor, router: dict, w: Weights, p: str) -> tuple[torch.Tensor, torch.Tensor]:
    """Chosen experts [T, top] and their weights: softmax scores; only experts of the groups whose
    best member scores highest may be chosen; the chosen scores over their sum, times a constant."""
    s = torch.softmax(project(h, w[p + "router"]), dim=-1)
    E, groups = int(router["experts"]), router.get("groups")
    allowed = torch.ones_like(s, dtype=torch.bool)
    if groups is not None:
        n, keep = int(groups["count"]), int(groups["keep"])
        best = torch.stack([s[:, j * (E // n):(j + 1) * (E // n)].max(dim=-1).values for j in range(n)], dim=-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter(1, torch.topk(best, keep, dim=-1).indices, True)
        allowed = kept.repeat_interleave(E // n, dim=-1)
    chosen = torch.topk(s.masked_fill(~allowed, -1.0), int(router["top"]), dim=-1).indices
    a = torch.gather(s, 1, chosen)
    return chosen, a / (a.sum(-1, keepdim=True) + 1e-20) * float(router["scale"])


def routed_ff(h: torch.Tensor, mlp: dict, w: Weights, p: str, chosen: Optional[torch.Tensor] = None,
              weights: Optional[torch.Tensor] = None) -> torch.Tensor:
    if chosen is None:
        chosen, weights = route(h, mlp["router"], w, p)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t].tolist(), weights[t]):
            pe = f"{p}e{e}."
            out[t] += a * project(silu(project(h[t], w[pe + "gate"])) * project(h[t], w[pe + "up"]), w[pe + "down"])
    return out


# ---------------------------------------------------------------------------
# the model


def forward_stream(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64,
                   rounding: Optional[Callable[[torch.Tensor], torch.Tensor]] = None) -> list[torch.Tensor]:
    """The residual stream [T, width] after the embedding and after every layer.  `rounding`, if
    given, is applied to what every sublayer reads (to see what a narrower number format does)."""
    eps = float(config["norm"]["eps"])
    rd = rounding if rounding is not None else (lambda t: t)
    positions = list(range(len(tokens)))
    x = embed(tokens, weights, config, dtype)
    streams = [x]
    first_values: Optional[torch.Tensor] = None
    for i, layer in enumerate(config["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = rd(rms_norm(x, weights[p + "norm1"], eps))
        if kind == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, positions, m, weights, p + "mix.", eps, first_values if mixes else None)
            if mixes and first_values is None:
                first_values = own
        elif kind == "retention":
            y = retention(h, positions, m, weights, p + "mix.", eps)
        elif kind == "channel_delta":
            y = channel_delta(h, m, weights, p + "mix.", eps)
        else:
            raise ValueError(f"unknown mixer {kind!r}")
        x = x + y
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rd(rms_norm(x, weights[p + "norm2"], eps))
            if mlp["kind"] == "dense":
                x = x + capped_ff(h, float(mlp["limit"]), weights, p + "mlp.")
            else:
                x = x + routed_ff(h, mlp, weights, p + "mlp.")
        streams.append(x)
    return streams


def forward_logits(tokens: Sequence[int], weights: Weights, config: dict, dtype=torch.float64,
                   rounding: Optional[Callable[[torch.Tensor], torch.Tensor]] = None) -> torch.Tensor:
    return output_logits(forward_stream(tokens, weights, config, dtype, rounding)[-1], weights, config)
