"""Host tests of Mugulorn: the plain model's mechanisms against independent restatements and against
properties the design implies, and the engine's configuration, specification and cache plan (no GPU)."""

import copy
import math

import pytest
import torch

from tests.mugulorn_configs import MUG, MUG_LONG, mugulorn_weights, random_ids, tensor_shapes
from tests.plain import mugulorn_plain as plain


def _w(cfg, seed=5, **kw):
    return {k: v.double() for k, v in mugulorn_weights(cfg, seed, **kw).items()}


def test_convolution_against_explicit_sums():
    g = torch.Generator().manual_seed(1)
    for taps in (1, 2, 3, 5):
        h, w, b = (torch.randn(*s, generator=g, dtype=torch.float64) for s in ((9, 4), (4, taps), (4,)))
        want = b[None, :].repeat(9, 1)
        for t in range(9):
            for j in range(taps):
                src = t - taps + 1 + j
                if src >= 0:
                    want[t] += w[:, j] * h[src]
        assert torch.allclose(plain.causal_conv(h, w, b), want, atol=1e-12)
        assert torch.allclose(plain.causal_conv(h, w, b)[0], b + w[:, -1] * h[0], atol=1e-12)  # the last tap weighs the current token


def test_gelu_and_norm():
    z = torch.linspace(-6, 6, 101, dtype=torch.float64)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(plain.rms_norm(x, torch.tensor([1.0, 2.0]), 0.5), torch.tensor([[3.0, 8.0]], dtype=torch.float64) / math.sqrt(12.5 + 0.5))


def test_recurrence_against_its_closed_form():
    """S_t = sum_j (prod_{j < s <= t} a_s) b_j, and the first token is no special case."""
    g = torch.Generator().manual_seed(2)
    T, C = 13, 3
    u = torch.randn(T, C, generator=g, dtype=torch.float64)
    r, i = torch.rand(T, C, generator=g, dtype=torch.float64), torch.rand(T, C, generator=g, dtype=torch.float64)
    lam = torch.tensor([-4.0, 0.0, 3.0], dtype=torch.float64)
    got = plain.gated_recurrence(u, r, i, lam)
    a = torch.exp(-8.0 * r * torch.log(1.0 + torch.exp(lam)))
    b = torch.sqrt(1.0 - a ** 2) * i * u
    for t in range(T):
        want = sum((a[j + 1:t + 1].prod(dim=0) * b[j] for j in range(t + 1)), torch.zeros(C, dtype=torch.float64))
        assert torch.allclose(got[t], want, atol=1e-12)
    assert torch.allclose(got[0], b[0], atol=1e-15)


def test_block_gates_are_block_diagonal_products():
    g = torch.Generator().manual_seed(3)
    u, w, b = (torch.randn(*s, generator=g, dtype=torch.float64) for s in ((5, 12), (3, 4, 4), (3, 4)))
    full = torch.zeros(12, 12, dtype=torch.float64)
    for j in range(3):
        full[4 * j:4 * j + 4, 4 * j:4 * j + 4] = w[j]
    assert torch.allclose(plain.block_gate(u, w, b), torch.sigmoid(u @ full.T + b.reshape(-1)), atol=1e-12)


def test_sink_is_a_key_without_a_value():
    g = torch.Generator().manual_seed(4)
    s = torch.randn(6, 6, generator=g, dtype=torch.float64)
    visible = plain.window_mask(6, 3)
    sink = torch.tensor(0.7, dtype=torch.float64)
    got = plain.softmax_with_sink(s, visible, sink)
    wide = torch.cat([s.masked_fill(~visible, float("-inf")), torch.full((6, 1), 0.7, dtype=torch.float64)], dim=1)
    assert torch.allclose(got, torch.softmax(wide, dim=-1)[:, :6], atol=1e-12)
    assert bool((got.sum(-1) < 1).all())
    # far above every score the sink takes nearly all the weight, far below none
    assert float(plain.softmax_with_sink(s, visible, torch.tensor(80.0)).sum(-1).max()) < 1e-25
    assert torch.allclose(plain.softmax_with_sink(s, visible, torch.tensor(-80.0)).sum(-1), torch.ones(6, dtype=torch.float64))


def test_window_edges():
    cfg = MUG["a"]
    W = _w(cfg, sharp=3.0)
    m, p, eps = cfg["layers"][0]["mixer"], "l0.mix.", cfg["norm"]["eps"]
    size = m["mask"]["size"]
    h = torch.randn(size + 6, cfg["width"], generator=torch.Generator().manual_seed(3), dtype=torch.float64)
    pos = list(range(h.shape[0]))

    def out(x):
        return plain.latent_attention(h, pos, m, W, p, eps, *plain.latent_rows(x, pos, m, W, p, eps))

    base, i = out(h), size + 2
    for j, seen in ((i - size, False), (i - size + 1, True), (i, True), (i + 1, False)):
        h2 = h.clone()
        h2[j] += 1.0
        assert (float((out(h2)[i] - base[i]).abs().max()) > 1e-6) == seen


def test_stretched_frequencies_and_half_rotation():
    f, mag = plain.stretched_frequencies(1000.0, 6, {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0})
    base = [1000.0 ** (-2 * i / 6) for i in range(3)]
    index = lambda turns: 6 * math.log(32 / (2 * math.pi * turns)) / (2 * math.log(1000.0))
    lo, hi = max(math.floor(index(8.0)), 0), min(math.ceil(index(1.0)), 5)
    for i in range(3):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        assert abs(float(f[i]) - (base[i] / 4.0 * ramp + base[i] * (1 - ramp))) < 1e-15
    assert abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    x = torch.arange(1.0, 9.0, dtype=torch.float64).view(1, 1, 8)
    y = plain.rotate_halves(x, [3], torch.tensor([0.5, 0.25, 0.0], dtype=torch.float64), 2.0)
    c, s = 2.0 * math.cos(1.5), 2.0 * math.sin(1.5)
    assert abs(float(y[0, 0, 0]) - (1 * c - 4 * s)) < 1e-12 and abs(float(y[0, 0, 3]) - (4 * c + 1 * s)) < 1e-12  # 0 turns with 0 + 3
    assert torch.equal(y[0, 0, 6:], x[0, 0, 6:])  # entries behind the rotated ones stay


def test_latent_attention_equals_its_absorbed_form():
    """Scores against the latent through U_k^T q, values through U_v on the weighted latent: what an engine may compute instead."""
    cfg = MUG["a"]
    W = _w(cfg)
    m, p, eps = cfg["layers"][0]["mixer"], "l0.mix.", cfg["norm"]["eps"]
    T = 27
    h = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(4), dtype=torch.float64)
    pos = list(range(T))
    c, kr = plain.latent_rows(h, pos, m, W, p, eps)
    want = plain.latent_attention(h, pos, m, W, p, eps, c, kr)
    H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = plain.rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).view(T, H, d + r)
    qr = plain.rotate_halves(q[..., d:], pos, *plain.stretched_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling")))
    uk, uv = W[p + "uk"].view(H, d, R), W[p + "uv"].view(H, e, R)
    heads = []
    for a in range(H):
        s = ((q[:, a, :d] @ uk[a]) @ c.T + qr[:, a] @ kr.T) * m["scale"]
        wts = plain.softmax_with_sink(s, plain.window_mask(T, m["mask"]["size"]), W[p + "sink"][a])
        heads.append((wts @ c) @ uv[a].T)
    gated = torch.cat(heads, -1) * torch.sigmoid(h @ W[p + "g"].T)
    assert torch.allclose(gated @ W[p + "o"].T, want, atol=1e-10)


@pytest.mark.parametrize("tag", sorted(MUG))
def test_a_prefix_gives_the_same_logits(tag):
    """Nothing looks ahead: convolutions, windows and recurrences see earlier tokens only."""
    cfg = MUG[tag]
    W = _w(cfg)
    ids = random_ids(cfg, 40, 9)
    whole = plain.forward_logits(ids, W, cfg)
    assert torch.allclose(whole[:23], plain.forward_logits(ids[:23], W, cfg), atol=1e-9)
    assert len(plain.forward_stream(ids, W, cfg)) == len(cfg["layers"]) + 1


def test_the_multiplier_and_the_embedding_scale():
    cfg = copy.deepcopy(MUG["e"])
    W = _w(cfg)
    ids = random_ids(cfg, 9, 1)
    x = W["embed"][torch.tensor(ids)] * 2.0
    h = plain.rms_norm(x, W["l0.norm1"], cfg["norm"]["eps"])
    x = x + 0.5 * plain.recurrent_mixer(h, W, "l0.mix.")
    x = x + 0.5 * plain.gelu_ff(plain.rms_norm(x, W["l0.norm2"], cfg["norm"]["eps"]), W, "l0.mlp.")
    assert torch.allclose(plain.forward_stream(ids, W, cfg)[1], x, atol=1e-12)
    cfg["embedding"]["scale"] = 7.0  # the output matrix is the table without its scale
    last = plain.forward_stream(ids, W, cfg)[-1]
    assert torch.allclose(plain.forward_logits(ids, W, cfg), plain.rms_norm(last, W["final.norm"], cfg["norm"]["eps"]) @ W["embed"].T, atol=1e-12)


@pytest.mark.parametrize("cfg", list(MUG.values()) + [MUG_LONG])
def test_the_engine_reads_the_configuration_and_wants_the_same_tensors(cfg):
    import tokensprint_b200.models  # noqa: F401
    from tokensprint_b200.config.registry import ARCHITECTURES

    arch = ARCHITECTURES["Mugulorn"]
    config = arch.config_from_dict(cfg)
    assert config.to_dict() == cfg
    spec = arch.build_spec(config)
    assert {s.name: tuple(s.shape) for s in spec.tensor_specs()} == tensor_shapes(cfg)
    for i, layer in enumerate(cfg["layers"]):
        if layer["mixer"].get("kv_from") is not None:
            run = spec.run_order[i]
            assert run.cache == layer["mixer"]["kv_from"] and not run.writes_cache


def test_a_shared_cache_serves_the_longest_window_of_its_readers():
    from tokensprint_b200.config.registry import ARCHITECTURES
    from tokensprint_b200.models.model import Model

    def windows(cfg):
        arch = ARCHITECTURES["Mugulorn"]
        model = Model(arch.build_spec(arch.config_from_dict(cfg)), "cpu", torch.float32)
        return [(e.need.kind, e.need.window) for e in model.cache_plan if e.need.kind != "none"]

    assert windows(MUG["a"]) == [("window", 33), ("full", 0)]  # 20 and a reader of 33; none and a reader of 7
    assert windows(MUG["b"]) == [("full", 0)]                  # 11 and a reader without a window
    assert windows(MUG["c"]) == [("window", 100), ("window", 1)]
    assert windows(MUG["e"]) == []


def test_needs_that_cannot_share_a_cache():
    from tokensprint_b200.parts.base import CacheNeed

    a = CacheNeed(kind="window", window=8, k_row=(12,), single_pool=True)
    assert a.covering(CacheNeed(kind="window", window=3, k_row=(12,), single_pool=True)).window == 8
    assert a.covering(CacheNeed(kind="full", k_row=(12,), single_pool=True)).kind == "full"
    with pytest.raises(ValueError):
        a.covering(CacheNeed(kind="window", window=8, k_row=(13,), single_pool=True))
    with pytest.raises(ValueError):
        a.covering(CacheNeed(kind="chunk", window=8, k_row=(12,), single_pool=True))


def test_configurations_the_engine_refuses():
    from tokensprint_b200.config.model_config import ConfigError
    from tokensprint_b200.models.mugulorn import MugulornConfig

    def refused(change):
        bad = copy.deepcopy(MUG["a"])
        change(bad)
        with pytest.raises(ConfigError):
            MugulornConfig.from_dict(bad)

    refused(lambda c: c["layers"][2]["mixer"].update(kv_from=1))       # a recurrent layer caches no latent rows
    refused(lambda c: c["layers"][2]["mixer"].update(kv_from=3))       # a later layer
    refused(lambda c: c["layers"][5]["mixer"].update(kv_from=2))       # a reader has no rows of its own (and another latent width)
    refused(lambda c: c["layers"][2]["mixer"].update(kv_rank=24))      # another latent width than its source's
    refused(lambda c: c["layers"][2]["mixer"]["rot"].update(base=7.0)) # another rotation
    refused(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    refused(lambda c: c["layers"][1]["mixer"].update(blocks=7))        # 60 channels in 7 parts
    refused(lambda c: c["layers"][1].update(type="delta"))
    refused(lambda c: c["layers"][1]["mlp"].update(kind="moe"))
    refused(lambda c: c.pop("residual_mult"))
