"""Host tests of Vepevik: the plain model's mechanisms against independent restatements and against
properties the design implies, and the engine's configuration and specification (no GPU)."""

import copy
import math

import pytest
import torch

from tests.plain import vepevik_plain as plain
from tests.vepevik_configs import RANKS, VEP, VEP_LONG, random_ids, tensor_shapes, unused_tensors, vepevik_weights

CASES = [(VEP[t], RANKS[t]) for t in sorted(VEP)] + [(VEP_LONG, RANKS["long"])]


def _w(tag, seed=5, **kw):
    return {k: v.double() for k, v in vepevik_weights(VEP[tag], seed, RANKS[tag], **kw).items()}


def _randn(*shape, seed):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_convolution_against_explicit_sums():
    for taps in (1, 2, 3, 5):
        h, w = _randn(9, 4, seed=1), _randn(4, taps, seed=2)
        want = torch.zeros_like(h)
        for t in range(9):
            for j in range(taps):
                src = t - taps + 1 + j
                if src >= 0:
                    want[t] += w[:, j] * h[src]
        assert torch.allclose(plain.causal_conv(h, w), want, atol=1e-12)


def test_rotation_turns_pairs_half_a_width_apart_and_leaves_the_rest():
    x = _randn(1, 1, 7, seed=3)
    y = plain.rotate_half(x, [3], 100.0, 4)
    for i in range(2):
        a = 3 * 100.0 ** (-2 * i / 4)
        u, v = float(x[0, 0, i]), float(x[0, 0, i + 2])
        assert abs(float(y[0, 0, i]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12
        assert abs(float(y[0, 0, i + 2]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12
    assert torch.equal(y[..., 4:], x[..., 4:])
    # scores of rotated rows depend on the distance alone
    q, k = _randn(1, 1, 6, seed=4), _randn(1, 1, 6, seed=5)
    dots = [float((plain.rotate_half(q, [p], 50.0, 6) * plain.rotate_half(k, [p - 9], 50.0, 6)).sum()) for p in (9, 30, 1000)]
    assert max(dots) - min(dots) < 1e-9


def test_chunks_count_from_position_zero():
    see = plain.visible_in_chunks(range(13), 5)
    for i in range(13):
        assert see[i].nonzero().flatten().tolist() == list(range(5 * (i // 5), i + 1))
    part = plain.visible_in_chunks(range(7, 13), 5)  # rows of a prompt's later portion: the same chunks
    assert torch.equal(part, see[7:, 7:])
    assert torch.equal(plain.visible_in_chunks(range(6), None), torch.ones(6, 6, dtype=torch.bool).tril())


def test_blended_values_and_head_gates():
    W = _w("a", sharp=2.0)
    m, eps = VEP["a"]["layers"][5]["mixer"], VEP["a"]["norm"]["eps"]
    h, first = _randn(9, 96, seed=6), _randn(9, 2, 28, seed=7)
    pos = list(range(9))
    y0, own = plain.attention(h, pos, m, W, "l5.mix.", eps, None)
    y1, own1 = plain.attention(h, pos, m, W, "l5.mix.", eps, first)
    assert torch.equal(own, own1)  # what a layer hands on is its own, unblended
    # attention is linear in the values: the blend of the branches is the branch of the blend
    lam = W["l5.mix.vmix"]
    W2 = dict(W, **{"l5.mix.vmix": torch.ones((), dtype=torch.float64)})
    y2, _ = plain.attention(h, pos, m, W2, "l5.mix.", eps, first)
    assert torch.allclose(y1, (1 - lam) * y0 + lam * y2, atol=1e-12)
    # a first token sees itself alone: each head is its value times the sigmoid of its gate
    H, G, e = m["heads"], m["kv_heads"], m["vdim"]
    g = torch.sigmoid(h[0] @ W["l5.mix.g"].T)
    row = torch.cat([own[0, a // (H // G)] * g[a] for a in range(H)])
    assert torch.allclose(y0[0], row @ W["l5.mix.o"].T, atol=1e-12) and row.numel() == H * e


def test_retention_against_its_sum_form():
    q, k, v = _randn(15, 4, seed=8), _randn(15, 4, seed=9), _randn(15, 3, seed=10)
    for decay in (0.5, 0.97, 1.0):
        want = torch.stack([sum(decay ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)) for t in range(15)])
        assert torch.allclose(plain.retention_recurrence(q, k, v, decay), want, atol=1e-12)


def test_channel_delta_rule_against_the_transition_form_and_one_decay_for_all():
    T, d, e = 12, 5, 3
    q, k, v = _randn(T, d, seed=11), _randn(T, d, seed=12), _randn(T, e, seed=13)
    k = k / k.norm(dim=-1, keepdim=True)
    decay, beta = torch.sigmoid(_randn(T, d, seed=14)), torch.sigmoid(_randn(T, seed=15))
    got = plain.channel_delta_recurrence(q, k, v, decay, beta)
    S = torch.zeros(d, e, dtype=torch.float64)
    for t in range(T):  # S_t = (I - beta k k^T) diag(g) S_(t-1) + beta k v^T
        S = (torch.eye(d, dtype=torch.float64) - beta[t] * torch.outer(k[t], k[t])) @ torch.diag(decay[t]) @ S + beta[t] * torch.outer(k[t], v[t])
        assert torch.allclose(got[t], S.T @ q[t], atol=1e-12)
    # with full write strength and a unit key, what was written for a key is read back as it was written, whatever the decay
    one = torch.ones(2, dtype=torch.float64)
    again = plain.channel_delta_recurrence(k[[0, 0]], k[[0, 0]], v[:2], decay[:2], one)
    assert torch.allclose(again, v[:2], atol=1e-12)


def test_channel_decays_lie_between_zero_and_one_and_use_the_heads_rate():
    W = _w("a")
    h = _randn(20, 96, seed=16)
    g = plain.channel_decay(h, W, "l1.mix.", 4, 12)
    assert g.shape == (20, 4, 12) and bool(((g > 0) & (g < 1)).all()) and float(g.std()) > 0.02
    W2 = dict(W, **{"l1.mix.A_log": W["l1.mix.A_log"] + math.log(2.0) * torch.tensor([0, 1, 0, 0], dtype=torch.float64)})
    g2 = plain.channel_decay(h, W2, "l1.mix.", 4, 12)
    assert torch.allclose(g2[:, 1], g[:, 1] ** 2, atol=1e-12) and torch.equal(g2[:, [0, 2, 3]], g[:, [0, 2, 3]])


def test_capped_feed_forward():
    W = {"gate": torch.tensor([[1.0], [-1.0]], dtype=torch.float64), "up": torch.tensor([[1.0], [1.0]], dtype=torch.float64),
         "down": torch.eye(2, dtype=torch.float64)}
    got = plain.capped_ff(torch.tensor([[5.0], [-5.0]], dtype=torch.float64), 2.0, W, "")
    f = lambda a, b: a / (1 + math.exp(-1.702 * a)) * (b + 1)
    want = torch.tensor([[f(2.0, 2.0), f(-5.0, 2.0)], [f(-5.0, -2.0), f(2.0, -2.0)]], dtype=torch.float64)  # a gate has no lower bound
    assert torch.allclose(got, want, atol=1e-12)


def test_routing_inside_groups():
    router = {"experts": 6, "top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}}
    W = {"router": torch.eye(6, dtype=torch.float64)}
    logits = torch.tensor([[1.0, 5.0, 4.5, 4.6, 0.0, 4.9], [0.0, 0.1, 3.0, 2.9, 2.8, 2.7]], dtype=torch.float64)
    chosen, a = plain.route(logits, router, W, "")
    assert sorted(chosen[0].tolist()) == [0, 1, 5]  # group {2, 3} holds the third and fourth scores and is left out; 0 comes in with its group
    assert sorted(chosen[1].tolist()) == [2, 3, 4]
    assert torch.allclose(a.sum(-1), torch.full((2,), 2.0, dtype=torch.float64))
    s = torch.softmax(logits, -1)
    assert torch.allclose(a[0] / a[0, 0], s[0, chosen[0]] / s[0, chosen[0, 0]], atol=1e-12)
    free, b = plain.route(logits, {"experts": 6, "top": 3, "scale": 1.0}, W, "")
    assert sorted(free[0].tolist()) == [1, 3, 5] and torch.allclose(b.sum(-1), torch.ones(2, dtype=torch.float64))


@pytest.mark.parametrize("tag", sorted(VEP))
def test_a_prefix_gives_the_same_logits(tag):
    """Nothing looks ahead."""
    cfg, W = VEP[tag], _w(tag)
    ids = random_ids(cfg, 40, 9)
    whole = plain.forward_logits(ids, W, cfg)
    assert torch.allclose(whole[:23], plain.forward_logits(ids[:23], W, cfg), atol=1e-9)
    streams = plain.forward_stream(ids, W, cfg)
    assert len(streams) == len(cfg["layers"]) + 1
    row = W["embed"][ids[0]]
    assert torch.allclose(streams[0][0], row / torch.sqrt((row ** 2).mean() + cfg["norm"]["eps"]) * W["embed.norm"], atol=1e-12)


def _spec(cfg):
    from tokensprint_b200.config.registry import architecture_for

    arch = architecture_for(cfg)
    config = arch.config_from_dict(cfg)
    return config, arch.build_spec(config)


@pytest.mark.parametrize("cfg, ranks", CASES)
def test_the_engine_reads_the_configuration_and_wants_the_same_tensors(cfg, ranks):
    config, spec = _spec(cfg)
    assert config.to_dict() == cfg
    want, unused = tensor_shapes(cfg, ranks), unused_tensors(cfg)
    got = {s.name: tuple(s.shape) for s in spec.tensor_specs()}
    assert set(got) == set(want) - unused and unused <= set(spec.ignorable_tensors)
    for name, shape in got.items():
        assert len(shape) == len(want[name]) and all(g in (-1, w) for g, w in zip(shape, want[name])), name
    assert spec.lm_head is None


def test_which_layer_hands_its_values_on():
    _, spec = _spec(VEP["a"])
    mixers = [l.params["mixer"].params for l in spec.layers]
    assert mixers[0]["shares_values"] is None and mixers[0]["value_mix"] is None
    assert mixers[2]["shares_values"] is not None and mixers[2]["value_mix"] is None
    assert mixers[4]["shares_values"] is None and mixers[4]["value_mix"] is None
    assert mixers[5]["shares_values"] is None and mixers[5]["value_mix"] == (mixers[2]["shares_values"], "l5.mix.vmix")


def test_the_inner_widths_may_be_named():
    from tokensprint_b200.weights.loader import RandomSource

    cfg = VEP["b"]
    with pytest.raises(ValueError, match="a1"):
        RandomSource(_spec(cfg)[1].tensor_specs(), 1)
    named = copy.deepcopy(cfg)
    for layer in named["layers"]:
        if layer["type"] == "channel_delta":
            layer["mixer"].update(decay_rank=4, gate_rank=11)
    config, spec = _spec(named)
    assert config.to_dict() == named
    shapes = RandomSource(spec.tensor_specs(), 1).shapes()
    assert shapes["l0.mix.a1"] == (4, 72) and shapes["l3.mix.a2"] == (120, 4) and shapes["l3.mix.g2"] == (60, 11)


def test_configurations_the_engine_refuses():
    from tokensprint_b200.config.model_config import ConfigError
    from tokensprint_b200.models.vepevik import VepevikConfig

    for path, value in ((("layers", 0, "type"), "gla"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "mask", "size"), 0),
                        (("layers", 0, "mixer", "rot", "dims"), 26), (("layers", 2, "mixer", "rot", "dims"), 3), (("layers", 3, "mixer", "decay"), [0.5]),
                        (("layers", 5, "mixer", "vdim"), 24), (("layers", 1, "mlp", "router", "groups", "count"), 4),
                        (("layers", 1, "mlp", "router", "groups", "keep"), 0), (("layers", 5, "mlp", "router", "top"), 2),
                        (("layers", 0, "mlp", "kind"), "swiglu"), (("layers", 1, "mixer", "conv"), 0), (("norm", "eps"), 0.0)):
        bad = copy.deepcopy(VEP["a"])
        node = bad
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        with pytest.raises(ConfigError):
            VepevikConfig.from_dict(bad)
    for path in (("layers", 0, "mixer", "scale"), ("layers", 0, "mlp", "limit"), ("layers", 1, "mixer", "conv"), ("width",)):
        bad = copy.deepcopy(VEP["a"])
        node = bad
        for key in path[:-1]:
            node = node[key]
        del node[path[-1]]
        with pytest.raises(ConfigError):
            VepevikConfig.from_dict(bad)


def test_the_preset_is_registered():
    from tokensprint_b200.config.registry import get_model_config, get_model_family

    assert get_model_family("vepevik-w2048") == "vepevik"
    config = get_model_config("vepevik/vepevik-w2048")
    assert {l.type for l in config.layers} == {"attention", "retention", "channel_delta"} and config.blending_layers == [0, 3]
