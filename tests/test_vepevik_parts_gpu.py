"""The mechanisms of Vepevik one at a time: each kernel and each mixer part against the plain
function of the same mechanism, whole prompts, portions down to one token, batches of unequal
sequences with slots and pages in any order and used again; inputs made so that a key just inside
or just outside a chunk, a far key, a value blended with another token's, a lost kept input or a state
that was not carried shows far beyond rounding."""

import pytest
import torch

from tests.plain import vepevik_plain as plain
from tests.mixer_harness import Harness, batch as _batch, dev as _dev, i32 as _i32, in_portions as _in_portions, inputs as _inputs, rand as _rand, rel as _rel
from tests.vepevik_configs import RANKS, VEP, VEP_LONG, vepevik_weights

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}


def _cfg(tag):
    return VEP_LONG if tag == "long" else VEP[tag]


# ---------------------------------------------------------------------------
# kernels alone


DELTA_SHAPES = [(1, 1, 7, 5), (6, 3, 20, 10), (2, 2, 64, 64), (4, 2, 128, 32), (3, 3, 9, 14), (2, 1, 256, 20), (2, 2, 1, 4), (1, 1, 520, 6)]


def _delta_inputs(H, G, d, e, T, seed):
    x = _rand((T, 2 * G * d + H * e), seed)
    beta, z = _rand((T, H), seed + 1), _rand((T, H * d), seed + 2) - 1.0
    a_log, dt_bias = 0.3 + 0.3 * _rand((H,), seed + 3), -1.5 + _rand((H * d,), seed + 4)
    return x, beta, z, a_log, dt_bias


def _delta_plain(x, beta, z, a_log, dt_bias, H, G, d, e):
    T = x.shape[0]
    x, z = x.double(), z.double()
    q = plain.unit_length(x[:, :G * d].view(T, G, d)) * d ** -0.5
    k = plain.unit_length(x[:, G * d:2 * G * d].view(T, G, d))
    v = x[:, 2 * G * d:].view(T, H, e)
    decay = torch.exp(-torch.exp(a_log.double())[None, :, None] * plain.softplus(z + dt_bias.double()).view(T, H, d))
    b = torch.sigmoid(beta.double())
    return torch.cat([plain.channel_delta_recurrence(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], decay[:, a], b[:, a]) for a in range(H)], -1)


def _delta_run(data, state, slots, lengths, H, G, d, e, ahead, beta_dtype=torch.float32):
    """`ahead`: the decays in a kernel of their own before the scan; else in the scan.  beta and z are column ranges."""
    from tokensprint_b200 import ops

    x, beta, z, a_log, dt_bias = data
    cu, _ = _batch(lengths)
    wide = torch.cat([_rand((z.shape[0], 3), 99), z], dim=1)
    rows, betas = _dev(wide)[:, 3:], _dev(torch.cat([beta, beta], dim=1), beta_dtype)[:, H:]
    a_log, dt_bias = _dev(a_log), _dev(dt_bias)
    if ahead:
        ops.channel_decay(rows, a_log, dt_bias, H, d)
        a_log = dt_bias = None
    out = torch.empty((x.shape[0], H * e), device="cuda")
    ops.delta_scan(_dev(x), 0, G * d, 2 * G * d, betas, rows, a_log, dt_bias, state, _i32(slots), cu, out, len(lengths), H, G, d, e, d ** -0.5, 1e-6,
                   max_seqlen=max(lengths))
    return out.cpu()


@pytest.mark.parametrize("ahead", [False, True])
@pytest.mark.parametrize("H, G, d, e", DELTA_SHAPES)
def test_channel_delta_scan_whole_in_portions_and_token_by_token(H, G, d, e, ahead):
    T = 150
    data = _delta_inputs(H, G, d, e, T, 10 * d + e)
    want = _delta_plain(*data, H, G, d, e)
    floats = H * d * e
    for sizes in ([T], [1, 2, 7, 1, 33, 2, 64, 3, 37], [1] * 40 + [110]):
        state = torch.zeros((4, floats + 3), device="cuda")  # a row stride that is no multiple of four
        got, at = [], 0
        for n in sizes:
            part = tuple(t[at:at + n] for t in data[:3]) + data[3:]
            got.append(_delta_run(part, state, [2], [n], H, G, d, e, ahead))
            at += n
        assert _rel(torch.cat(got), want) < 3e-5, (sizes[:3], H, G, d, e)
        assert float(state[[0, 1, 3]].abs().max()) == 0.0 and float(state[2, floats:].abs().max()) == 0.0  # nobody else's slot, nothing behind the state


@pytest.mark.parametrize("H, G, d, e", [(6, 3, 20, 10), (2, 2, 64, 64)])
def test_channel_delta_scan_many_sequences_side_by_side_against_each_alone(H, G, d, e):
    """Forty sequences of unequal length (one of them empty: a padded lane) in one launch, their slots in
    any order, write strengths in bfloat16: each as it is alone."""
    lengths = [(7 * i) % 23 + (0 if i == 5 else 1) for i in range(40)]
    lengths[5] = 0
    data = [_delta_inputs(H, G, d, e, max(n, 1), 100 + 7 * i) for i, n in enumerate(lengths)]
    a_log, dt_bias = data[0][3], data[0][4]
    state = torch.zeros((40, H * d * e), device="cuda")
    slots = [(3 * i) % 40 for i in range(40)]  # 3 and 40 have no common factor: every slot once
    state[slots[5]] = 7.0  # the empty lane's slot must stay as it is
    x, beta, z = (torch.cat([data[i][j][:n] for i, n in enumerate(lengths)]) for j in range(3))
    beta = beta.to(torch.bfloat16).float()
    got = _delta_run((x, beta, z, a_log, dt_bias), state, slots, lengths, H, G, d, e, False, torch.bfloat16)
    at = 0
    for i, n in enumerate(lengths):
        if n:
            want = _delta_plain(x[at:at + n], beta[at:at + n], z[at:at + n], a_log, dt_bias, H, G, d, e)
            assert _rel(got[at:at + n], want) < 3e-5, i
        at += n
    assert float((state[slots[5]] - 7.0).abs().max()) == 0.0


def test_a_channel_that_forgets_at_once_and_one_that_never_does():
    """Decays of exactly zero and one (rates beyond float32's reach): rows of the state that are wiped and rows that stay."""
    H, G, d, e, T = 1, 1, 8, 4, 60
    x, beta, z, a_log, dt_bias = _delta_inputs(H, G, d, e, T, 5)
    z[:, :3], z[:, 3:6] = 300.0, -300.0
    data = (x, beta, z, a_log, dt_bias)
    want = _delta_plain(*data, H, G, d, e)
    for ahead in (False, True):
        for n in (T, 1):
            state = torch.zeros((1, H * d * e), device="cuda")
            got = torch.cat([_delta_run(tuple(t[i:i + n] for t in data[:3]) + data[3:], state, [0], [min(n, T - i)], H, G, d, e, ahead)
                             for i in range(0, T, n)])
            assert _rel(got, want) < 3e-5, (ahead, n)


RETENTION_SHAPES = [([0.9], 7, 5, 6), ([0.5, 1.0, 0.97], 20, 11, 8), ([0.99, 0.75], 64, 64, 64), ([0.998] * 4, 130, 36, 0), ([0.9, 0.99], 15, 20, 2),
                    ([0.96875], 60, 33, 34), ([0.9], 128, 40, 128), ([0.5, 0.99], 100, 17, 70), ([0.99], 300, 24, 260), ([0.9, 1.0], 2, 70, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay, d, e, rot", RETENTION_SHAPES)
def test_retention_scan_whole_in_portions_and_token_by_token(decay, d, e, rot, dtype):
    """Rows that are rotated as they are read (all of a head, its first entries, none) against the plain recurrence."""
    from tokensprint_b200 import ops

    H, T = len(decay), 1100
    proj = _rand((T, H * (2 * d + e) + 5), d + e).to(dtype)
    q, k, v = (proj[:, a:b].double().view(T, H, -1) for a, b in ((0, H * d), (H * d, 2 * H * d), (2 * H * d, H * (2 * d + e))))
    pos = list(range(T))
    qr, kr = plain.rotate_half(q, pos, 100.0, rot), plain.rotate_half(k, pos, 100.0, rot)
    want = torch.cat([plain.retention_recurrence(qr[:, a], kr[:, a] * d ** -0.5, v[:, a], decay[a]) for a in range(H)], -1)
    inv = torch.as_tensor(100.0, dtype=torch.float64) ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    constants = torch.tensor(decay, dtype=torch.float32, device="cuda")
    rows = _dev(proj)
    for sizes in ((T,), (1, 2, 600, 1, 1, 31), (1,)):
        state, out, at, i = torch.zeros((3, H * d * e + 2), device="cuda"), [], 0, 0
        while at < T and not (sizes == (1,) and at >= 120):
            n = min(sizes[i % len(sizes)], T - at)
            table = ops.rope_table(_i32(pos[at:at + n]), _dev(inv), 1.0, n) if rot else None
            o = torch.empty((n, H * e), device="cuda")
            ops.retention_scan(rows[at:at + n], 0, H * d, 2 * H * d, table, constants, d ** -0.5, state, _i32([1]), _i32([0, n]), o, 1, H, H, d, e,
                               max_seqlen=n)
            out.append(o.cpu())
            at, i = at + n, i + 1
        got = torch.cat(out)
        assert _rel(got, want[:got.shape[0]]) < 5e-5, sizes
        assert float(state[[0, 2]].abs().max()) == 0.0 and float(state[1, H * d * e:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, e, rot", [(6, 2, 12, 10, 4), (4, 4, 64, 64, 64), (4, 1, 40, 70, 0)])
def test_retention_scan_many_sequences_side_by_side_against_each_alone(H, G, d, e, rot, dtype):
    """Thirty sequences of unequal length (one of them empty) in one launch, q and k heads shared by groups of value heads,
    slots in any order; then one more token of each."""
    from tokensprint_b200 import ops

    lengths = [(7 * i) % 23 + 1 for i in range(30)]
    lengths[5] = 0
    decay = [1.0 - 0.5 ** (h + 1) for h in range(H)]
    xs = [_rand((n + 1, 2 * G * d + H * e), 200 + i).to(dtype) for i, n in enumerate(lengths)]
    want = []
    for x in xs:
        p, pos = x.double(), list(range(x.shape[0]))
        q, k = (plain.rotate_half(p[:, a:a + G * d].view(-1, G, d), pos, 50.0, rot) for a in (0, G * d))
        v = p[:, 2 * G * d:].view(-1, H, e)
        want.append(torch.cat([plain.retention_recurrence(q[:, a // (H // G)] * d ** -0.5, k[:, a // (H // G)], v[:, a], decay[a]) for a in range(H)], -1))
    state = torch.zeros((30, H * d * e), device="cuda")
    slots = [(7 * i) % 30 for i in range(30)]
    state[slots[5]] = 3.0
    inv = torch.as_tensor(50.0, dtype=torch.float64) ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    for first in (True, False):
        parts = [(0, n) if first else (n, n + 1) for n in lengths]
        if not first:
            parts[5] = (0, 0)
        rows = torch.cat([x[a:b] for x, (a, b) in zip(xs, parts)])
        pos = [t for a, b in parts for t in range(a, b)]
        cu, _ = _batch([b - a for a, b in parts])
        out = torch.empty((rows.shape[0], H * e), device="cuda")
        table = ops.rope_table(_i32(pos), _dev(inv), 1.0, len(pos)) if rot else None
        ops.retention_scan(_dev(rows), 0, G * d, 2 * G * d, table, torch.tensor(decay, device="cuda"), d ** -0.5, state, _i32(slots), cu, out, 30, H, G,
                           d, e, max_seqlen=max(b - a for a, b in parts))
        assert _rel(out.cpu(), torch.cat([w[a:b] for w, (a, b) in zip(want, parts)])) < 3e-5, first
    assert float((state[slots[5]] - 3.0).abs().max()) == 0.0  # the empty lane's slot


@pytest.mark.parametrize("dtype", DTYPES)
def test_norms_rotation_and_blended_values_between_projection_and_cache(dtype):
    from tokensprint_b200 import ops

    T, nq, nkv, d, e, D, rot, eps, share = 13, 3, 2, 10, 14, 16, 6, 1e-3, 0.3
    width = nq * d + nkv * d + nkv * e
    proj, first = _rand((T, width + 3), 1).to(dtype), _rand((T, nkv * e + 2), 2).to(dtype)
    qn, kn = 1.0 + 0.3 * _rand((d,), 3), 1.0 + 0.3 * _rand((d,), 4)
    pos = [5 + 3 * t for t in range(T)]
    inv = torch.as_tensor(30.0, dtype=torch.float64) ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)
    table = ops.rope_table(_i32(pos), _dev(inv), 1.0, T)
    p = proj.double()
    want_q = plain.rotate_half(plain.rms_norm(p[:, :nq * d].view(T, nq, d), qn, eps), pos, 30.0, rot)
    want_k = plain.rotate_half(plain.rms_norm(p[:, nq * d:nq * d + nkv * d].view(T, nkv, d), kn, eps), pos, 30.0, rot)
    own = p[:, nq * d + nkv * d:width].view(T, nkv, e)
    slots = [(5 * t) % 17 for t in range(T)]
    slots[4] = -1  # a token whose keys are not kept
    rows = _dev(proj)
    for blend in (False, True):
        want_v = plain.blend_values(own, first[:, :nkv * e].double().view(T, nkv, e), torch.tensor(share, dtype=torch.float64)) if blend else own
        k = torch.full((17, nkv, D), 7.0, device="cuda", dtype=dtype)
        v = torch.full_like(k, 7.0)
        q = torch.empty((T, nq * D), device="cuda", dtype=dtype)
        ops.qkv_prepare(rows, 0, nq * d, nq * d + nkv * d, None, None, None, table, False, eps, q, k, v, _i32(slots), nq, nkv, d, e, D,
                        q_norm=_dev(qn), k_norm=_dev(kn), first_values=_dev(first)[:, :nkv * e] if blend else None, value_share=share)
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        kept = [t for t in range(T) if slots[t] >= 0]
        at = torch.tensor([slots[t] for t in kept])
        q = q.view(T, nq, D).cpu()
        assert _rel(q[..., :d], want_q) < tol and float(q[..., d:].abs().max()) == 0.0
        assert _rel(k.cpu()[at][..., :d], want_k[kept]) < tol and float(k.cpu()[at][..., d:].abs().max()) == 0.0
        assert _rel(v.cpu()[at][..., :e], want_v[kept]) < tol and float(v.cpu()[at][..., e:].abs().max()) == 0.0
        untouched = [s for s in range(17) if s not in slots]
        assert float((k.cpu()[untouched].float() - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, H, e, D", [(7, 5, 12, 16), (9, 2, 64, 64), (3, 3, 9, 9), (70, 3, 40, 40)])
def test_one_gate_per_head(T, H, e, D, dtype):
    from tokensprint_b200 import ops

    a, gate = _rand((T, H, D), 1).to(dtype), _rand((T, H + 4), 2).to(dtype)
    out = torch.empty((T, H * e), device="cuda", dtype=dtype)
    ops.gate_rows(_dev(a), _dev(gate)[:, 3:3 + H], out, H, e, D, per_head=True)
    want = (a[..., :e].double() * torch.sigmoid(gate[:, 3:3 + H].double())[..., None]).reshape(T, H * e)
    assert _rel(out.cpu(), want) < (1e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("activation", ["silu", "sigmoid"])
@pytest.mark.parametrize("weighted", [True, False])
@pytest.mark.parametrize("gate_dtype, dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.float32, torch.bfloat16)])
def test_head_norm_and_gate(activation, weighted, gate_dtype, dtype):
    from tokensprint_b200 import ops

    for T, H, e in ((11, 3, 10), (5, 2, 64), (4, 1, 132)):
        o, gate, w = _rand((T, H * e), 1), _rand((T, H * e + 8), 2).to(gate_dtype), 1.0 + 0.3 * _rand((e,), 3)
        out = torch.empty((T, H * e), device="cuda", dtype=dtype)
        ops.gla_norm_gate(_dev(o), _dev(gate)[:, 8:], _dev(w) if weighted else None, out, H, e, 1e-4, activation=activation)
        g = gate[:, 8:].double()
        y = plain.unit_rms(o.double().view(T, H, e), 1e-4) * (w.double() if weighted else 1.0)
        want = y.reshape(T, H * e) * (plain.silu(g) if activation == "silu" else torch.sigmoid(g))
        assert _rel(out.cpu(), want) < (1e-5 if dtype == torch.float32 else 1e-2), (T, H, e)


def _clear_choice(s, top, groups, margin):
    """Tokens (rows of scores s) whose choice and its order hang on no difference below `margin`: between the last group
    kept and the first left out, between the chosen experts and between the last of them and the next allowed one."""
    T, E = s.shape
    count, keep = groups if groups is not None else (1, 1)
    best = s.view(T, count, E // count).max(-1).values
    clear = torch.ones(T, dtype=torch.bool)
    if keep < count:
        ranked = best.sort(-1, descending=True).values
        clear = (ranked[:, keep - 1] - ranked[:, keep]) > margin
    kept = torch.zeros_like(best, dtype=torch.bool).scatter(1, best.topk(keep, -1).indices, True).repeat_interleave(E // count, -1)
    ranked = s.masked_fill(~kept, -1.0).sort(-1, descending=True).values[:, :top + 1]
    return clear & ((ranked[:, :-1] - ranked[:, 1:]).min(-1).values > margin) if ranked.shape[1] > 1 else clear


@pytest.mark.parametrize("E, top, count, keep, scale", [(8, 2, 4, 2, 1.0), (12, 3, 3, 1, 2.5), (6, 4, 6, 5, 0.5), (40, 4, 5, 3, 1.7), (5, 2, 1, 1, 3.0), (66, 6, 33, 10, 1.0)])
def test_router_with_groups_of_experts(E, top, count, keep, scale):
    from tokensprint_b200 import ops

    for T in (1, 60, 2100):
        rows, router = _rand((T, 44), 1), _rand((E, 44), 2) * 0.4
        spec = {"experts": E, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}
        want_ids, want_w = plain.route(rows.double(), spec, {"router": router.double()}, "")
        s = torch.softmax(rows.double() @ router.double().T, -1)
        clear = _clear_choice(s, top, (count, keep), 1e-6)
        assert float(clear.float().mean()) > 0.8
        for use_topk in (False, True):
            ids = torch.empty((T, top), device="cuda", dtype=torch.int32)
            wts = torch.empty((T, top), device="cuda")
            if use_topk:
                ops.router_topk(_dev((rows.double() @ router.double().T).float()), top, True, ids, wts, score="softmax_all", groups=(count, keep), scale=scale)
            else:
                ops.router(_dev(rows), _dev(router), top, True, ids, wts, score="softmax_all", groups=(count, keep), scale=scale)
            assert torch.equal(ids.cpu().long()[clear], want_ids[clear])
            assert _rel(wts.cpu()[clear], want_w[clear]) < 1e-5
    with pytest.raises(ops.KernelError):
        ops.router(_dev(rows), _dev(router), top, True, ids, wts, score="softmax_all", groups=(E + 1, 1))


def test_the_norm_on_the_embedding_rows():
    from tokensprint_b200.parts.base import BuildContext, PartSpec, build_part

    for width in (100, 256):
        part = build_part("transform", PartSpec("rmsnorm", {"dim": width, "eps": 1e-3, "weight": "w"}), BuildContext(torch.device("cuda"), torch.bfloat16))
        w, x = 1.0 + 0.2 * _rand((width,), 1), 0.05 * _rand((9, width), 2)
        part.load({"w": _dev(w)})
        got = part.forward(_dev(x), None)
        assert got.dtype == torch.float32 and _rel(got.cpu(), plain.rms_norm(x.double(), w, 1e-3)) < 1e-6


# ---------------------------------------------------------------------------
# parts


def _layer_parts(cfg, layer, dtype, seed, sharp, ranks):
    """Mixer and feed-forward of one layer, built from the engine's own specification, with the tests' weights."""
    from tokensprint_b200.models.vepevik import VepevikConfig, build_vepevik_spec
    from tokensprint_b200.parts.base import BuildContext, build_part

    W = vepevik_weights(cfg, seed, ranks, sharp=sharp)
    params = build_vepevik_spec(VepevikConfig.from_dict(cfg)).layers[layer].params
    ctx = BuildContext(torch.device("cuda"), dtype)
    parts = {}
    for kind, key in (("mixer", "mixer"), ("feed_forward", "feed_forward")):
        if params.get(key) is not None:
            part = build_part(kind, params[key], ctx)
            part.load({s.name: _dev(W[s.name], torch.float32 if s.role == "vector" else dtype) for s in part.tensor_specs()})
            parts[key] = part
    return parts, {k: v.double() for k, v in W.items()}


def _blends(layer):
    return layer["type"] == "attention" and bool(layer["mixer"].get("v_mix"))


def _takes_values(cfg, layer):
    return _blends(cfg["layers"][layer]) and any(_blends(l) for l in cfg["layers"][:layer])


def _plain_mixer(cfg, layer, W):
    entry, eps, p = cfg["layers"][layer], cfg["norm"]["eps"], f"l{layer}.mix."
    m = entry["mixer"]
    if entry["type"] == "attention":
        return lambda x: plain.attention(x, list(range(x.shape[0])), m, W, p, eps, None)[0]
    if entry["type"] == "retention":
        return lambda x: plain.retention(x, list(range(x.shape[0])), m, W, p, eps)
    return lambda x: plain.channel_delta(x, m, W, p, eps)


def _settled(cfg, layer, W, x, dtype):
    """Rows whose result does not hang on the rounding of q, k and v: a retention head's read-out is divided by its root
    mean square, so where its terms nearly cancel (a first token with q . k close to zero keeps only its sign) a
    bfloat16 run may be far off.  All rows in float32 and for the other mixers."""
    entry = cfg["layers"][layer]
    ok = torch.ones(x.shape[0], dtype=torch.bool)
    if entry["type"] != "retention" or dtype == torch.float32:
        return ok
    m, p, pos = entry["mixer"], f"l{layer}.mix.", list(range(x.shape[0]))
    T, H = x.shape[0], m["heads"]
    q, k = (plain.rotate(plain.project(x.double(), W[p + n]).view(T, H, m["dim"]), pos, m) for n in ("q", "k"))
    v = plain.project(x.double(), W[p + "v"]).view(T, H, m["vdim"])
    for a in range(H):
        o = plain.retention_recurrence(q[:, a], k[:, a], v[:, a], m["decay"][a]).pow(2).mean(-1).sqrt()
        ok &= o > 0.2 * o.median()
    return ok


ALONE = [(tag, i) for tag, cfg in sorted(VEP.items()) for i in range(len(cfg["layers"])) if not _takes_values(cfg, i)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", ALONE)
def test_mixers_in_every_cutting(tag, layer, dtype):
    """Whole, in portions down to one token, token by token over several chunks, and in a batch of
    unequal sequences whose pages and slots were used before, against the plain mechanism."""
    cfg = VEP[tag]
    parts, W = _layer_parts(cfg, layer, dtype, 21, 2.0, RANKS[tag])
    mixer, f = parts["mixer"], _plain_mixer(cfg, layer, W)
    xs = {name: _inputs(n, cfg["width"], 30 + i, dtype) for i, (name, n) in enumerate((("a", 75), ("b", 9), ("c", 41)))}
    want = {name: f(x.double()) for name, x in xs.items()}
    ok = {name: _settled(cfg, layer, W, x, dtype) for name, x in xs.items()}
    assert float(ok["a"].float().mean()) > 0.75

    def err(got, name):
        return _rel(got[ok[name]], want[name][ok[name]])

    for page in (16, 8):
        h = Harness(mixer, dtype, page=page)
        assert err(h.step({"a": xs["a"]})["a"], "a") < TOL[dtype], "whole"
        h.end("a")
        assert err(_in_portions(h, "a", xs["a"], (1, 2, 5, 1, 16, 2, 3)), "a") < TOL[dtype], "portions"
        h.end("a")
        assert err(_in_portions(h, "a", xs["a"], (1,)), "a") < TOL[dtype], "token by token"
        h.end("a")
        got = {name: [] for name in xs}
        for step in ({"a": 30, "b": 1, "c": 2}, {"a": 1, "b": 1}, {"a": 44, "b": 7, "c": 39}):
            at = {name: sum(t.shape[0] for t in got[name]) for name in step}
            for name, rows in h.step({name: xs[name][at[name]:at[name] + n] for name, n in step.items()}).items():
                got[name].append(rows)
        for name in xs:
            assert err(torch.cat(got[name]), name) < TOL[dtype], f"batch, {name}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", [("a", 0), ("a", 2), ("b", 4), ("c", 0)])
def test_a_key_on_both_sides_of_a_chunks_edge(tag, layer, dtype):
    """Three tokens' inputs are made ten times as large (the first and the last of a chunk, and one far back: their
    keys and values then dominate wherever they are seen): the queries that have them in their chunk, the first of the
    next chunk, which must not, and everything behind agree with the plain mechanism, in a prompt, with portions
    that end around the edge, and token by token."""
    cfg = VEP[tag]
    size = cfg["layers"][layer]["mixer"]["mask"]["size"]
    parts, W = _layer_parts(cfg, layer, dtype, 22, 3.0, RANKS[tag])
    if _takes_values(cfg, layer):
        parts["mixer"].value_mix = None  # alone here, without another layer's values
    f = _plain_mixer(cfg, layer, W)
    x = _inputs(3 * size + 5, cfg["width"], 40, dtype)
    quiet = f(x.double())
    loud = (size, 2 * size - 1, 1)
    x[list(loud)] *= 10.0
    want = f(x.double())
    moved = (want - quiet).abs().amax(-1)
    # seen to the chunk's end and nowhere behind it
    assert float(moved[size:2 * size].median()) > 1e-2 and float(moved[2 * size - 1]) > 1e-2 and float(moved[2 * size:].max()) == 0.0
    for sizes in ((x.shape[0],), (2 * size - 1, 1, 1, 2), (size + 1, size - 2, 2, 2), (1,)):
        h = Harness(parts["mixer"], dtype, page=8)
        got = _in_portions(h, "s", x, sizes)
        assert _rel(got, want) < TOL[dtype], sizes
        # the quiet rows behind the edge on their own scale
        assert _rel(got[2 * size:], want[2 * size:]) < TOL[dtype], ("behind the edge", sizes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", [(t, i) for t in sorted(VEP) for i in range(len(VEP[t]["layers"])) if _takes_values(VEP[t], i)])
def test_values_blended_with_the_first_layers(tag, layer, dtype):
    """Two layers of a step: the first leaves its values, the other takes them in token by token (each token's first
    values differ from its neighbours'); whole, in portions, one by one, beside another sequence."""
    from tokensprint_b200 import ops

    cfg, eps = VEP[tag], VEP[tag]["norm"]["eps"]
    first = next(i for i, l in enumerate(cfg["layers"]) if _blends(l))
    built = {i: _layer_parts(cfg, i, dtype, 23, 2.0, RANKS[tag]) for i in (first, layer)}
    W = built[first][1]
    xs = {name: {i: _inputs(T, cfg["width"], 50 + i + T, dtype) for i in (first, layer)} for name, T in (("s", 60), ("t", 23))}
    want = {}
    for name, x in xs.items():
        pos = list(range(x[first].shape[0]))
        _, values = plain.attention(x[first].double(), pos, cfg["layers"][first]["mixer"], W, f"l{first}.mix.", eps, None)
        want[name] = plain.attention(x[layer].double(), pos, cfg["layers"][layer]["mixer"], W, f"l{layer}.mix.", eps, values)[0]

    class Pair:
        """Both mixers' harnesses, with what a step's layers share handed from one to the other."""

        def __init__(self):
            self.h = {i: Harness(built[i][0]["mixer"], dtype, page=16) for i in (first, layer)}

        def step(self, parts):
            shared = {}
            out = None
            for i in (first, layer):
                mixer = built[i][0]["mixer"]
                forward = mixer.forward

                def with_shared(x, step, cache, forward=forward):
                    step.shared = shared
                    return forward(x, step, cache)

                mixer.forward = with_shared
                try:
                    out = self.h[i].step({name: xs[name][i][a:b] for name, (a, b) in parts.items()})
                finally:
                    del mixer.forward
            return out

    for sizes in ((60,), (1, 2, 7, 1, 33, 2), (1,)):
        pair, got, at, k = Pair(), {"s": [], "t": []}, {"s": 0, "t": 0}, 0
        while at["s"] < 60:
            n = sizes[k % len(sizes)]
            parts = {name: (at[name], min(at[name] + n, x[first].shape[0])) for name, x in xs.items() if at[name] < x[first].shape[0]}
            for name, rows in pair.step(parts).items():
                got[name].append(rows)
                at[name] = parts[name][1]
            k += 1
        for name in xs:
            assert _rel(torch.cat(got[name]), want[name]) < TOL[dtype], (sizes, name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [1, 2])
def test_a_far_key_through_the_recurrences(layer, dtype):
    """Only the first tokens carry input, the hundreds behind them (almost) none but their queries: what they read out is
    what the state still holds, in one piece, over cuts and one by one."""
    cfg = VEP_LONG
    parts, W = _layer_parts(cfg, layer, dtype, 26, 1.0, RANKS["long"])
    f = _plain_mixer(cfg, layer, W)
    T = 640
    x = _inputs(T, cfg["width"], 41, dtype)
    x[3:] *= 2.0 ** -6
    x[:3] *= 4.0
    want = f(x.double())
    for sizes in ((T,), (2, 300, 1, 1, 2, 400), (1, 1, 1, 1, 1, 635)):
        h = Harness(parts["mixer"], dtype, page=16)
        got = _in_portions(h, "s", x, sizes)
        for part in (slice(0, 3), slice(3, 100), slice(100, T)):
            assert _rel(got[part], want[part]) < 2 * TOL[dtype], (sizes, part)


FEED_FORWARDS = [(tag, i) for tag, cfg in sorted(VEP.items()) for i, l in enumerate(cfg["layers"]) if l["mlp"] is not None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", FEED_FORWARDS)
def test_feed_forwards_on_the_same_rows(tag, layer, dtype):
    """Engine and plain model read the same rows; tokens whose choice hangs on less than 1e-4 of a score are left out."""
    cfg = VEP[tag]
    parts, W = _layer_parts(cfg, layer, dtype, 24, 1.0, RANKS[tag])
    mlp, p = cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    for T in (1, 3, 70):
        x = _inputs(T, cfg["width"], 60 + T, dtype)
        got = parts["feed_forward"].forward(_dev(x.to(dtype)), None).float().cpu()
        clear = torch.ones(T, dtype=torch.bool)
        if mlp["kind"] == "dense":
            want = plain.capped_ff(x.double(), mlp["limit"], W, p)
        else:
            want = plain.routed_ff(x.double(), mlp, W, p)
            s = torch.softmax(x.double() @ W[p + "router"].T, -1)
            groups = mlp["router"].get("groups")
            clear = _clear_choice(s, mlp["router"]["top"], None if groups is None else (groups["count"], groups["keep"]), 1e-4)
        assert _rel(got[clear], want[clear]) < TOL[dtype] if bool(clear.any()) else True, T
