"""The mechanisms of Mugulorn one at a time: each kernel and each mixer part against the plain
function of the same mechanism, whole prompts, portions down to one token, batches of unequal
sequences with slots and pages in any order and used again; inputs made so that a key just inside
or just outside a window, a far key, a sink that is left out, a lost kept input or a state that was
not carried shows far beyond rounding."""

import pytest
import torch

from tests.mixer_harness import Harness, batch, dev, i32, in_portions, inputs, rand, rel
from tests.mugulorn_configs import MUG, MUG_LONG, mugulorn_weights
from tests.plain import mugulorn_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}


# ---------------------------------------------------------------------------
# kernels alone


@pytest.mark.parametrize("C", [37, 64])
@pytest.mark.parametrize("taps", [1, 2, 3, 5])
@pytest.mark.parametrize("dtype", DTYPES)
def test_convolution_with_a_bias_on_its_inputs(C, taps, dtype):
    """The bias of the rows is added to every input but not to the zeros before a sequence's start, and the kept
    inputs carry it: portions of 1, 2 and more tokens side by side, a slot that is used again."""
    from tokensprint_b200 import ops

    w, bias, in_bias = rand((C, taps), 1) * 0.7, rand((C,), 2), 2.0 + rand((C,), 3)
    seqs = {k: rand((n, C), 4 + i).to(dtype).float() for i, (k, n) in enumerate((("a", 23), ("b", 9), ("c", 40), ("d", 6)))}
    state = torch.full((3, 8 + (taps - 1) * C), float("nan"), device="cuda")
    view = state[:, 8:] if taps > 1 else None
    slot_of, done, got = {"a": 2, "b": 0, "c": 1}, {k: 0 for k in seqs}, {k: [] for k in seqs}
    for slot in slot_of.values():
        state[slot].zero_()
    for step in ({"a": 1, "b": 2, "c": 7}, {"a": 2, "c": 1}, {"b": 7, "a": 20, "c": 32}, {"d": 1}, {"d": 2}, {"d": 3}):
        if "d" in step and "d" not in slot_of:
            slot_of["d"] = slot_of.pop("b")
            state[slot_of["d"]].zero_()
        names = sorted(step)
        rows = torch.cat([seqs[k][done[k]:done[k] + step[k]] for k in names])
        cu, seq = batch([step[k] for k in names])
        out = torch.empty(rows.shape, device="cuda", dtype=dtype)
        ops.causal_conv(dev(rows, dtype), dev(w.t().contiguous()), dev(bias), view, i32([slot_of[k] for k in names]), cu, seq, len(names), out,
                        in_bias=dev(in_bias))
        at = 0
        for k in names:
            got[k].append(out[at:at + step[k]].float().cpu())
            at += step[k]
            done[k] += step[k]
    for k, x in seqs.items():
        want = plain.causal_conv(x.double() + in_bias.double(), w.double(), bias.double())
        assert rel(torch.cat(got[k]), want) < (1e-5 if dtype == torch.float32 else 1e-2), (k, taps)


def _recurrence_inputs(w, T, dtype, seed, spread=1.5):
    u, y = rand((T, w), seed).to(dtype).float(), rand((T, w), seed + 1).to(dtype).float()
    pre = spread * rand((T, 2, w), seed + 2)
    return u, y, pre, 0.5 * rand((w,), seed + 3), 0.5 * rand((w,), seed + 4), -3.0 + 2.0 * rand((w,), seed + 5), 0.3 * rand((w,), seed + 6)


def _recurrence_plain(u, y, pre, br, bi, lam, yb):
    u, pre = u.double(), pre.double()
    s = plain.gated_recurrence(u, torch.sigmoid(pre[:, 0] + br.double()), torch.sigmoid(pre[:, 1] + bi.double()), lam)
    return s, s * plain.gelu_tanh(y.double() + yb.double())


def _pre_as_stored(pre, blocks):
    """[T, 2, w] as the block products leave it: per block the r products, then the i products."""
    T, _, w = pre.shape
    return pre.view(T, 2, blocks, w // blocks).transpose(1, 2).reshape(T, 2 * w).contiguous()


def _scan(case, blocks, dtype, state, slots, lengths, decode_seqs=0):
    from tokensprint_b200 import ops

    u, y, pre, br, bi, lam, yb = case
    T, w = u.shape
    both = torch.full((T, 2 * w + 8), float("nan"), device="cuda", dtype=dtype)  # y as a column range of a wider matrix
    both[:, :w] = dev(y, dtype)
    cu, seq = batch(lengths)
    out = torch.empty((T, w), device="cuda", dtype=dtype)
    ops.rglru_scan(dev(u, dtype), dev(_pre_as_stored(pre, blocks)), dev(br), dev(bi), dev(lam), 8.0, both[:, :w], dev(yb), state, i32(slots), cu, seq,
                   out, len(lengths), blocks, max(lengths), decode_seqs)
    return out.float().cpu()


def _rows(case, a, b):
    return tuple(t[a:b] for t in case[:3]) + tuple(case[3:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w, blocks", [(45, 15), (64, 4), (21, 1), (34, 17), (128, 2)])
def test_recurrence_whole_in_portions_and_token_by_token(w, blocks, dtype):
    """700 tokens are more than a round of the kernel in either of its shapes."""
    T = 700
    case = _recurrence_inputs(w, T, dtype, 10 * w)
    states, want = _recurrence_plain(*case)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    for sizes in ([T], [1, 2, 7, 1, 33, 2, 257, 3, 129, 265], [1] * 40 + [128, 256, 276]):
        state = torch.zeros((4, w + 3), device="cuda")
        got, at = [], 0
        for n in sizes:
            got.append(_scan(_rows(case, at, at + n), blocks, dtype, state, [2], [n]))
            at += n
        assert at == T
        assert rel(torch.cat(got), want) < tol, sizes
        # the state is float32 whatever the compute dtype
        assert rel(state[2, :w], states[-1]) < 3e-5, sizes
        assert float(state[[0, 1, 3]].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_of_many_channels(dtype):
    """More channel groups than SMs: the kernel's other CTA shape."""
    w, T = 2400, 300
    case = _recurrence_inputs(w, T, dtype, 5)
    states, want = _recurrence_plain(*case)
    state = torch.zeros((1, w), device="cuda")
    assert rel(_scan(case, 10, dtype, state, [0], [T]), want) < (2e-5 if dtype == torch.float32 else 1e-2)
    assert rel(state[0], states[-1]) < 3e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_of_unequal_sequences_against_each_alone(dtype):
    w, blocks = 48, 3
    lengths = [1, 1, 1, 2, 140, 5, 300]
    case = _recurrence_inputs(w, sum(lengths), dtype, 77)
    slots = [5, 0, 3, 6, 1, 2, 4]
    state = rand((8, w), 9).cuda()
    before = state.clone()
    got = _scan(case, blocks, dtype, state, slots, lengths, decode_seqs=3)
    at = 0
    for slot, n in zip(slots, lengths):
        alone = before.clone()
        one = _scan(_rows(case, at, at + n), blocks, dtype, alone, [slot], [n])
        assert rel(got[at:at + n], one) < (1e-6 if dtype == torch.float32 else 1e-2)
        assert rel(state[slot], alone[slot].cpu()) < 1e-5
        at += n
    assert torch.equal(state[7], before[7])


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_at_the_ends_of_its_range(dtype):
    """Gates that are shut or wide open, channels that never forget and channels that forget at once: finite and right."""
    w, T = 32, 40
    u, y, pre, br, bi, lam, yb = _recurrence_inputs(w, T, dtype, 3)
    pre[:10, 0], pre[10:20, 0], pre[20:30, 1], pre[30:, 1] = -200.0, 200.0, -200.0, 200.0
    lam = torch.linspace(-25.0, 12.0, w)
    case = (u, y, pre, br, bi, lam, yb)
    states, want = _recurrence_plain(*case)
    state = torch.zeros((1, w), device="cuda")
    got = _scan(case, 4, dtype, state, [0], [T])
    assert bool(torch.isfinite(got).all()) and rel(got, want) < (3e-5 if dtype == torch.float32 else 1e-2)
    # channel by channel: a slow channel's small state counts as much as a fast one's large one
    worst = ((state[0].cpu().double() - states[-1]).abs() / states[-1].abs().clamp_min(1e-12)).max()
    assert float(worst) < 2e-4


@pytest.mark.parametrize("blocks, k", [(1, 8), (3, 16), (2, 24), (4, 40), (2, 256), (1, 264), (2, 136)])
@pytest.mark.parametrize("T", [1, 7, 33, 70])
def test_decode_step_with_the_gate_products_in_the_kernel(blocks, k, T):
    """Against the plain gates and recurrence on the same bfloat16 rows; a token of no sequence gets zeros and
    touches no state."""
    from tokensprint_b200 import ops

    w = blocks * k
    bf = torch.bfloat16
    u, y = rand((T, w), 1).to(bf), rand((T, w), 2).to(bf)
    ra, ri = ((2.0 * rand((blocks, k, k), s) / k ** 0.5).to(bf) for s in (3, 4))
    br, bi, yb, lam = 0.5 * rand((w,), 5), 0.5 * rand((w,), 6), 0.3 * rand((w,), 7), -3.0 + 2.0 * rand((w,), 8)
    r = plain.block_gate(u.double(), ra.double(), br.view(blocks, k).double())
    i = plain.block_gate(u.double(), ri.double(), bi.view(blocks, k).double())
    log_a = -8.0 * r * plain.softplus(lam.double())
    slots = torch.randperm(T + 3, generator=torch.Generator().manual_seed(T))[:T].tolist()
    seq = list(range(T))
    if T > 2:
        seq[2] = -1
    state = rand((T + 3, w + 8), 9).cuda()
    before = state.cpu().double()
    S = torch.exp(log_a) * before[slots, :w] + torch.sqrt(-torch.expm1(2 * log_a)) * i * u.double()
    want = S * plain.gelu_tanh(y.double() + yb.double())
    out = torch.full((T, w), float("nan"), device="cuda", dtype=bf)
    gates = dev(torch.cat([ra, ri], dim=1).contiguous())
    ops.rglru_step(dev(u), gates, dev(br), dev(bi), dev(lam), 8.0, dev(y), dev(yb), state, i32(slots), i32(seq), out)
    here = [t for t in range(T) if seq[t] >= 0]
    assert rel(out[here], want[here]) < 1e-2
    assert rel(state[:, :w][[slots[t] for t in here]], S[here]) < 3e-5
    if T > 2:
        assert float(out[2].abs().max()) == 0.0 and torch.equal(state[slots[2]].cpu().double(), before[slots[2]])
    assert torch.equal(state[:, w:].cpu().double(), before[:, w:])


def _attend_plain(q, rows, rank, scale, window, sink, positions):
    """q [T, H, D] at `positions`, cached rows [n, D]."""
    T, H, _ = q.shape
    s = torch.einsum("thd,nd->thn", q.double(), rows.double()) * scale
    dist = torch.tensor(positions)[:, None] - torch.arange(rows.shape[0])[None, :]
    visible = (dist >= 0) & ((dist < window) if window else (dist >= 0))
    out = torch.zeros(T, H, rank, dtype=torch.float64)
    for h in range(H):
        p = plain.softmax_with_sink(s[:, h], visible, sink[h].double() if sink is not None else torch.tensor(float("-inf")))
        out[:, h] = p @ rows[:, :rank].double()
    return out


@pytest.mark.parametrize("rank, rot", [(20, 6), (64, 16), (32, 32)])
@pytest.mark.parametrize("window", [0, 1, 37, 64, 65])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_standing_out_key_at_the_windows_edge_and_a_sink(rank, rot, window, dtype):
    """One key's score stands far above the others; it lies just inside the window of one query and just outside of the
    next one's (or far back, without a window).  Sinks of every size: far below the scores, about as high as the key that
    stands out, far above (the heads' outputs then nearly vanish).  In a prompt, and for single tokens whose keys are cut into ranges."""
    from tokensprint_b200 import ops

    if window == 0 and rank == 20:
        pytest.skip("covered by the other sizes")
    n, H, page, scale, D = 200, 5, 16, 0.25, rank + rot
    sink = torch.tensor([-30.0, 0.5, 16.0, 40.0, 2.0])
    for key in (3, 63, 64, 150):
        rows = (0.1 * rand((n, D), 1)).to(dtype).float()
        rows[key, 0], rows[key, rank:] = 8.0, 0.0
        q = (0.1 * rand((n, H, D), 2)).to(dtype).float()
        q[:, :, 0] = 8.0  # score 16 with the key, small ones with the others
        table = torch.randperm(40, generator=torch.Generator().manual_seed(3))[: -(-n // page)].tolist()
        pages = torch.full((40, page, D), float("nan"), device="cuda", dtype=dtype)
        for p in range(n):
            pages[table[p // page], p % page] = dev(rows[p], dtype)
        bt = i32(table).view(1, -1)
        want = _attend_plain(q, rows, rank, scale, window, sink, list(range(n)))
        bare = _attend_plain(q, rows, rank, scale, window, None, list(range(n)))
        assert rel(bare, want) > 0.3  # leaving the sink out would show
        mma = dtype == torch.bfloat16 and ops.latent_attention_mma_supported(rank, rot)
        for positions in (list(range(n)), [key + (window or 100) - 1], [key + (window or 100)], [n - 1]):
            positions = [p for p in positions if p < n]
            if not positions:
                continue
            qs = dev(q[positions].contiguous(), dtype)
            out = torch.empty((len(positions), H, rank), device="cuda", dtype=dtype)
            if mma:
                splits = 1 if len(positions) > 1 else 3
                ops.latent_attention_mma(qs, pages, out, None, i32([0, len(positions)]), i32([positions[-1] + 1]), bt, page, 1, len(positions), H, rank,
                                         rot, scale, window, splits, sink=dev(sink))
            else:
                ops.latent_attention_simple(qs, pages, out, None, i32(positions), i32([0] * len(positions)), bt, page, H, rank, rot, scale, window,
                                            sink=dev(sink))
            got, ref = out.double().cpu(), want[positions]
            assert float((got - ref).abs().max()) < (1e-4 if dtype == torch.float32 else 2e-2) * 8.0, (key, positions[:2])


@pytest.mark.parametrize("dtype", DTYPES)
def test_small_kernels_with_their_new_options(dtype):
    from tokensprint_b200 import ops

    tol = 1e-6 if dtype == torch.float32 else 1e-2
    for T, W in ((1, 96), (5, 100), (70, 37), (9, 256)):
        hidden, delta, wt = rand((T, W), 1), rand((T, W), 2).to(dtype).float(), 1.0 + 0.1 * rand((W,), 3)
        out = torch.empty((T, W), device="cuda", dtype=dtype)
        h = dev(hidden.clone())
        ops.add_rmsnorm(h, dev(delta, dtype), dev(wt), out, 1e-5, delta_scale=0.3)
        want = hidden.double() + 0.3 * delta.double()
        assert rel(h, want) < 1e-6 and rel(out, plain.rms_norm(want, wt, 1e-5)) < tol
        h = dev(hidden.clone())
        rows = torch.tensor([T - 1, 0])
        some = torch.empty((2, W), device="cuda", dtype=dtype)
        ops.add_rmsnorm(h, dev(delta, dtype), dev(wt), some, 1e-5, i32(rows.tolist()), delta_scale=0.3)
        assert rel(some, plain.rms_norm(want, wt, 1e-5)[rows]) < tol and torch.equal(h.cpu(), hidden)
        ops.residual_add(h, dev(delta, dtype), -1.7)
        assert rel(h, hidden.double() - 1.7 * delta.double()) < 1e-6
        # rows that are a column range of a wider matrix
        wide = dev(rand((T, W + 24), 4), dtype)
        normed = torch.empty((T, W), device="cuda", dtype=dtype)
        ops.rmsnorm_rows(wide[:, 8:8 + W], dev(wt), normed, 1e-3)
        assert rel(normed, plain.rms_norm(wide[:, 8:8 + W].double().cpu(), wt, 1e-3)) < tol
        gated = torch.empty((T, W), device="cuda", dtype=dtype)
        ops.gate_rows(normed, wide[:, 16:16 + W], gated, 1, W, W)
        assert rel(gated, normed.double().cpu() * torch.sigmoid(wide[:, 16:16 + W].double().cpu())) < tol
        gu = dev(2.0 * rand((T, 2 * W), 5), dtype)
        act = torch.empty((T, W), device="cuda", dtype=dtype)
        ops.swiglu(gu, act, 0, "gelu_tanh")
        g = gu.double().cpu()
        assert rel(act, plain.gelu_tanh(g[:, :W]) * g[:, W:]) < (1e-5 if dtype == torch.float32 else tol)


@pytest.mark.parametrize("T", [1, 8, 31])
def test_fused_products_with_a_multiplier_and_gelu(T):
    """The few-row product that adds into the stream multiplies its result; the one with the activation in its epilogue applies gelu."""
    from tokensprint_b200 import ops

    K, N = 128, 192
    bf = torch.bfloat16
    x, w = rand((T, K), 1).to(bf), (rand((N, K), 2) / K ** 0.5).to(bf)
    hidden, nw = rand((T, N), 3), 1.0 + 0.1 * rand((N,), 4)
    h, xp = dev(hidden.clone()), torch.empty((T, N), device="cuda", dtype=bf)
    ssq = torch.empty((2, T), device="cuda")
    ops.gemm_skinny_fused(dev(x), dev(w), mode=ops.GEMM_EPILOGUE_RESIDUAL_NORM, hidden=h, norm_weight=dev(nw), xprime=xp, ssq_out=ssq, branch_scale=0.35)
    want = hidden.double() + 0.35 * (x.double() @ w.double().T)
    assert rel(h, want) < 1e-5 and rel(xp, want * nw.double()) < 1e-2 and rel(ssq.sum(0), want.pow(2).sum(-1)) < 1e-4
    w2 = (rand((256, K), 5) / K ** 0.5).to(bf)  # blocks of 64 gate rows and their 64 up rows
    out = torch.empty((T, 128), device="cuda", dtype=bf)
    ops.gemm_skinny_fused(dev(x), dev(w2), out=out, mode=ops.GEMM_EPILOGUE_SWIGLU, activation="gelu_tanh")
    p = (x.double() @ w2.double().T).view(T, 2, 2, 64)
    assert rel(out, (plain.gelu_tanh(p[:, :, 0]) * p[:, :, 1]).reshape(T, 128)) < 1e-2


# ---------------------------------------------------------------------------
# mixers and feed-forwards


def _layer_parts(cfg, layer, dtype, seed, sharp):
    from tokensprint_b200.models.mugulorn import MugulornConfig, build_mugulorn_spec
    from tokensprint_b200.parts.base import BuildContext, build_part

    W = mugulorn_weights(cfg, seed, sharp=sharp)
    params = build_mugulorn_spec(MugulornConfig.from_dict(cfg)).layers[layer].params
    ctx = BuildContext(torch.device("cuda"), dtype)
    parts = {}
    for kind in ("mixer", "feed_forward"):
        if params.get(kind) is not None:
            part = build_part(kind, params[kind], ctx)
            part.load({s.name: dev(W[s.name], torch.float32 if s.role == "vector" else dtype) for s in part.tensor_specs()})
            parts[kind] = part
    return parts, {k: v.double() for k, v in W.items()}


RECURRENT = [(tag, i) for tag, cfg in sorted(MUG.items()) for i, l in enumerate(cfg["layers"]) if l["type"] == "rglru"]
WRITERS = [(tag, i) for tag, cfg in sorted(MUG.items()) for i, l in enumerate(cfg["layers"])
           if l["type"] == "latent_attention" and l["mixer"].get("kv_from") is None] + [("long", 0)]
DENSE = [(tag, i) for tag, cfg in sorted(MUG.items()) for i, l in enumerate(cfg["layers"]) if l["mlp"] is not None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", RECURRENT)
def test_recurrent_mixer_in_every_cutting(tag, layer, dtype):
    """Whole, in portions down to one token, token by token, and in a batch of unequal sequences whose slots were used
    before, against the plain mechanism."""
    cfg = MUG[tag]
    parts, W = _layer_parts(cfg, layer, dtype, 21, 1.0)
    mixer, p = parts["mixer"], f"l{layer}.mix."
    xs = {name: inputs(n, cfg["width"], 30 + i, dtype) for i, (name, n) in enumerate((("a", 75), ("b", 9), ("c", 41)))}
    want = {name: plain.recurrent_mixer(x.double(), W, p) for name, x in xs.items()}
    h = Harness(mixer, dtype, page=16)
    assert rel(h.step({"a": xs["a"]})["a"], want["a"]) < TOL[dtype], "whole"
    for sizes in ((1, 2, 5, 1, 16, 2, 3), (1,)):
        h.end("a")
        assert rel(in_portions(h, "a", xs["a"], sizes), want["a"]) < TOL[dtype], sizes
    h.end("a")
    got = {name: [] for name in xs}
    for step in ({"a": 30, "b": 1, "c": 2}, {"a": 1, "b": 1}, {"a": 44, "b": 7, "c": 39}):
        at = {name: sum(t.shape[0] for t in got[name]) for name in step}
        out = h.step({name: xs[name][at[name]:at[name] + n] for name, n in step.items()})
        for name in step:
            got[name].append(out[name])
    for name in xs:
        assert rel(torch.cat(got[name]), want[name]) < TOL[dtype], f"batch, {name}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", WRITERS)
def test_latent_attention_and_the_layers_that_read_its_rows(tag, layer, dtype):
    """A writer and its readers on the same pages, with windows, sinks, gates and matrices of their own: whole, in portions, token by token."""
    cfg = MUG_LONG if tag == "long" else MUG[tag]
    eps = cfg["norm"]["eps"]
    readers = [i for i, l in enumerate(cfg["layers"]) if l["mixer"].get("kv_from") == layer]
    sharp = 2.0 if dtype == torch.float32 else 1.0
    built = {i: _layer_parts(cfg, i, dtype, 22, sharp) for i in [layer] + readers}
    W = built[layer][1]
    T = 300 if tag == "long" else 70
    xs = {i: inputs(T, cfg["width"], 50 + i, dtype) for i in [layer] + readers}
    pos = list(range(T))
    c, kr = plain.latent_rows(xs[layer].double(), pos, cfg["layers"][layer]["mixer"], W, f"l{layer}.mix.", eps)
    want = {i: plain.latent_attention(xs[i].double(), pos, cfg["layers"][i]["mixer"], W, f"l{i}.mix.", eps, c, kr) for i in xs}
    for sizes in ((T,), (1, 2, 7, 1, 33, 2), (1,)):
        h = Harness(built[layer][0]["mixer"], dtype, page=16, readers=[built[i][0]["mixer"] for i in readers])
        at, k, got = 0, 0, {i: [] for i in xs}
        while at < T:
            n = min(sizes[k % len(sizes)], T - at)
            for which, i in enumerate([layer] + readers):  # the writer first, as in the model's run order
                got[i].append(h.step({"s": xs[i][at:at + n]}, which)["s"])
            at, k = at + n, k + 1
            if sizes == (1,) and at >= 40:
                break
        for i in xs:
            rows = torch.cat(got[i])
            assert rel(rows, want[i][:rows.shape[0]]) < TOL[dtype], (sizes, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag, layer", DENSE)
def test_gelu_feed_forward(tag, layer, dtype):
    cfg = MUG[tag]
    parts, W = _layer_parts(cfg, layer, dtype, 24, 1.0)
    for T in (1, 3, 70):
        x = inputs(T, cfg["width"], 60 + T, dtype)
        got = parts["feed_forward"].forward(dev(x.to(dtype)), None).float().cpu()
        assert rel(got, plain.gelu_ff(x.double(), W, f"l{layer}.mlp.")) < TOL[dtype], T
