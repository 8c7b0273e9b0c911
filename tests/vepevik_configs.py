"""The tests' own small Vepevik configurations and weights (no product code here).

The configurations differ from one another in every size and option: head counts and grouping (every
query head with its own keys, all with one), key widths against value widths, chunks of one position to
none, rotations of a whole head, of its first entries and none, attention layers that blend their
values with those of the first that does, layers between them that do not, retention with constants from
a half to one, delta layers with one head and with six, whose q and k heads are shared or not, one to
five taps, narrow pairs of two inner widths that are multiples of nothing; layers without a
feed-forward, capped dense ones whose cap bites and ones whose cap never does, routed experts in one
group, in groups of one expert, with all groups kept, with one kept, one to four choices per token.
Weights come from the tests' integer-hash generator under the checkpoint's tensor names; RANKS gives
the inner widths of the delta layers' pairs, which no configuration key need name.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Optional

import torch

from tests.tiny_configs import seeded_normal


def _rot(base, dims):
    return {"base": base, "dims": dims}


def _att(heads, kv_heads, dim, vdim, scale, chunk, rot=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = rot
    if chunk:
        m["mask"] = {"size": chunk}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m}


def _ret(decay, dim, vdim, rot=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        m["rot"] = rot
    return {"type": "retention", "mixer": m}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(ff, experts, top, scale=1.0, groups=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def _model(vocab, width, eps, layers):
    return {"architecture": "Vepevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# all three mixers; the first blending layer is not the first attention layer, and one between two blending ones
# does not blend; part of a head turns; a layer without a feed-forward
VEP_A = _model(211, 96, 1e-5, [
    _layer(_att(4, 2, 24, 16, 0.3, 20, _rot(1000.0, 12)), _dense(40, 0.8)),
    _layer(_delta(4, 2, 12, 10, 3), _moe(24, 6, 2, 1.5, (3, 2))),
    _layer(_att(4, 2, 16, 28, 0.4, 11, _rot(100.0, 16), v_mix=True), None),
    _layer(_ret([0.5, 0.97, 1.0], 10, 6, _rot(500.0, 6)), _moe(16, 5, 3, 2.0)),
    _layer(_att(2, 1, 18, 8, 0.5, 0, _rot(50.0, 2)), _dense(20, 3.0)),
    _layer(_att(6, 2, 14, 28, 0.35, 32, None, v_mix=True), _moe(8, 4, 1, 0.5, (4, 1))),
])

# one head everywhere a layer can have one, odd widths, one tap (nothing kept), chunks of one position, no rotation, layers that
# begin with the delta rule; as many groups as experts
VEP_B = _model(130, 72, 3e-6, [
    _layer(_delta(1, 1, 7, 5, 1), _moe(10, 3, 2, 1.0, (3, 2))),
    _layer(_ret([0.9], 9, 11), None),
    _layer(_att(5, 1, 12, 28, 0.2, 1, _rot(300.0, 4), v_mix=True), _dense(20, 0.5)),
    _layer(_delta(6, 3, 20, 10, 5), _dense(33, 2.0)),
    _layer(_att(3, 1, 6, 28, 0.6, 7, _rot(300.0, 6), v_mix=True), _moe(12, 8, 4, 3.0, (2, 1))),
])

# widths the tensor-core kernels take (heads of 64 and 128, expert widths that are multiples of 8), every blending layer
# with its own head count, a layer that sees every earlier key
VEP_C = _model(300, 128, 1e-6, [
    _layer(_att(4, 2, 64, 64, 0.25, 48, _rot(50000.0, 32), v_mix=True), _moe(32, 8, 2, 2.0, (4, 2))),
    _layer(_delta(2, 2, 64, 64, 4), _dense(96, 1.0)),
    _layer(_ret([0.75, 0.9375, 0.98046875, 0.99609375], 32, 64, _rot(10000.0, 32)), _moe(64, 16, 3, 1.0, (2, 2))),
    _layer(_att(2, 2, 128, 64, 0.15, 0, _rot(50000.0, 128), v_mix=True), _dense(64, 5.0)),
    _layer(_att(8, 2, 48, 64, 0.3, 17, _rot(100.0, 48), v_mix=True), None),
    _layer(_delta(4, 1, 128, 32, 2), _moe(16, 4, 4, 1.25)),
])

# a width and a vocabulary that are multiples of nothing useful, three heads everywhere, no attention that blends
VEP_D = _model(97, 100, 2e-5, [
    _layer(_ret([0.6, 0.95, 0.999], 14, 9, _rot(77.0, 14)), _moe(12, 9, 3, 0.7, (3, 1))),
    _layer(_delta(3, 3, 9, 14, 3), _dense(52, 1.5)),
    _layer(_att(3, 3, 10, 14, 0.6, 5, _rot(777.0, 10)), _moe(9, 2, 1, 4.0, (1, 1))),
    _layer(_ret([1.0, 0.8], 5, 16), None),
])

VEP = {"a": VEP_A, "b": VEP_B, "c": VEP_C, "d": VEP_D}

# for one long request: chunks of 200 positions that begin and end in prompts and in decoded tokens, a second attention whose chunk
# is longer than the request's first portions, prompt attention over hundreds of keys, states that live through all of it
VEP_LONG = _model(500, 256, 1e-6, [
    _layer(_att(8, 2, 64, 32, 0.25, 200, _rot(100000.0, 16), v_mix=True), _dense(96, 1.0)),
    _layer(_ret([0.875, 0.96875, 0.9921875, 0.998046875], 32, 48, _rot(10000.0, 16)), _moe(32, 8, 2, 1.5, (4, 3))),
    _layer(_delta(4, 2, 32, 48, 4), _dense(64, 2.0)),
    _layer(_att(4, 2, 128, 32, 0.15, 700, _rot(100000.0, 64), v_mix=True), None),
])

RANKS = {"a": (6, 9), "b": (3, 5), "c": (16, 8), "d": (7, 2), "long": (12, 20)}


def tensor_shapes(cfg: dict, ranks: tuple[int, int]) -> dict[str, tuple[int, ...]]:
    """Every tensor a checkpoint of this configuration has (the share of the first blending layer among them, which nothing reads)."""
    V, W = cfg["vocab"], cfg["width"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
        shapes[p + "norm1"] = (W,)
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            shapes.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * e, W), q + "q.norm": (d,), q + "k.norm": (d,), q + "g": (H, W),
                           q + "o": (W, H * e)})
            if m.get("v_mix"):
                shapes[q + "vmix"] = ()
        elif layer["type"] == "retention":
            shapes.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * e, W), q + "g": (H * e, W), q + "o": (W, H * e)})
        else:
            G, K = m["kv_heads"], m["conv"]
            ra, rg = m.get("decay_rank", ranks[0]), m.get("gate_rank", ranks[1])
            shapes.update({q + "q": (G * d, W), q + "q.conv": (G * d, K), q + "k": (G * d, W), q + "k.conv": (G * d, K), q + "v": (H * e, W),
                           q + "v.conv": (H * e, K), q + "b": (H, W), q + "A_log": (H,), q + "a1": (ra, W), q + "a2": (H * d, ra),
                           q + "dt_bias": (H * d,), q + "norm": (e,), q + "g1": (rg, W), q + "g2": (H * e, rg), q + "o": (W, H * e)})
        mlp = layer["mlp"]
        if mlp is not None:
            shapes[p + "norm2"] = (W,)
            f = p + "mlp."
            if mlp["kind"] == "dense":
                shapes.update({f + "gate": (mlp["ff"], W), f + "up": (mlp["ff"], W), f + "down": (W, mlp["ff"])})
            else:
                shapes[f + "router"] = (mlp["router"]["experts"], W)
                for e in range(mlp["router"]["experts"]):
                    shapes.update({f"{f}e{e}.gate": (mlp["expert"]["ff"], W), f"{f}e{e}.up": (mlp["expert"]["ff"], W),
                                   f"{f}e{e}.down": (W, mlp["expert"]["ff"])})
    return shapes


def unused_tensors(cfg: dict) -> set[str]:
    first = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "attention" and l["mixer"].get("v_mix")][:1]
    return {f"l{i}.mix.vmix" for i in first}


def vepevik_weights(cfg: dict, seed: int, ranks: tuple[int, int], *, sharp: float = 1.0, routed_share: float = 1.0) -> dict[str, torch.Tensor]:
    """Float32 weights whose values are all representable in bfloat16 (a bfloat16 run reads exactly
    what the plain model reads).  Matrices N(0, 1/fan_in), norm weights around one, the embedding
    table N(0, 1); shares of the first values around a half; taps around a third; decay rates and
    biases such that a delta state's rows live for a few to a hundred tokens.  `sharp` multiplies the
    attention layers' query norms (a softmax that picks few keys shows one wrong key or a chunk that
    is one position off far beyond rounding).  `routed_share` multiplies the experts' last matrices: a
    router is a step function of its input, so a run in a narrower number format, which now and then
    chooses another expert than the plain model, is compared with a small share."""
    out: dict[str, torch.Tensor] = {}
    shapes = tensor_shapes(cfg, ranks)
    for name, shape in shapes.items():
        x = seeded_normal(shape if shape else (1,), f"vepevik:{seed}:{name}")
        if not shape:
            x = (0.5 + 0.2 * x).reshape(())
        elif name == "embed":
            pass
        elif name.endswith(".conv"):
            x = 0.5 * x / float(shape[1]) ** 0.5 + 0.3
        elif name.endswith("dt_bias"):
            x = -3.0 + 1.2 * x
        elif name.endswith("A_log"):
            x = 0.3 + 0.4 * x
        elif len(shape) == 1:
            x = 1.0 + 0.1 * x
            if name.endswith(".q.norm"):
                x = x * sharp
        else:
            x = x / float(shape[1]) ** 0.5
            if name.endswith((".mix.b", ".mix.a2", ".mlp.router")) or (name.endswith(".mix.g") and name[:-1] + "q.norm" in shapes):
                x = x * 2.0  # gates and choices that depend on the token
            if ".mlp.e" in name and name.endswith(".down"):
                x = x * routed_share
        out[name] = x.to(torch.bfloat16).to(torch.float32)
    return out


def write_vepevik_folder(folder: Path, cfg: dict, weights: dict[str, torch.Tensor], dtype: Optional[torch.dtype] = torch.bfloat16) -> Path:
    """config.json + model.safetensors, written with the safetensors package (not the engine's writer)."""
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: (v if dtype is None else v.to(dtype)).contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return folder


def random_ids(cfg: dict, n: int, seed: int) -> list[int]:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
