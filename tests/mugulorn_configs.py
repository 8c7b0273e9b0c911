"""The tests' own small Mugulorn configurations and weights (no product code here).

The configurations differ from one another in every size and option: one head to six, key widths against
value widths, latents of 20 to 96 entries with rotated parts of 6 to 32, with stretched frequencies and
plain ones, windows from one position to none, layers that read another layer's cached rows through a
window shorter than, equal to and longer than the window of the layer that made them (also where the
maker has none, or the reader has none), two readers of one layer, readers that are not neighbours,
recurrent layers with one block and with as many blocks as channels, blocks of an odd number of
channels, one tap to five, layers with and without a feed-forward, branch multipliers below, above and
equal to one, layer orders that begin with either mixer.  Weights come from the tests' integer-hash
generator under the checkpoint's tensor names.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Optional

import torch

from tests.tiny_configs import seeded_normal


def _yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, scaling=None, window=0, kv_from=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = scaling
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "rot": rot}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _rec(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def _layer(mixer, ff=0):
    return dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)


def _model(vocab, width, eps, embed_scale, mult, layers):
    return {"architecture": "Mugulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "residual_mult": mult, "layers": layers}


# a reader with a longer window than the rows' maker, not its neighbour; a layer without a window whose reader has one
_A_ROT = (1000.0, _yarn(4.0, 32, 8.0, 1.0))
MUG_A = _model(211, 96, 1e-5, 0.7, 0.4, [
    _layer(_lat(3, 10, 8, 12, 20, 14, 0.25, *_A_ROT, window=20), 40),
    _layer(_rec(60, 5, 4), 72),
    _layer(_lat(2, 6, 8, 9, 20, 10, 0.4, *_A_ROT, window=33, kv_from=0), 56),
    _layer(_rec(96, 8, 2)),
    _layer(_lat(4, 12, 10, 16, 24, 30, 0.2, 500.0, _yarn(2.0, 64, 4.0, 0.5)), 64),
    _layer(_lat(1, 8, 10, 20, 24, 12, 0.3, 500.0, _yarn(2.0, 64, 4.0, 0.5), window=7, kv_from=4)),
])

# odd widths; one tap (nothing kept), five taps; one block and blocks of three channels; a reader without a window of
# rows whose maker has one
MUG_B = _model(130, 72, 3e-6, 3.0, 1.0, [
    _layer(_rec(45, 15, 5)),
    _layer(_lat(5, 4, 6, 28, 36, 18, 0.2, 100.0, window=11), 20),
    _layer(_lat(3, 7, 6, 5, 36, 9, 0.35, 100.0, kv_from=1), 50),
    _layer(_rec(21, 1, 1), 24),
    _layer(_rec(33, 33, 3)),
])

# widths the tensor-core kernels take (latent 64 + 16, blocks and feed-forwards that are multiples of 64); two readers of
# the first layer's rows with other windows than its own
_C_ROT = (50000.0, _yarn(8.0, 64, 16.0, 2.0))
MUG_C = _model(300, 128, 1e-6, 1.5, 0.25, [
    _layer(_lat(4, 32, 16, 32, 64, 48, 0.15, *_C_ROT, window=48), 128),
    _layer(_rec(128, 2, 4)),
    _layer(_lat(2, 16, 16, 64, 64, 32, 0.2, *_C_ROT, window=100, kv_from=0), 64),
    _layer(_lat(6, 48, 16, 16, 64, 64, 0.12, *_C_ROT, window=16, kv_from=0), 192),
    _layer(_rec(192, 4, 3), 64),
    _layer(_lat(4, 24, 32, 48, 32, 56, 0.12, 10000.0, window=1)),
])

# a width and a vocabulary that are multiples of nothing useful, a multiplier above one, recurrent layers only around one
# attention; frequencies whose ramp ends on one pair
MUG_D = _model(97, 100, 2e-5, 1.0, 1.3, [
    _layer(_rec(52, 13, 2), 52),
    _layer(_rec(40, 2, 4), 28),
    _layer(_lat(3, 2, 12, 14, 18, 9, 0.35, 777.0, _yarn(3.0, 24, 1.0, 1.0), window=2), 52),
    _layer(_rec(36, 4, 3)),
])

# recurrences alone: a model without a page
MUG_E = _model(64, 48, 1e-6, 2.0, 0.5, [_layer(_rec(64, 4, 3), 64), _layer(_rec(80, 5, 4))])

MUG = {"a": MUG_A, "b": MUG_B, "c": MUG_C, "d": MUG_D, "e": MUG_E}

# for one long request: more than a thousand positions against an `original` length of 128, windows that pass over
# hundreds of decoded tokens, decoded tokens whose keys are split over several CTAs, states that live through all of it
_L_ROT = (100000.0, _yarn(8.0, 128, 32.0, 1.0))
MUG_LONG = _model(500, 256, 1e-6, 1.0, 0.6, [
    _layer(_lat(4, 32, 32, 48, 96, 64, 0.12, *_L_ROT, window=200), 192),
    _layer(_rec(256, 4, 4)),
    _layer(_lat(4, 32, 32, 32, 96, 48, 0.12, *_L_ROT, window=500, kv_from=0), 128),
    _layer(_rec(320, 5, 3), 64),
    _layer(_lat(2, 16, 32, 32, 96, 48, 0.12, *_L_ROT, kv_from=0)),
])


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    V, W = cfg["vocab"], cfg["width"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
        shapes[p + "norm1"] = (W,)
        if layer["type"] == "latent_attention":
            H, d, r, e, R, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            shapes.update({q + "dq": (Q, W), q + "dq.norm": (Q,), q + "uq": (H * (d + r), Q), q + "uk": (H * d, R), q + "uv": (H * e, R),
                           q + "sink": (H,), q + "g": (H * e, W), q + "o": (W, H * e)})
            if m.get("kv_from") is None:
                shapes.update({q + "dkv": (R + r, W), q + "dkv.norm": (R,)})
        else:
            w, B, K = m["width"], m["blocks"], m["conv"]
            k = w // B
            shapes.update({q + "y": (w, W), q + "y.b": (w,), q + "x": (w, W), q + "x.b": (w,), q + "conv": (w, K), q + "conv.b": (w,),
                           q + "ra": (B, k, k), q + "ra.b": (B, k), q + "ri": (B, k, k), q + "ri.b": (B, k), q + "lam": (w,), q + "o": (W, w)})
        if layer["mlp"] is not None:
            f, n = p + "mlp.", layer["mlp"]["ff"]
            shapes.update({p + "norm2": (W,), f + "gate": (n, W), f + "up": (n, W), f + "down": (W, n)})
    return shapes


def mugulorn_weights(cfg: dict, seed: int, *, sharp: float = 1.0) -> dict[str, torch.Tensor]:
    """Float32 weights whose values are all representable in bfloat16 (a bfloat16 run reads exactly what
    the plain model reads).  Matrices N(0, 1/fan_in), norm weights around one, embedding rows N(0, 1); taps
    around a third; sinks of about one (of the order of the largest scores, so that leaving one out
    shows); every bias of a few tenths; decay parameters such that channels forget within a few tokens to
    a few hundred.  `sharp` multiplies the matrices that make queries (a softmax that picks few keys shows
    one wrong key or a window that is one position off far beyond rounding)."""
    out: dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(cfg).items():
        x = seeded_normal(shape, f"mugulorn:{seed}:{name}")
        if name == "embed":
            pass
        elif name.endswith(".conv"):
            x = 0.5 * x / float(shape[1]) ** 0.5 + 0.3
        elif name.endswith(".sink"):
            x = 1.0 + x
        elif name.endswith(".lam"):
            x = -3.5 + 1.5 * x
        elif name.endswith(".b"):
            x = 0.3 * x
        elif len(shape) == 1:
            x = 1.0 + 0.1 * x
        else:
            x = x / float(shape[-1]) ** 0.5
            if name.endswith(".uq"):
                x = x * sharp
            if name.endswith((".ra", ".ri", ".g")):
                x = x * 2.0  # gates that depend on the token
        out[name] = x.to(torch.bfloat16).to(torch.float32)
    return out


def write_mugulorn_folder(folder: Path, cfg: dict, weights: dict[str, torch.Tensor], dtype: Optional[torch.dtype] = torch.bfloat16) -> Path:
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
