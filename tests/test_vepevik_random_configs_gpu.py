"""Vepevik models of random shapes through the engine: widths, head counts, key and value widths, inner
widths and rotated parts that are multiples of nothing in particular, any order of the three mixers,
chunks from one position to none, attention layers that blend values and ones that do not, one to five
taps, experts in any grouping, layers without a feed-forward.  Each model runs whole, in portions, with
a decoded tail and mixed with pages and slots used again, in float32 against the float64 plain model
(sharpened queries), and in bfloat16 for finite logits that agree between the cuttings (the routed
layers get a small share of the stream there: a router is a step function of its input)."""

import random

import numpy as np
import pytest

from tests.plain import vepevik_plain as plain
from tests.replay_helpers import replay_in_process, trace_decode_tail, trace_mixed, trace_portions, trace_whole
from tests.vepevik_configs import random_ids, vepevik_weights, write_vepevik_folder

pytestmark = pytest.mark.gpu


def random_config(rng: random.Random) -> dict:
    blend_kv, blend_e = rng.choice([1, 2, 3]), rng.choice([4, 10, 16, 32, 64])  # blending layers share these

    def rot(dim):
        if rng.random() < 0.15:
            return None
        return {"base": rng.choice([30.0, 1000.0, 1e6]), "dims": 2 * rng.randint(1, dim // 2) if rng.random() < 0.5 else dim - dim % 2}

    def attention():
        blends = rng.random() < 0.75
        kv = blend_kv if blends else rng.choice([1, 2, 4])
        dim = rng.choice([6, 8, 16, 24, 32, 48, 64, 80, 128])
        m = {"heads": kv * rng.choice([1, 2, 3, 4]), "kv_heads": kv, "dim": dim, "vdim": blend_e if blends else rng.choice([5, 8, 20, 64, 128]),
             "scale": rng.choice([0.05, 0.1, 0.2])}
        if blends:
            m["v_mix"] = True
        if rng.random() < 0.85:
            m["mask"] = {"size": rng.choice([1, 2, 5, 16, 17, 33, 64, 100, 500])}
        return {"type": "attention", "mixer": m}

    def retention():
        H = rng.choice([1, 2, 3, 5, 8])
        dim = rng.choice([3, 8, 12, 16, 32, 50, 64, 128])
        return {"type": "retention", "mixer": {"heads": H, "dim": dim, "vdim": rng.choice([3, 4, 9, 16, 32, 64]),
                                               "decay": [rng.choice([0.25, 0.5, 0.9, 0.96875, 0.998046875, 1.0]) for _ in range(H)]}}

    def delta():
        kv = rng.choice([1, 2, 3])
        return {"type": "channel_delta", "mixer": {
            "heads": kv * rng.choice([1, 2, 4]), "kv_heads": kv, "dim": rng.choice([1, 3, 8, 12, 16, 32, 40, 64, 96, 128]),
            "vdim": rng.choice([3, 4, 8, 10, 16, 32, 64]), "conv": rng.choice([1, 2, 3, 4, 5])}}

    layers = []
    for _ in range(rng.randint(2, 6)):
        k = rng.random()
        if k < 0.2:
            mlp = None
        elif k < 0.5:
            mlp = {"kind": "dense", "ff": rng.choice([24, 64, 100, 256]), "limit": rng.choice([0.5, 1.0, 7.0])}
        else:
            count, size = rng.choice([1, 1, 2, 3, 8]), rng.choice([1, 2, 4, 5])
            keep = rng.randint(1, count)
            mlp = {"kind": "moe", "expert": {"ff": rng.choice([8, 24, 36, 64])},
                   "router": {"experts": count * size, "top": rng.randint(1, min(keep * size, 4)), "scale": rng.choice([0.5, 1.0, 2.5])}}
            if rng.random() < 0.85:
                mlp["router"]["groups"] = {"count": count, "keep": keep}
            elif mlp["router"]["top"] > count * size:
                mlp["router"]["top"] = count * size
        layer = dict(rng.choice([attention, retention, delta])(), mlp=mlp)
        if layer["type"] != "channel_delta":
            turn = rot(layer["mixer"]["dim"])
            if turn is not None:
                layer["mixer"]["rot"] = turn
        layers.append(layer)
    return {"architecture": "Vepevik", "vocab": rng.choice([50, 211, 333, 1000]), "width": rng.choice([40, 56, 64, 100, 128, 136, 200, 264]),
            "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}


@pytest.mark.parametrize("seed", range(10))
def test_random_model_in_every_cutting(tmp_path, seed):
    from tokensprint_b200.engine.replay import TraceReplayer

    rng = random.Random(3000 + seed)
    cfg = random_config(rng)
    ranks = (rng.choice([1, 3, 8, 20, 32]), rng.choice([1, 5, 8, 16]))
    requests = {f"r{i}": random_ids(cfg, n, seed * 100 + i) for i, n in enumerate([1, 7, 40, 90, 131])}
    for dtype, sharp in (("float32", 2.0), ("bfloat16", 1.0)):
        weights = vepevik_weights(cfg, seed, ranks, sharp=sharp, routed_share=1.0 if dtype == "float32" else 0.01)
        folder = write_vepevik_folder(tmp_path / dtype, cfg, weights)
        want = {k: plain.forward_logits(v, weights, cfg).numpy() for k, v in requests.items()}
        runs = {}
        for name, steps, max_tokens in (("whole", trace_whole(requests), 512), ("portions", trace_portions(requests), 512),
                                        ("tail", trace_decode_tail(requests, 8), 512), ("mixed", trace_mixed(requests, 320, seed=seed, max_live=3), 320)):
            replayer = TraceReplayer.from_folder(folder, dtype, max_tokens, page_size=16, max_live=3)
            replayer.runner.poison_freed_pages = True
            runs[name] = got = replay_in_process(replayer, steps)
            assert len(got) == sum(len(v) for v in requests.values())
            for (rid, pos), row in got.items():
                assert np.isfinite(row).all(), f"{dtype} {name}: request {rid} position {pos} is not finite\n{cfg}"
                if dtype == "float32":
                    err = float(np.abs(row - want[rid][pos]).max() / np.abs(want[rid]).max())
                    assert err < 3e-4, f"float32 {name}: request {rid} position {pos}: error {err:.3g}\n{cfg}"
        tol = 1e-4 if dtype == "float32" else 5e-2
        for name in ("portions", "tail", "mixed"):
            for key, row in runs["whole"].items():
                scale = float(np.abs(want[key[0]]).max())
                assert float(np.abs(row - runs[name][key]).max()) <= tol * scale, f"{dtype}: whole and {name} differ at {key}\n{cfg}"
