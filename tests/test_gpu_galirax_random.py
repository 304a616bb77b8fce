"""Galirax configurations drawn at random (sizes, head counts, order of layers, windows and kept tokens, passes, groups,
constants, seeds), each run whole, as a prompt followed by single tokens and as one unequal batch, in both dtypes, against
the plain restatement."""
import json

import numpy as np
import pytest

import plain_galirax as plain
from gpu_util import run_steps, steps_batches, steps_tail, steps_whole
from test_gpu_galirax import BOUND, Rec, forced_of, relative_error

from esp_b200.engine import Engine
from esp_b200.weights import write_safetensors

pytestmark = pytest.mark.gpu


def draw(rng):
    pick = lambda *xs: xs[int(rng.integers(0, len(xs)))]
    width = pick(64, 70, 72, 100, 128, 160, 320)
    layers = []
    for i in range(int(rng.integers(2, 6))):
        kind = pick("attention", "attention_2", "attention_2", "lightning")
        if kind == "lightning":
            heads = pick(1, 2, 3, 5)
            mixer = {"heads": heads, "dim": pick(8, 16, 18, 20, 48, 64, 128), "vdim": pick(8, 10, 16, 24, 40, 64, 96),
                     "decay": [float(1 - 10 ** -rng.uniform(0.2, 3.5)) for _ in range(heads)]}
        else:
            kv, dim = pick(1, 1, 2, 3), pick(8, 16, 20, 24, 32, 48, 64, 80, 112, 128)
            mixer = {"heads": kv * pick(1, 2, 3, 5, 8, 17), "kv_heads": kv, "dim": dim, "vdim": pick(dim, dim, 8, 24, 40, 72, 128),
                     "scale": float(rng.uniform(0.5, 1.5)) / dim ** 0.5}
            if rng.integers(0, 6) > 0:
                mixer["rot"] = {"dims": 2 * int(rng.integers(1, dim // 2 + 1)), "base": pick(50.0, 1000.0, 10000.0, 500000.0)}
                if kind == "attention" and rng.integers(0, 3):
                    mixer["rot"]["scaling"] = {"factor": pick(2.0, 4.0, 8.0), "low": pick(0.5, 1.0), "high": pick(2.0, 4.0),
                                               "original": pick(32, 100, 1024)}
            if kind == "attention_2" and rng.integers(0, 6) > 0:
                mixer["mask"] = {"size": pick(1, 3, 17, 41, 63, 64, 65, 100, 128, 500), "keep_first": pick(0, 1, 4, 5, 64, 65, 130)}
        mlp = None
        if rng.integers(0, 5) > 0:
            per, count = pick(1, 2, 3, 5), pick(1, 2, 3, 4)
            keep = int(rng.integers(1, count + 1))
            mlp = {"kind": "moe", "router": {"experts": per * count, "top": int(rng.integers(1, min(per * keep, 5) + 1)),
                                             "scale": float(rng.uniform(0.5, 3.0)), "groups": {"count": count, "keep": keep}},
                   "expert": {"ff": pick(8, 16, 24, 32, 64)}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    raw = {"architecture": "Galirax", "vocab": pick(97, 256, 301, 513), "width": width, "norm": {"eps": pick(1e-6, 1e-5)},
           "logit_softcap": pick(5.0, 20.0, 50.0), "layers": layers}
    if rng.integers(0, 4) > 0:
        start = int(rng.integers(0, len(layers)))
        raw["loop"] = {"start": start, "stop": int(rng.integers(start + 1, len(layers) + 1)), "times": pick(1, 2, 3)}
    return raw


LENGTHS = (1, 70, 190)


@pytest.mark.parametrize("seed", list(range(16)))
def test_random_configuration(tmp_path, seed):
    rng = np.random.default_rng(5200 + seed)
    lengths = LENGTHS
    raw = draw(rng)
    stored = plain.random_weights(raw, 90 + seed)
    reqs = {f"r{i}": [int(t) for t in rng.integers(0, raw["vocab"], n)] for i, n in enumerate(lengths)}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    write_safetensors(tmp_path / "model.safetensors", stored)
    ids = list(reqs)
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(tmp_path, dtype=dtype, max_tokens=1024)
        eng.rt.record_routing = True
        for what, steps in (("whole", steps_whole(reqs)), ("prompt + single tokens", steps_tail(reqs, tail=40)),
                            ("one batch", steps_batches(reqs, [ids], {rid: max(1, len(t) - 25) for rid, t in reqs.items()}))):
            rec = Rec(raw)
            run_steps(eng, steps, rec)
            for rid, toks in reqs.items():
                forced = forced_of(rec, rid, len(toks))
                ref = plain.forward(raw, stored, toks, forced_routing=forced or None).numpy()
                err = relative_error(rec.logits_of(rid, list(range(len(toks)))), ref)
                assert err.max() <= BOUND[dtype], (f"seed {seed}, {dtype}, {what}, request {rid}: position {int(err.argmax())} is off by "
                                                   f"{err.max():.3e}; configuration {json.dumps(raw)}")
                if dtype == "float32" and forced:
                    # in 32-bit the engine's choices are the restatement's own, but for scores within rounding of each other
                    own = plain.forward(raw, stored, toks).numpy()
                    assert relative_error(rec.logits_of(rid, list(range(len(toks)))), own).max() <= 1e-2
        del eng
