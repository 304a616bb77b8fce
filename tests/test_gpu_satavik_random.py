"""Satavik configurations drawn at random (sizes, head counts, readers of other layers' keys, masks, constants, seeds), each run
whole, as a prompt followed by single tokens and as one unequal batch, in both dtypes, against the plain restatement."""
import json

import numpy as np
import pytest
import torch

import plain_satavik as plain
from gpu_util import run_steps, steps_batches, steps_tail, steps_whole
from test_gpu_satavik import Rec, allowed, relative_error

from esp_b200.engine import Engine
from esp_b200.weights import write_safetensors

pytestmark = pytest.mark.gpu


def draw(rng):
    pick = lambda *xs: xs[int(rng.integers(0, len(xs)))]
    width = pick(64, 72, 100, 128, 160, 256)
    layers = []
    for i in range(int(rng.integers(2, 7))):
        owners = [j for j, l in enumerate(layers) if "kv_from" not in l["mixer"]]
        group = pick(1, 2, 3, 5, 8, 12)
        if owners and rng.integers(0, 3) == 0:          # reads another layer's keys and values
            j = pick(*owners)
            mixer = {k: v for k, v in layers[j]["mixer"].items() if k in ("kv_heads", "dim", "vdim", "rot")}
            mixer.update(kv_from=j, heads=mixer["kv_heads"] * group)
        else:
            dim = pick(8, 16, 20, 24, 32, 48, 64, 64, 80, 128)
            mixer = {"kv_heads": pick(1, 1, 2, 3), "dim": dim, "vdim": pick(2 * dim, 2 * dim, dim, 8, 40, 72, 128)}
            mixer["heads"] = mixer["kv_heads"] * group
            if rng.integers(0, 6) > 0:
                mixer["rot"] = {"dims": 2 * int(rng.integers(1, dim // 2 + 1)), "base": pick(50.0, 1000.0, 10000.0, 500000.0)}
        mixer.update(scale=float(rng.uniform(0.5, 1.5)) / mixer["dim"] ** 0.5, diff=float(rng.uniform(0.1, 0.8)))
        if rng.integers(0, 6) > 0:
            mixer["softcap"] = pick(3.0, 10.0, 20.0, 30.0, 50.0, 80.0)
        if rng.integers(0, 6) > 0:
            mixer["mask"] = {"size": pick(1, 3, 17, 41, 63, 64, 65, 100, 128, 500)}
        mlp = None
        if rng.integers(0, 5) > 0:
            experts = pick(1, 2, 3, 6, 9, 16, 40)
            mlp = {"kind": "moe", "router": {"experts": experts, "top": int(rng.integers(1, min(experts, 5) + 1))},
                   "expert": {"ff": pick(8, 16, 24, 32, 64), "limit": pick(0.5, 1.0, 3.0, 7.0)}}
            if rng.integers(0, 3):
                mlp["shared"] = {"ff": pick(8, 16, 48), "limit": pick(0.4, 2.0, 7.0)}
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Satavik", "vocab": pick(97, 256, 301, 513), "width": width, "norm": {"eps": pick(1e-6, 1e-5)},
            "embedding": {"scale": pick(1.0, 7.5, 12.0)}, "layers": layers}


LENGTHS = (1, 70, 190)


@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configuration(tmp_path, seed):
    rng = np.random.default_rng(4100 + seed)
    lengths = LENGTHS
    raw = draw(rng)
    stored = plain.random_weights(raw, 70 + seed)
    reqs = {f"r{i}": [int(t) for t in rng.integers(0, raw["vocab"], n)] for i, n in enumerate(lengths)}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    write_safetensors(tmp_path / "model.safetensors", stored)
    ids = list(reqs)
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(tmp_path, dtype=dtype, max_tokens=1024)
        eng.rt.record_routing = True
        for what, steps in (("whole", steps_whole(reqs)), ("prompt + single tokens", steps_tail(reqs, tail=40)),
                            ("one batch", steps_batches(reqs, [ids], {rid: max(1, len(t) - 25) for rid, t in reqs.items()}))):
            rec = Rec(raw["vocab"])
            run_steps(eng, steps, rec)
            for rid, toks in reqs.items():
                forced = {layer: torch.from_numpy(chosen.astype(np.int64)) for layer, chosen in rec.forced(rid, len(toks)).items()}
                ref = plain.forward(raw, stored, toks, forced_routing=forced or None).numpy()
                err = relative_error(rec.logits_of(rid, list(range(len(toks)))), ref)
                bound = allowed(raw, stored, toks, forced or None, dtype, ref, err)
                assert (err <= bound).all(), (f"seed {seed}, {dtype}, {what}, request {rid}: position {int((err / bound).argmax())} "
                                              f"is {(err / bound).max():.2f} of its bound, worst error {err.max():.3e}; configuration {json.dumps(raw)}")
                if dtype == "float32" and forced:
                    # in 32-bit the engine's choices are the restatement's own, but for scores within rounding of each other
                    own = plain.forward(raw, stored, toks).numpy()
                    assert relative_error(rec.logits_of(rid, list(range(len(toks)))), own).max() <= 1e-2
        del eng
