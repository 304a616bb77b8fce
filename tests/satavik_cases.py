"""Small configurations of the Satavik design for the tests.  They differ from one another in every size, in which layers
read another layer's keys and values, and in which options are present."""
import copy


def _moe(experts, top, ff, limit, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


# six heads on two key heads; blocks of 37 positions (no multiple of a page) and of 70 (longer than a page); a layer
# that reads keys two layers back under blocks of another size; half of a map's channels rotated; a soft cap that bends
# most scores; a layer without feed-forward; limits that cut; a scale other than the root of the channels
CASE_A = {
    "architecture": "Satavik", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.31, "softcap": 4.0, "diff": 0.45,
                                        "rot": {"dims": 12, "base": 500.0}, "mask": {"size": 37}},
         "mlp": _moe(7, 2, 40, 0.8, (56, 1.5))},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 4, "dim": 64, "vdim": 128, "scale": 0.125, "softcap": 30.0, "diff": 0.2,
                                        "rot": {"dims": 64, "base": 10000.0}, "mask": {"size": 70}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 12, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.2, "softcap": 9.0, "diff": 0.6,
                                        "rot": {"dims": 12, "base": 500.0}, "mask": {"size": 100}, "kv_from": 0},
         "mlp": _moe(5, 1, 24, 2.5, (16, 0.5))},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 24, "scale": 0.4, "softcap": 75.0, "diff": 0.8,
                                        "rot": {"dims": 2, "base": 77.0}, "mask": {"size": 64}},
         "mlp": _moe(4, 4, 32, 1.0)},
    ],
}

# a width that is no multiple of 8; one head; blocks of one position (the query alone); no mask at all on a layer whose
# reader has one and the other way round; no rotation; no soft cap; every expert chosen (no choice can flip under
# rounding); no shared expert; one expert; sizes that no tensor-core kernel takes; values wider than 128 channels
CASE_B = {
    "architecture": "Satavik", "vocab": 97, "width": 100, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5},
    "layers": [
        {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 20, "vdim": 12, "scale": 0.3, "softcap": 10.0, "diff": 0.1,
                                        "rot": {"dims": 6, "base": 100.0}, "mask": {"size": 1}},
         "mlp": _moe(3, 3, 36, 1.2, (20, 3.0))},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 72, "vdim": 136, "scale": 0.12, "softcap": 15.0, "diff": 0.35},
         "mlp": _moe(1, 1, 28, 0.7)},
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 1, "dim": 72, "vdim": 136, "scale": 0.1, "softcap": 25.0, "diff": 0.5,
                                        "mask": {"size": 50}, "kv_from": 1},
         "mlp": None},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 8, "scale": 0.25, "diff": 0.25,
                                        "rot": {"dims": 32, "base": 10000.0}, "mask": {"size": 1000}},
         "mlp": _moe(6, 6, 44, 2.0, (8, 1.0))},
    ],
}

# blocks of exactly one page and of two pages; two readers of one layer; heads of 128 channels a map; as many key heads
# as heads; sixteen heads on one key head; thirteen experts of which four are chosen
CASE_C = {
    "architecture": "Satavik", "vocab": 150, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0},
    "layers": [
        {"type": "attention", "mixer": {"heads": 16, "kv_heads": 1, "dim": 32, "vdim": 64, "scale": 0.18, "softcap": 12.0, "diff": 0.3,
                                        "rot": {"dims": 8, "base": 50.0}, "mask": {"size": 128}},
         "mlp": _moe(13, 4, 32, 1.3, (48, 0.9))},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 32, "vdim": 64, "scale": 0.22, "softcap": 6.0, "diff": 0.7,
                                        "rot": {"dims": 8, "base": 50.0}, "mask": {"size": 128}, "kv_from": 0},
         "mlp": _moe(6, 2, 16, 0.6)},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 128, "vdim": 32, "scale": 0.09, "softcap": 20.0, "diff": 0.4,
                                        "rot": {"dims": 128, "base": 1000.0}, "mask": {"size": 64}},
         "mlp": _moe(8, 3, 24, 4.0, (40, 2.0))},
        {"type": "attention", "mixer": {"heads": 5, "kv_heads": 1, "dim": 32, "vdim": 64, "scale": 0.2, "softcap": 18.0, "diff": 0.5,
                                        "rot": {"dims": 8, "base": 50.0}, "mask": {"size": 5}, "kv_from": 0},
         "mlp": _moe(3, 1, 56, 1.0, (24, 1.1))},
    ],
}

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C}

# one layer each: the mechanisms alone (sizes unlike the three cases')
_PLAIN_MIX = {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 16, "scale": 0.3, "softcap": 11.0, "diff": 0.3,
              "rot": {"dims": 4, "base": 60.0}, "mask": {"size": 200}}
SINGLE = {
    "blocks": {"type": "attention", "mixer": dict(_PLAIN_MIX, heads=4, kv_heads=2, dim=40, vdim=56, mask={"size": 9}), "mlp": None},
    "cap": {"type": "attention", "mixer": dict(_PLAIN_MIX, scale=1.7, softcap=2.5, dim=56), "mlp": None},
    "no_cap": {"type": "attention", "mixer": {k: v for k, v in dict(_PLAIN_MIX, dim=48, vdim=88).items() if k != "softcap"}, "mlp": None},
    "all_keys": {"type": "attention", "mixer": {k: v for k, v in _PLAIN_MIX.items() if k not in ("mask", "rot")}, "mlp": None},
    "experts": {"type": "attention", "mixer": dict(_PLAIN_MIX), "mlp": _moe(9, 3, 24, 0.9, (40, 1.7))},
}


def single_config(which):
    return {"architecture": "Satavik", "vocab": 83, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
            "layers": [copy.deepcopy(SINGLE[which])]}


def case(name):
    return single_config(name[1:]) if name.startswith("+") else copy.deepcopy(CASES[name])
