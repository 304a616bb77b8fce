"""Small configurations of the Galirax design for the tests.  They differ from one another in every size, in the order
of the layers, in the run of layers that is passed through again, and in which options are present."""
import copy


def _moe(experts, top, groups, ff, scale):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff}}


# the run that is passed through again starts at the first layer and has all three mixers; key and value heads of different
# sizes, six query heads on two key heads; a window of 37 positions (no multiple of a page) with three kept tokens, and one of
# 70 (longer than a page) with 66 kept tokens (a page and two positions); slow frequencies scaled within 64 positions; head
# size 64 with the whole head rotated; a layer without feed-forward; three groups of which two are kept
CASE_A = {
    "architecture": "Galirax", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "logit_softcap": 9.0,
    "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        {"type": "lightning", "mixer": {"heads": 3, "dim": 40, "vdim": 24, "decay": [0.3, 0.97, 0.9995]},
         "mlp": _moe(9, 2, (3, 2), 40, 1.7)},
        {"type": "attention_2", "mixer": {"heads": 6, "kv_heads": 2, "dim": 40, "vdim": 24, "scale": 0.21,
                                          "rot": {"dims": 16, "base": 500.0}, "mask": {"size": 37, "keep_first": 3}},
         "mlp": _moe(6, 1, (2, 1), 24, 0.8)},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.25,
                                        "rot": {"dims": 20, "base": 300.0,
                                                "scaling": {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 64}}}, "mlp": None},
        {"type": "attention_2", "mixer": {"heads": 2, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.13,
                                          "rot": {"dims": 64, "base": 10000.0}, "mask": {"size": 70, "keep_first": 66}},
         "mlp": _moe(8, 3, (4, 2), 32, 2.2)},
    ],
}

# a width that is no multiple of 8; one head; a window of one position (the query alone, beside the sink and the kept
# token); a window longer than any test sequence; no window; no kept tokens; no rotation; decays of zero and one; every
# expert chosen in all layers (no choice can flip under rounding); no groups, and one group; one expert; no second pass; no
# cap on the logits
CASE_B = {
    "architecture": "Galirax", "vocab": 97, "width": 100, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "attention_2", "mixer": {"heads": 1, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.4,
                                          "rot": {"dims": 8, "base": 100.0}, "mask": {"size": 1, "keep_first": 1}},
         "mlp": _moe(4, 4, (1, 1), 36, 1.0)},
        {"type": "lightning", "mixer": {"heads": 2, "dim": 12, "vdim": 36, "decay": [0.0, 1.0]}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 1, "dim": 72, "vdim": 8, "scale": 0.1}, "mlp": _moe(3, 3, None, 28, 0.6)},
        {"type": "attention_2", "mixer": {"heads": 4, "kv_heads": 1, "dim": 128, "vdim": 128, "scale": 0.08,
                                          "rot": {"dims": 2, "base": 10000.0}, "mask": {"size": 1000, "keep_first": 2}},
         "mlp": _moe(1, 1, None, 44, 3.0)},
        {"type": "attention_2", "mixer": {"heads": 2, "kv_heads": 2, "dim": 24, "vdim": 8, "scale": 0.25}, "mlp": None},
        {"type": "attention_2", "mixer": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 16, "scale": 0.3,
                                          "rot": {"dims": 8, "base": 30.0}, "mask": {"size": 50}}, "mlp": _moe(2, 2, (2, 2), 16, 1.5)},
    ],
}

# the run that is passed through again ends at the last layer and is passed three times; windows of exactly one page and of
# two, with kept tokens that end on a page border, and that are more than the window; twenty query heads on one key head;
# groups of one expert each; head sizes of two tiles (132 channels are no multiple of 8: the plain kernels)
CASE_C = {
    "architecture": "Galirax", "vocab": 150, "width": 64, "norm": {"eps": 1e-5}, "logit_softcap": 40.0,
    "loop": {"start": 2, "stop": 4, "times": 3},
    "layers": [
        {"type": "attention", "mixer": {"heads": 20, "kv_heads": 1, "dim": 16, "vdim": 32, "scale": 0.3,
                                        "rot": {"dims": 16, "base": 1000.0,
                                                "scaling": {"factor": 2.0, "low": 0.5, "high": 4.0, "original": 100}}},
         "mlp": _moe(12, 4, (6, 3), 16, 2.0)},
        {"type": "lightning", "mixer": {"heads": 1, "dim": 132, "vdim": 64, "decay": [0.99]}, "mlp": _moe(5, 2, (5, 3), 24, 1.3)},
        {"type": "attention_2", "mixer": {"heads": 2, "kv_heads": 1, "dim": 128, "vdim": 32, "scale": 0.09,
                                          "rot": {"dims": 32, "base": 1000.0}, "mask": {"size": 64, "keep_first": 64}},
         "mlp": _moe(8, 2, (2, 1), 32, 0.9)},
        {"type": "lightning", "mixer": {"heads": 4, "dim": 16, "vdim": 16, "decay": [0.5, 0.9, 0.99, 0.999]}, "mlp": None},
    ],
}

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C}

# one layer each: the mechanisms alone (sizes unlike the three cases')
_TINY = {"type": "lightning", "mixer": {"heads": 1, "dim": 8, "vdim": 8, "decay": [0.8]}}
SINGLE = {
    "scaled": {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 32, "vdim": 24, "scale": 0.2,
                                              "rot": {"dims": 24, "base": 200.0, "scaling": {"factor": 3.0, "low": 1.0, "high": 2.0,
                                                                                             "original": 30}}}, "mlp": None},
    "kept": {"type": "attention_2", "mixer": {"heads": 4, "kv_heads": 2, "dim": 48, "vdim": 48, "scale": 0.17,
                                              "rot": {"dims": 12, "base": 40.0}, "mask": {"size": 9, "keep_first": 2}}, "mlp": None},
    "decay": {"type": "lightning", "mixer": {"heads": 2, "dim": 20, "vdim": 28, "decay": [0.9, 0.998]}, "mlp": None},
    "experts": dict(_TINY, mlp=_moe(10, 3, (5, 2), 24, 1.9)),
}


def case(name):
    if name.startswith("+"):
        return {"architecture": "Galirax", "vocab": 83, "width": 72, "norm": {"eps": 1e-5}, "logit_softcap": 6.0,
                "loop": {"start": 0, "stop": 1, "times": 2}, "layers": [copy.deepcopy(SINGLE[name[1:]])]}
    return copy.deepcopy(CASES[name])
