"""Configuration of the Satavik design, its plan and its tensor list, without a GPU; how far its caches must reach; and the
plain restatement against itself (causality; a block's edge; the two maps; the soft cap; the chosen logits' softmax; the
clamped unit; the rotation)."""
import math

import pytest
import torch

import plain_satavik as plain
from satavik_cases import case

from esp_b200.cache.book import GroupBook, KvLayout
from esp_b200.config import config_from_dict, config_from_json
from esp_b200.config.satavik import SatavikConfig
from esp_b200.errors import InvalidConfig, Unsupported
from esp_b200.weights.random_init import parameter_specs, write_model_folder


def test_registry_finds_the_design_by_its_architecture_string():
    cfg = config_from_dict(case("A"))
    assert isinstance(cfg, SatavikConfig)
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


@pytest.mark.parametrize("name", ["A", "B", "C", "+experts"])
def test_tensor_names_and_shapes_are_the_designs(name):
    raw = case(name)
    mine = {s.name: tuple(s.shape) for s in parameter_specs(config_from_dict(raw))}
    assert mine == plain.tensor_shapes(raw)


def test_plan_takes_every_size_and_constant_from_the_configuration():
    plan = config_from_dict(case("A")).plan()
    assert (plan.head_weight, plan.embed_weight, plan.embed_scale) == ("head", "embed", 3.0)
    a, b, c, d = (blk.mixer for blk in plan.blocks)
    assert (a.num_heads, a.num_kv_heads, a.key_dim, a.value_dim, a.scale, a.softcap, a.diff, a.chunk) == (6, 2, 24, 40, 0.31, 4.0, 0.45, 37)
    assert (a.position.rotary_dim, a.position.theta, a.eps) == (12, 500.0, 1e-5)
    assert (c.num_heads, c.num_kv_heads, c.softcap, c.chunk) == (12, 2, 9.0, 100)
    assert [m.own_kv for m in (a, b, c, d)] == [True, True, False, True]
    assert [e.cache_of for e in plan.schedule] == [None, None, 0, None]
    moe = plan.blocks[0].ffn
    assert (moe.num_experts, moe.top_k, moe.expert_intermediate, moe.shared_intermediate) == (7, 2, 40, 56)
    assert (moe.glu, moe.shared_glu, moe.chosen_softmax) == ((0.8, 1.702, 1.0), (1.5, 1.702, 1.0), True)
    assert plan.blocks[3].ffn.shared_intermediate is None and plan.blocks[3].ffn.shared_glu is None
    assert plan.blocks[1].ffn is None and plan.blocks[1].ffn_post_norm is None
    assert plan.blocks[0].mixer_post_norm.weight == "l0.norm1" and plan.blocks[0].kind == "output_norm_residual"


def test_a_cache_reaches_as_far_as_the_widest_of_its_readers():
    """Layer 0 of case A is read under blocks of 37 and of 100 positions: its pages stay as long as a window of 100 does.
    Layer 1 of case B has no mask, its reader has blocks of 50: nothing is given back.  Two readers with equal blocks
    (and one of five positions) in case C; a layer alone keeps its own blocks."""
    mix = lambda name, i: config_from_dict(case(name)).plan().blocks[i].mixer
    assert (mix("A", 0).keep_window, mix("A", 0).keep_chunk) == (100, None)
    assert (mix("A", 1).keep_window, mix("A", 1).keep_chunk) == (None, 70)
    assert (mix("B", 1).keep_window, mix("B", 1).keep_chunk) == (None, None)
    assert (mix("C", 0).keep_window, mix("C", 0).keep_chunk) == (128, None)
    raw = case("C")
    raw["layers"].pop()
    plan = config_from_dict(raw).plan()
    assert (plan.blocks[0].mixer.keep_window, plan.blocks[0].mixer.keep_chunk) == (None, 128)
    # whatever the position, a window as long as the larger block begins no later than either block does
    book = GroupBook(KvLayout(1, 8, window=100), 4)
    for p in range(400):
        assert book.first_needed(p) <= min(p - p % 37, p - p % 100)


def _set(path, value):
    def change(raw):
        d = raw
        for key in path[:-1]:
            d = d[key]
        if value is KeyError:
            del d[path[-1]]
        else:
            d[path[-1]] = value
    return change


MIX = ("layers", 0, "mixer")


@pytest.mark.parametrize("change, error", [
    (_set(("layers", 0, "type"), "mamba"), Unsupported),
    (_set(MIX + ("kv_heads",), 4), InvalidConfig),
    (_set(MIX + ("rot", "dims"), 11), InvalidConfig),
    (_set(MIX + ("rot", "dims"), 26), InvalidConfig),
    (_set(MIX + ("mask", "size"), 0), InvalidConfig),
    (_set(MIX + ("softcap",), 0.0), InvalidConfig),
    (_set(MIX + ("scale",), 0.0), InvalidConfig),
    (_set(MIX + ("diff",), KeyError), InvalidConfig),
    (_set(("layers", 2, "mixer", "kv_from"), 2), InvalidConfig),
    (_set(("layers", 2, "mixer", "kv_from"), 3), InvalidConfig),
    (_set(("layers", 3, "mixer", "kv_from"), 2), InvalidConfig),          # layer 2 has no keys of its own
    (_set(("layers", 2, "mixer", "dim"), 16), InvalidConfig),
    (_set(("layers", 2, "mixer", "rot"), {"dims": 12, "base": 501.0}), InvalidConfig),
    (_set(("layers", 0, "mlp", "kind"), "dense"), Unsupported),
    (_set(("layers", 0, "mlp", "router", "top"), 8), InvalidConfig),
    (_set(("layers", 0, "mlp", "expert", "limit"), -1.0), InvalidConfig),
    (_set(("layers", 0, "mlp", "shared", "ff"), 0), InvalidConfig),
    (_set(("norm", "eps"), 0.0), InvalidConfig),
])
def test_refusals(change, error):
    raw = case("A")
    change(raw)
    with pytest.raises(error):
        config_from_dict(raw)


def test_a_reader_may_leave_out_what_it_shares_with_the_caches_owner():
    raw = case("A")
    for key in ("kv_heads", "dim", "vdim", "rot"):
        del raw["layers"][2]["mixer"][key]
    assert config_from_dict(raw).plan() == config_from_dict(case("A")).plan()


def test_random_model_folder_round_trips(tmp_path):
    cfg = config_from_dict(case("C"))
    write_model_folder(cfg, 5, tmp_path)
    assert config_from_json(tmp_path).to_dict() == cfg.to_dict()
    from esp_b200.weights.loader import FolderSource
    src = FolderSource(tmp_path)
    assert {n: tuple(src.shape(n)) for n in src.names()} == plain.tensor_shapes(case("C"))


# ------------------------------------------------------------------------------------ the restatement against itself
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_plain_restatement_is_causal_and_finite(name):
    raw = case(name)
    w = plain.random_weights(raw, 3)
    g = torch.Generator().manual_seed(1)
    toks = torch.randint(0, raw["vocab"], (90,), generator=g).tolist()
    full = plain.forward(raw, w, toks)
    assert torch.isfinite(full).all()
    other = list(toks)
    other[-1] = (other[-1] + 1) % raw["vocab"]
    moved = plain.forward(raw, w, other)
    assert torch.equal(full[:-1], moved[:-1]) and not torch.equal(full[-1], moved[-1])
    assert torch.allclose(plain.forward(raw, w, toks[:40]), full[:40], atol=1e-9)


def test_blocks_are_counted_from_the_first_position():
    seen = plain.visible_keys(11, 4)
    for i in range(11):
        assert [j for j in range(11) if seen[i, j]] == list(range(i - i % 4, i + 1))


def test_second_map_is_taken_off_the_first():
    """One visible key each: both maps return its value, what is left is (1 - lambda) v, and the norm makes it a unit
    vector times the sign of 1 - lambda."""
    K, V = 4, 6
    mix = {"heads": 1, "kv_heads": 1, "dim": K, "vdim": V, "scale": 1.0, "diff": 0.25, "mask": {"size": 1}}
    g = torch.Generator().manual_seed(0)
    h = torch.randn(3, V, dtype=torch.float64, generator=g)
    w = {n: torch.randn(r, V, dtype=torch.float64, generator=g) for n, r in (("q", 2 * K), ("k", 2 * K))}
    w.update({"v": torch.eye(V, dtype=torch.float64), "o": torch.eye(V, dtype=torch.float64), "g": torch.zeros(1, V, dtype=torch.float64),
              "q.norm": torch.ones(K), "k.norm": torch.ones(K), "lq1": torch.zeros(K), "lk1": torch.zeros(K),
              "lq2": torch.full((K,), 0.5), "lk2": torch.full((K,), 0.5)})
    lam = 1 - math.exp(1.0) + 0.25
    assert abs(float(plain.second_map_weight(w, "", 0.25)) - lam) < 1e-6
    y, _ = plain.differential_attention(h, w, "", mix, 1e-12, torch.arange(3))
    assert torch.allclose(y, plain.unit_rms(h, 1e-12) * math.copysign(1, 1 - lam) * 0.75 * 0.5, atol=1e-6)


def test_soft_cap_bounds_scores_and_leaves_small_ones():
    s = torch.tensor([0.01, -5.0, 1e4], dtype=torch.float64)
    c = plain.capped(s, 10.0)
    assert abs(float(c[0]) - 0.01) < 1e-6 and abs(float(c[1]) + 10 * math.tanh(0.5)) < 1e-12 and float(c[2]) == 10.0
    assert torch.equal(plain.capped(s, None), s)


def test_router_weights_the_chosen_logits_alone():
    D = 3
    w = {"router": torch.zeros(4, D, dtype=torch.float64), "router.b": torch.tensor([0.0, 0.0, 0.0, 2.5], dtype=torch.float64)}
    w["router"][:, 0] = torch.tensor([3.0, 2.0, 1.0, 0.0])
    h = torch.zeros(1, D, dtype=torch.float64)
    h[0, 0] = 1.0
    ids, wts, _ = plain.route(h, w, "", 2)
    assert ids[0].tolist() == [0, 3]                              # the last one is chosen through its bias, which counts in its weight
    e = math.exp(-0.5)
    assert torch.allclose(wts[0], torch.tensor([1 / (1 + e), e / (1 + e)], dtype=torch.float64))


def test_clamped_unit_bounds_the_gate_above_and_the_other_branch_on_both_sides():
    one = torch.ones(1, 1, dtype=torch.float64)
    def f(g, u, limit):
        return float(plain.clamped_unit(one, {"gate": one * g, "up": one * u, "down": one}, "", limit))
    act = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert abs(f(5.0, 7.0, 2.0) - act(2.0, 2.0)) < 1e-12
    assert abs(f(-5.0, -7.0, 2.0) - act(-5.0, -2.0)) < 1e-12      # the gate has no lower limit


def test_rotation_pairs_the_halves_and_leaves_the_rest():
    x = torch.arange(8, dtype=torch.float64).view(1, 1, 8) + 1
    y = plain.rotate_halves(x, torch.tensor([3]), 4, 10.0)
    assert torch.equal(y[..., 4:], x[..., 4:])
    for i in range(2):
        a = 3 * 10.0 ** (-2.0 * i / 4)
        u, v = float(x[0, 0, i]), float(x[0, 0, i + 2])
        assert abs(float(y[0, 0, i]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12
        assert abs(float(y[0, 0, i + 2]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12
