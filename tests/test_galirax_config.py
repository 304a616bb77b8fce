"""Configuration of the Galirax design, its plan and its tensor list, and the cache's bookkeeping for a window that keeps
the first tokens, without a GPU; and the plain restatement against itself (causality, the window's edge and the kept
tokens, the sink, the passes, the choice among groups, the recurrence against its closed form, scaled frequencies)."""
import math

import numpy as np
import pytest
import torch

import plain_galirax as plain
from galirax_cases import case

from esp_b200.cache.book import PAGE, CacheBook, KvLayout
from esp_b200.config import config_from_dict, config_from_json
from esp_b200.config.galirax import GaliraxConfig
from esp_b200.errors import InvalidConfig, Unsupported
from esp_b200.weights.random_init import parameter_specs, write_model_folder


def test_registry_finds_the_design_by_its_architecture_string():
    cfg = config_from_dict(case("A"))
    assert isinstance(cfg, GaliraxConfig)
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_tensor_names_and_shapes_are_the_designs(name):
    raw = case(name)
    mine = {s.name: tuple(s.shape) for s in parameter_specs(config_from_dict(raw))}
    assert mine == plain.tensor_shapes(raw)


def test_plan_takes_every_size_and_constant_from_the_configuration():
    raw = case("A")
    plan = config_from_dict(raw).plan()
    assert (plan.embed_weight, plan.head_weight, plan.logit_softcap) == ("embed", "head", 9.0)
    assert (plan.final_norm.kind, plan.final_norm.weight, plan.final_norm.bias) == ("layernorm", "final.norm", "final.norm.b")
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 0, 1, 2, 3] and all(e.cache_of is None for e in plan.schedule)
    lin, kept, scaled, kept2 = (b.mixer for b in plan.blocks)
    assert (lin.num_heads, lin.key_dim, lin.value_dim, lin.decay, lin.eps) == (3, 40, 24, (0.3, 0.97, 0.9995), 1e-5)
    assert (kept.num_heads, kept.num_kv_heads, kept.key_dim, kept.value_dim, kept.scale) == (6, 2, 40, 24, 0.21)
    assert (kept.window, kept.keep_first, kept.chunk, kept.qkv_bias, kept.learned_sink) == (37, 3, None, True, True)
    assert (kept.position.rotary_dim, kept.position.theta, kept.position.factor) == (16, 500.0, None)
    p = scaled.position
    assert (p.rotary_dim, p.theta, p.factor, p.low, p.high, p.original) == (20, 300.0, 5.0, 1.0, 3.0, 64.0)
    assert (scaled.window, scaled.qkv_bias, scaled.unit_heads, scaled.learned_sink, scaled.value_blend) == (None, False, False, True, None)
    assert (kept2.window, kept2.keep_first) == (70, 66)
    moe = plan.blocks[0].ffn
    assert (moe.num_experts, moe.top_k, moe.groups, moe.keep_groups, moe.group_top, moe.weight_scale) == (9, 2, 3, 2, 2, 1.7)
    assert moe.sigmoid_scores and moe.norm_topk and moe.correction == "correction" and moe.shared_intermediate is None
    assert plan.blocks[2].ffn is None
    plain_b = config_from_dict(case("B")).plan()
    assert plain_b.logit_softcap is None and [e.layer for e in plain_b.schedule] == [0, 1, 2, 3, 4, 5]
    assert plain_b.blocks[4].mixer.window is None and plain_b.blocks[5].mixer.keep_first == 0


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


@pytest.mark.parametrize("change, error", [
    (_set(("layers", 0, "type"), "mamba2"), Unsupported),
    (_set(("layers", 0, "mixer", "decay"), [0.5, 0.5]), InvalidConfig),               # three heads
    (_set(("layers", 0, "mixer", "decay"), [0.5, 0.5, math.inf]), InvalidConfig),
    (_set(("layers", 1, "mixer", "kv_heads"), 4), InvalidConfig),
    (_set(("layers", 1, "mixer", "rot", "dims"), 15), InvalidConfig),
    (_set(("layers", 1, "mixer", "rot", "dims"), 42), InvalidConfig),
    (_set(("layers", 1, "mixer", "mask", "size"), 0), InvalidConfig),
    (_set(("layers", 1, "mixer", "mask", "keep_first"), -1), InvalidConfig),
    (_set(("layers", 1, "mixer", "scale"), 0.0), InvalidConfig),
    (_set(("layers", 2, "mixer", "mask"), {"size": 5}), Unsupported),                 # this kind of layer sees every key
    (_set(("layers", 2, "mixer", "rot", "scaling", "low"), 3.0), InvalidConfig),      # not below high
    (_set(("layers", 2, "mixer", "rot", "scaling", "factor"), KeyError), InvalidConfig),
    (_set(("layers", 0, "mlp", "router", "groups", "count"), 2), InvalidConfig),      # nine experts in two groups
    (_set(("layers", 0, "mlp", "router", "groups", "keep"), 4), InvalidConfig),
    (_set(("layers", 0, "mlp", "router", "scale"), KeyError), InvalidConfig),
    (_set(("layers", 0, "mlp", "router", "top"), 10), InvalidConfig),
    (_set(("layers", 0, "mlp", "kind"), "dense"), Unsupported),
    (_set(("loop", "stop"), 5), InvalidConfig),
    (_set(("loop", "start"), 3), InvalidConfig),
    (_set(("loop", "times"), 0), InvalidConfig),
    (_set(("logit_softcap",), -1.0), InvalidConfig),
    (_set(("norm", "eps"), 0.0), InvalidConfig),
])
def test_refusals(change, error):
    raw = case("A")
    change(raw)
    with pytest.raises(error):
        config_from_dict(raw)


def test_kept_groups_must_hold_the_chosen_experts():
    raw = case("C")
    raw["layers"][2]["mlp"]["router"]["top"] = 5          # two groups of four experts, one kept
    with pytest.raises(InvalidConfig):
        config_from_dict(raw)


def test_random_model_folder_round_trips(tmp_path):
    cfg = config_from_dict(case("C"))
    write_model_folder(cfg, 5, tmp_path)
    again = config_from_json(tmp_path)
    assert again.to_dict() == cfg.to_dict()
    from esp_b200.weights.loader import FolderSource
    src = FolderSource(tmp_path)
    assert {n: tuple(src.shape(n)) for n in src.names()} == plain.tensor_shapes(case("C"))


# ------------------------------------------------------------------------------ pages of a window with kept first tokens
@pytest.mark.parametrize("window, keep", [(37, 3), (70, 66), (64, 64), (1, 130), (100, 0), (200, 1)])
@pytest.mark.parametrize("portions", [[1], [2, 31, 64, 3], [200, 1, 1]])
def test_pages_of_a_window_with_kept_first_tokens(window, keep, portions):
    """After every step the slot holds every page that the next query can see, and no other."""
    book = CacheBook([KvLayout(1, 8, window, keep_first=keep), KvLayout(1, 8)], 30 * PAGE, 2, 1 << 20)
    slot, length, i = book.open(), 0, 0
    while length < 700:
        n = portions[i % len(portions)]
        book.reserve({slot: n})
        held = book.groups[0].tables[slot]
        for p in range(length, length + n):               # while the step runs: all that its queries see, and where they write
            seen = [j for j in range(p + 1) if p - j < window or j < keep]
            assert all(held[j // PAGE] >= 0 for j in seen)
        book.commit({slot: n})
        length += n
        i += 1
        held = book.groups[0].tables[slot]
        # written positions that the query at the next position sees; the last page may be partly written
        need = {j // PAGE for j in range(length) if length - j < window or j < keep}
        have = {k for k, page in enumerate(held) if page >= 0}
        assert need <= have
        slack = {k for k in have - need}
        assert len(slack) <= 1 and all(k == (length - 1) // PAGE or k == length // PAGE for k in slack), (length, need, have)
        assert len(set(p for p in held if p >= 0)) == len(have)
    book.close(slot)
    assert all(g.pool.available == g.pool.n for g in book.groups)


def test_a_cancelled_step_gives_its_pages_back_and_keeps_the_kept_ones():
    book = CacheBook([KvLayout(1, 8, 10, keep_first=70)], 12 * PAGE, 1, 1 << 20)
    slot = book.open()
    book.reserve({slot: 400})
    book.commit({slot: 400})
    before, free = list(book.groups[0].tables[slot]), book.groups[0].pool.available
    assert [p >= 0 for p in before] == [True, True, False, False, False, False, True]
    receipts = book.reserve({slot: 200})
    book.cancel(receipts)
    assert book.groups[0].tables[slot] == before and book.groups[0].pool.available == free


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


def test_window_holds_the_query_its_predecessors_and_the_first_tokens():
    vis = plain.visible_keys(12, {"size": 4, "keep_first": 2})
    assert vis[9].tolist() == [True, True, False, False, False, False, True, True, True, True, False, False]
    assert vis[4].tolist() == [True] * 5 + [False] * 7
    assert plain.visible_keys(12, None)[11].all()


def test_sink_takes_its_share():
    p = plain.sink_softmax(torch.zeros(1, 3, 3, dtype=torch.float64), plain.visible_keys(3, None), torch.tensor([math.log(2.0)], dtype=torch.float64))
    assert torch.allclose(p.sum(-1)[0], torch.tensor([1 / 3, 2 / 4, 3 / 5], dtype=torch.float64))


def test_passes_repeat_a_run_of_layers():
    assert plain.layer_runs(case("A")) == [0, 1, 2, 0, 1, 2, 3]
    assert plain.layer_runs(case("C")) == [0, 1, 2, 3, 2, 3, 2, 3]
    assert plain.layer_runs(case("B")) == config_from_dict(case("B")).layer_runs()


def test_groups_are_ranked_by_their_two_best_and_negative_scores_stay_in_the_running():
    router = {"top": 2, "groups": {"count": 2, "keep": 1}}
    s = torch.tensor([[0.1, 0.1, 0.1, 0.9, 0.05, 0.05]])
    correction = torch.tensor([-0.4, -0.4, -0.5, -1.0, -1.3, -1.2])
    # corrected: -0.3 -0.3 -0.4 | -0.1 -1.25 -1.15: the second group has the best expert, the first the better two
    assert sorted(plain.choose(s, correction, router)[0].tolist()) == [0, 1]
    w = plain.route_weights(s, torch.tensor([[0, 3]]), 2.0)
    assert torch.allclose(w, torch.tensor([[0.2, 1.8]]), atol=1e-6)


def test_recurrence_against_its_closed_form():
    g = torch.Generator().manual_seed(2)
    T, H, K, V = 20, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (K, K, V))
    decay = torch.tensor([0.7, 0.99], dtype=torch.float64)
    o, S = plain.decayed_sums(q, k, v, decay)
    for h in range(H):
        for t in (0, 5, 19):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)
    first, mid = plain.decayed_sums(q[:7], k[:7], v[:7], decay)
    rest, end = plain.decayed_sums(q[7:], k[7:], v[7:], decay, state=mid)
    assert torch.allclose(torch.cat([first, rest]), o) and torch.allclose(end, S)


def test_slow_frequencies_are_scaled_and_the_library_scales_them_alike():
    from esp_b200.parts.position import RopeNeighbourPairs
    rot = {"dims": 24, "base": 500.0, "scaling": {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 200}}
    f = plain.frequencies(rot)
    base = plain.frequencies({"dims": 24, "base": 500.0})
    ratio = (f / base).numpy()
    length = 2 * math.pi / base.numpy()
    assert (ratio[length < 50] == 1).all() and np.allclose(ratio[length > 200], 1 / 6)
    between = ratio[(length > 50) & (length < 200)]
    assert len(between) >= 2 and ((between < 1) & (between > 1 / 6)).all() and (np.diff(between) < 0).all()
    mine, magnitude = RopeNeighbourPairs(GaliraxConfig._rotation(rot), None).exact_frequencies()
    assert magnitude == 1.0 and np.allclose(mine, f.numpy(), rtol=1e-14)
