"""The kernels behind the Galirax design, each alone against a float64 statement of the same mechanism, at sizes the model
tests do not have, with inputs made so that a fault shows: one key whose score stands out just inside and just outside a
window, at the last kept first token and just behind it; rows with a mean that dwarfs their spread; corrections that make
every choice score negative; groups whose best expert and whose two best disagree; decays of nearly one."""
import math

import numpy as np
import pytest
import torch

import plain_galirax as plain

from esp_b200.csrc import ops

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def dev(t, dtype=None):
    return t.to(DEV, dtype if dtype is not None else t.dtype).contiguous()


def i32(values):
    return torch.tensor(np.asarray(values), dtype=torch.int32, device=DEV)


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def paged(rows, table, n_pages, dtype):
    """rows [T, G, W] of one sequence -> pool [n_pages, G, PAGE, W] with position p in page table[p // PAGE]."""
    T, G, W = rows.shape
    pool = torch.zeros(n_pages, G, PAGE, W, dtype=dtype)
    for p in range(T):
        if table[p // PAGE] >= 0:
            pool[table[p // PAGE], :, p % PAGE] = rows[p].to(dtype)
    return pool


# ------------------------------------------------------------------------------------------------ attention
KERNELS = ["plain32", "plain16", "tensor16", "tmem16", "split16", "split16_long"]


def takes(kernel, K, V):
    if kernel.startswith("plain"):
        return True
    fits = K % 8 == 0 and V % 8 == 0
    return fits and (kernel.startswith("split") or max(K, V) <= 128)


def run_attention(kernel, q, k_pool, v_pool, out, table, first, new, H, G, K, V, scale, sink, window, keep):
    st = status()
    args = (q, k_pool, v_pool, out)
    tables = i32([table])
    opts = dict(vd=V, scale=scale, sink=sink, keep=keep)
    if kernel in ("tensor16", "tmem16"):
        rows = 64 if kernel == "tensor16" else ops.ATTN_TC05_TILE_ROWS
        firsts = list(range(0, new, rows))
        run = ops.attn_prefill if kernel == "tensor16" else ops.attn_prefill_tc05
        run(*args, i32([0] * len(firsts)), i32(firsts), i32([0, new]), i32([first]), tables, PAGE, H, G, K, window, st, **opts)
    elif kernel.startswith("split16"):
        split = 64 if kernel == "split16" else 256
        n_splits = (len(table) * PAGE + split - 1) // split
        part_o = torch.zeros(new, H, n_splits, ops.attn_decode_tile(K, V), device=DEV)
        part_ml = torch.zeros(new, H, n_splits, 2, device=DEV)
        counters = torch.zeros(ops.ATTN_DECODE_COUNTERS, dtype=torch.int32, device=DEV)
        for past in (None, i32([first])):                # with the positions cached before the step, early loads
            ops.attn_decode(*args, part_o, part_ml, counters, i32([0] * new), i32(list(range(first, first + new))), tables, PAGE, H,
                            G, K, window, split, n_splits, st, seq_past=past, **opts)
            assert int(counters.abs().sum().item()) == 0
    else:
        ops.attn_simt(*args, i32([0] * new), i32(list(range(first, first + new))), tables, PAGE, H, G, K, window, st, **opts)
    assert int(st.item()) == 0


def attention_rows(q, k, v, scale, first, mask, sink):
    """float64: rows first .. of one sequence; q [n, H, K], k [T, G, K], v [T, G, V]."""
    n, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    seen = plain.visible_keys(k.shape[0], mask)[first:first + n]
    scores = torch.einsum("thk,shk->hts", q, k.repeat_interleave(rep, dim=1)) * scale
    return torch.einsum("hts,shv->thv", plain.sink_softmax(scores, seen, sink), v.repeat_interleave(rep, dim=1))


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("H, G, K, V, window, keep", [
    (4, 2, 16, 40, 37, 3), (3, 1, 56, 88, 100, 1), (2, 2, 128, 128, 70, 66), (8, 2, 64, 64, 64, 64), (2, 1, 96, 96, 129, 5),
    (2, 1, 24, 24, 1, 130), (2, 2, 64, 64, 400, 10), (20, 1, 40, 72, 90, 200), (2, 2, 192, 136, 65, 63), (2, 1, 112, 8, 200, 300),
    (2, 1, 80, 128, 50, 0)])
@pytest.mark.parametrize("new", [200, 3])
def test_window_edges_and_kept_tokens_from_prompt_rows_and_from_single_rows(kernel, H, G, K, V, window, keep, new):
    """620 cached positions in pages handed out in no order, those that nobody sees given back; the new tokens are the last
    200 (a prompt's portion) or the last 3 (decoding).  For probed queries one key gets a large score: the oldest position
    the window holds, the one before it, the last kept first token, the one behind it, the first token, the query itself."""
    if not takes(kernel, K, V):
        pytest.skip("the tensor-core kernels want multiples of 8; those of many rows at most 128")
    dtype = torch.float32 if kernel == "plain32" else torch.bfloat16
    g = torch.Generator().manual_seed(window * 7 + new + keep)
    T = 620
    first = T - new
    q, k = torch.randn(new, H, K, generator=g) * 0.3, torch.randn(T, G, K, generator=g) * 0.3
    v = torch.randn(T, G, V, generator=g)
    used, kinds = set(), set()
    rows = sorted(set([0, 1, 2, new - 1, new // 2, new // 3, new // 4, new // 5, new - 2, new // 7, new // 9, new - 3]))
    for n, row in enumerate(rows):
        pos = first + row
        kind = (n + window) % 6
        key = [pos - window + 1, pos - window, keep - 1, keep, 0, pos][kind]
        if key < 0 or key > pos or (key, row % H // (H // G)) in used:
            continue
        used.add((key, row % H // (H // G)))
        kinds.add(kind)
        direction = torch.randn(K, generator=g)
        direction /= direction.norm()
        k[key, row % H // (H // G)] = direction * 6
        q[row, row % H] = direction * 6
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    sink = torch.randn(H, generator=g).double()
    scale = 0.9
    at = lambda size, kept: attention_rows(q, k, v, scale, first, {"size": size, "keep_first": kept}, sink)
    want = at(window, keep)
    # the probes tell a window or a run of kept tokens that is one position off
    for kind, other in ((0, (window - 1, keep)), (1, (window + 1, keep)), (2, (window, keep - 1)), (3, (window, keep + 1))):
        outside = keep <= first - window            # else the two meet and the edge is no edge
        if kind in kinds and other[0] > 0 and other[1] >= 0 and outside:
            assert (at(*other) - want).abs().max() > 0.3, kind
    needed = lambda i: any(first - window < p or p < keep for p in range(i * PAGE, (i + 1) * PAGE))
    order = [7, 2, 11, 0, 5, 13, 1, 9, 14, 3]
    table = [order[i] if needed(i) else -1 for i in range((T + PAGE - 1) // PAGE)]
    k_pool, v_pool = paged(k, table, 16, dtype), paged(v, table, 16, dtype)
    free = [p for p in range(16) if p not in table]
    k_pool[free], v_pool[free] = 50.0, 1000.0           # what must not be read
    out = torch.full((new, H, V), float("nan"), dtype=dtype, device=DEV)
    run_attention(kernel, dev(q, dtype).view(new, -1), dev(k_pool), dev(v_pool), out, table, first, new, H, G, K, V, scale,
                  dev(sink.float()), window, keep)
    err = (out.double().cpu() - want).abs()
    worst = int(err.amax((1, 2)).argmax())
    assert err.max() < (2e-5 if dtype == torch.float32 else 5e-2), (first + worst, float(err.max()))


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("width", [64, 100, 1000, 1030, 4096])
@pytest.mark.parametrize("n", [3, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("add", [True, False])
def test_layer_norm_behind_an_add(width, n, dtype, add):
    """Rows whose mean is a hundred times their spread: a variance as the mean square less the squared mean would lose it."""
    g = torch.Generator().manual_seed(width + n)
    x, y = torch.randn(n, width, generator=g) + 100.0 * torch.randn(n, 1, generator=g), torch.randn(n, width, generator=g)
    w, b, eps = 1 + 0.3 * torch.randn(width, generator=g), torch.randn(width, generator=g), 1e-3
    v = x.double() + (y.double() if add else 0)
    want = plain.layer_norm((x + y if add else x).double(), w.double(), b.double(), eps)
    xd, h, h32 = dev(x), torch.zeros(n, width, dtype=dtype, device=DEV), torch.zeros(n, width, device=DEV)
    ops.add_rmsnorm(xd, dev(y) if add else None, dev(w), h, eps, h32=h32, beta=dev(b))
    assert (xd.cpu().double() - v).abs().max() < 1e-4
    assert (h32.cpu().double() - want).abs().max() < 2e-4          # the mean is a float of the order of 100
    near = 2e-4 if dtype == torch.float32 else 2.0 ** -8 * float(want.abs().max())
    assert (h.cpu().double() - want).abs().max() < near
    rows = i32([n - 1, 0])
    picked = torch.zeros(2, width, dtype=dtype, device=DEV)
    ops.add_rmsnorm(dev(x), dev(y) if add else None, dev(w), picked, eps, rows=rows, write_x=False, beta=dev(b))
    assert (picked.cpu().double() - want[[n - 1, 0]]).abs().max() < near


@pytest.mark.parametrize("width, n, top", [(64, 5, 2), (1024, 3, 4), (2048, 300, 3)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sum_of_experts_and_mixer_then_layer_norm(width, n, top, dtype):
    g = torch.Generator().manual_seed(width)
    E = 7
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)]).int()
    inverse = torch.randperm(n * top, generator=g).view(n, top).int()
    rows, mixed = torch.randn(n * top, width, generator=g), torch.randn(n, width, generator=g)
    x, w, b = torch.randn(n, width, generator=g) * 3 + 20, 1 + 0.3 * torch.randn(width, generator=g), torch.randn(width, generator=g)
    v = x.double() + mixed.double() + rows.double()[inverse.long()].sum(1)
    want = plain.layer_norm(v, w.double(), b.double(), 1e-5)
    xd, h, h32 = dev(x), torch.zeros(n, width, dtype=dtype, device=DEV), torch.zeros(n, width, device=DEV)
    ops.moe_combine_add_rmsnorm(dev(rows), dev(ids), dev(inverse), None, dev(mixed), xd, dev(w), h, 1e-5, h32=h32, beta=dev(b))
    assert (xd.cpu().double() - v).abs().max() < 1e-4
    assert (h32.cpu().double() - want).abs().max() < 1e-4
    assert (h.cpu().double() - want).abs().max() < (1e-4 if dtype == torch.float32 else 3e-2)


# ------------------------------------------------------------------------------------------------ rotation
@pytest.mark.parametrize("H, G, K, V, rot", [(3, 1, 24, 40, 8), (2, 2, 64, 64, 64), (4, 2, 16, 8, 2), (1, 1, 128, 128, 0),
                                             (5, 5, 10, 12, 10), (3, 3, 36, 20, 30), (16, 16, 96, 96, 96), (40, 40, 128, 128, 64), (50, 50, 128, 128, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_biases_norms_over_the_projection_and_rotation_of_neighbours(H, G, K, V, rot, dtype):
    """Positions from 0 to beyond a million, every one in a sequence of its own; one head is a hundred times larger than the
    others: a norm per head would not show it in them."""
    g = torch.Generator().manual_seed(K + rot)
    positions = [0, 1, 63, 64, 65, 1000, 99999, 1048575]
    n, width = len(positions), H * K + G * K + G * V
    qkv, bias = torch.randn(n, width, generator=g), torch.randn(width, generator=g)
    qkv[:, :K] *= 100.0
    q_w, k_w, eps = 1 + 0.3 * torch.randn(H * K, generator=g), 1 + 0.3 * torch.randn(G * K, generator=g), 1e-5
    spec = {"dims": rot, "base": 300.0, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 500}} if rot else None
    x = qkv.double() + bias.double()
    q_want = (plain.unit_rms(x[:, :H * K], eps) * q_w.double()).view(n, H, K)
    k_want = (plain.unit_rms(x[:, H * K:(H + G) * K], eps) * k_w.double()).view(n, G, K)
    v_want = x[:, (H + G) * K:].view(n, G, V)
    f = lo = None
    if rot:
        exact = plain.frequencies(spec)
        f = exact.float()
        lo = (exact - f.double()).float()
        q_want, k_want = (plain.rotate_neighbours(t, torch.tensor(positions), spec) for t in (q_want, k_want))
    pages_per, n_pages = max(positions) // PAGE + 1, 24
    table = torch.full((n, pages_per), -1, dtype=torch.int32)
    for i, p in enumerate(positions):
        table[i, p // PAGE] = n_pages - 1 - 2 * i
    k_cache, v_cache = torch.zeros(n_pages, G, PAGE, K, dtype=dtype, device=DEV), torch.zeros(n_pages, G, PAGE, V, dtype=dtype, device=DEV)
    q_out, st = torch.zeros(n, H * K, dtype=dtype, device=DEV), status()
    ops.widenorm_rope_kvwrite(dev(qkv), dev(q_w), dev(k_w), eps, dev(f) if rot else None, rot, 1.0, i32(list(range(n))),
                              i32(positions), q_out, k_cache, v_cache, dev(table), PAGE, H, G, K, V, True, st, bias=dev(bias),
                              neighbour=True, inv_freq_lo=dev(lo) if rot else None)
    assert int(st.item()) == 0
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    big = float(q_want.abs().max())
    assert (q_out.double().cpu().view(n, H, K) - q_want).abs().max() < tol * big
    for i, p in enumerate(positions):
        page = n_pages - 1 - 2 * i
        assert (k_cache[page, :, p % PAGE].double().cpu() - k_want[i]).abs().max() < tol * 5
        assert (v_cache[page, :, p % PAGE].double().cpu() - v_want[i]).abs().max() < tol * 5
    assert int((k_cache != 0).any(-1).sum().item()) <= n * G and int((v_cache != 0).any(-1).sum().item()) <= n * G


# ------------------------------------------------------------------------------------------------ router
@pytest.mark.parametrize("n, width, wdtype", [(5, 96, torch.float32), (40, 128, torch.bfloat16), (100, 96, torch.float32),
                                              (300, 256, torch.bfloat16), (70, 100, torch.bfloat16)])
@pytest.mark.parametrize("experts, top, groups, keep, scale", [(18, 4, 3, 1, 2.5), (9, 2, 3, 2, 1.0), (6, 6, 0, 0, 0.7), (12, 4, 4, 2, 3.0),
                                                               (40, 8, 1, 1, 1.5), (5, 2, 5, 3, 2.0), (64, 8, 8, 4, 2.5)])
def test_sigmoid_scores_in_groups_ranked_by_their_two_best(n, width, wdtype, experts, top, groups, keep, scale):
    """Every path of the router against the float64 choice.  The corrections make every choice score negative, so a shut-out
    group counted as zero would win; every group has one expert whose correction makes it the best of all now and then, so
    that ranking groups by their best alone chooses otherwise."""
    g = torch.Generator().manual_seed(n + experts)
    h = torch.randn(n, width, generator=g)
    w_router = (torch.randn(experts, width, generator=g) * (1.5 / math.sqrt(width))).to(wdtype).float()
    correction = torch.randn(experts, generator=g) * 0.4 - 3.0
    spec = {"experts": experts, "top": top}
    if groups:
        spec["groups"] = {"count": groups, "keep": keep}
    s = plain.sigmoid(h.double() @ w_router.double().T)
    ids_want = plain.choose(s, correction.double(), spec)
    if groups > 2 and keep < groups and experts // groups > 1:
        per = experts // groups
        scores = (s + correction.double()).view(n, groups, per)
        by_one = scores.max(-1).values.topk(keep, dim=-1).indices.sort(-1).values
        by_two = scores.topk(2, dim=-1).values.sum(-1).topk(keep, dim=-1).indices.sort(-1).values
        assert n < 40 or (by_one != by_two).any()         # the inputs tell the two rankings apart
    ids, wts = torch.zeros(n, top, dtype=torch.int32, device=DEV), torch.zeros(n, top, device=DEV)
    logits, st = torch.zeros(n, experts + 1, device=DEV), status()
    choice = (dev(correction), groups, keep, 2)
    hd, wd = dev(h), dev(w_router, wdtype)
    if n <= ops.ROUTE_SMALL_TOKENS:
        ints = lambda k: torch.zeros(k, dtype=torch.int32, device=DEV)
        ops.route_small(hd, wd, None, logits, ids, wts, None, top, True, ints(experts + 1), ints(n * top),
                        torch.zeros(n * top, device=DEV), ints(n * top).view(n, top), st, choice=choice, sigmoid=True, scale=scale)
    else:
        ops.router_topk(hd, wd, None, ids, wts, None, top, True, st, logits=logits, choice=choice, sigmoid=True, scale=scale)
    assert int(st.item()) == 0
    got, w = ids.cpu().long(), wts.cpu().double()
    differ = sum(set(got[t].tolist()) != set(ids_want[t].tolist()) for t in range(n))
    assert differ <= n // 100                            # scores that 32-bit rounding cannot tell apart
    assert all(len(set(got[t].tolist())) == top for t in range(n))
    assert (w - plain.route_weights(s, got, scale)).abs().max() < 1e-5 * scale


def test_scores_that_all_vanish_leave_no_weight():
    """Logits of minus two hundred: every score is zero in 32-bit, the sum is divided by with 1e-20 added, nothing is
    reported and nothing is not a number."""
    h, w = torch.full((3, 64), -1.0), torch.full((4, 64), 200.0 / 64)
    ids, wts, st = torch.zeros(3, 2, dtype=torch.int32, device=DEV), torch.full((3, 2), 9.0, device=DEV), status()
    ops.router_topk(dev(h), dev(w), None, ids, wts, None, 2, True, st, choice=(dev(torch.zeros(4)), 0, 0, 2), sigmoid=True, scale=2.0)
    assert int(st.item()) == 0 and float(wts.abs().max()) == 0.0


# ------------------------------------------------------------------------------------------------ linear attention
def lightning_inputs(rows, H, K, V, g):
    q, k, v = (torch.randn(rows, H * n, generator=g) * 1.5 for n in (K, K, V))
    return q, k, v


def lightning_want(q, k, v, H, decay, state):
    """state [H, K, V] float64 -> ([rows, H * V], new state)."""
    n = q.shape[0]
    o, S = plain.decayed_sums(*(plain.silu(t.double()).view(n, H, -1) for t in (q, k, v)), torch.tensor(decay, dtype=torch.float64), state)
    return o.reshape(n, -1), S


def halves(decay):
    exact = np.asarray(decay, dtype=np.float64)
    return dev(torch.from_numpy(exact.astype(np.float32))), dev(torch.from_numpy((exact - exact.astype(np.float32)).astype(np.float32)))


@pytest.mark.parametrize("H, K, V, decay", [(3, 16, 24, [0.2, 0.97, 0.9999]), (2, 10, 7, [0.0, 1.0]), (1, 256, 40, [0.995]),
                                            (2, 64, 128, [0.9, 0.9995]), (1, 132, 4, [0.98]), (2, 36, 100, [0.3, 1.0])])
@pytest.mark.parametrize("cuts", [[150], [1] * 12 + [138], [2, 3, 64, 81], [149, 1]])
@pytest.mark.parametrize("kernel", ["scan", "steps"])
def test_recurrence_with_a_fixed_decay_over_any_cutting(H, K, V, decay, cuts, kernel):
    """Two sequences in slots 3 and 0.  Every cutting ends in the float64 outputs and states, by the kernel that walks its
    rows through shared memory and by the one that keeps the state in registers."""
    if kernel == "steps" and not ops.linear_attn_chunks_fits(K, V):
        pytest.skip("this kernel wants multiples of 4")
    g = torch.Generator().manual_seed(K + V)
    total = sum(cuts)
    seqs = [lightning_inputs(total, H, K, V, g) for _ in range(2)]
    start = torch.randn(2, H, K, V, generator=g, dtype=torch.float64)
    state = torch.zeros(5, H * V * K + 4, device=DEV)
    for slot, s0 in zip((3, 0), start):
        state[slot, :H * V * K] = dev(s0.transpose(1, 2).reshape(-1).float())
    d, rest = halves(decay)
    outs, at = [[], []], 0
    for n in cuts:
        q, k, v = (dev(torch.cat([seqs[0][i][at:at + n], seqs[1][i][at:at + n]])) for i in range(3))
        o = torch.zeros(2 * n, H * V, device=DEV)
        if kernel == "scan":
            ops.gated_scan(ops.SCAN_FIXED_DECAY, q, k, d, v, None, rest, None, state, i32([0, n, 2 * n]), i32([3, 0]), o, 2, H, K, V)
        else:
            rows = torch.cat([q, k, v], dim=1)
            ops.linear_attn_steps(rows[:, :H * K], rows[:, H * K:2 * H * K], rows[:, 2 * H * K:], d, rest, state, i32([0, n, 2 * n]),
                                  i32([3, 0]), o, 2, H, K, V)
        outs[0].append(o[:n].cpu())
        outs[1].append(o[n:].cpu())
        at += n
    for i, slot in enumerate((3, 0)):
        want, S = lightning_want(*seqs[i], H, decay, start[i])
        got = torch.cat(outs[i]).double()
        tol = 3e-6 if kernel == "scan" else 1e-5            # the second takes its SiLUs from the fast exponential
        assert (got - want).abs().max() < tol * want.abs().max()
        end = state[slot, :H * V * K].cpu().double().view(H, V, K).transpose(1, 2)
        assert (end - S).abs().max() < tol * S.abs().max()
    assert float(state[1].abs().max()) == 0 and float(state[:, H * V * K:].abs().max()) == 0


def test_a_decay_of_nearly_one_over_thousands_of_tokens():
    """One token is written, 6,000 empty ones follow: what is left is decay^6000, which the decay's own rounding to 32 bits
    would move by 1e-4."""
    decay, T = [0.9997], 6000
    q, k, v = torch.full((T + 1, 1), 2.0), torch.full((T + 1, 1), -200.0), torch.full((T + 1, 1), 2.0)   # SiLU(-200) is zero
    k[0] = 2.0
    d, rest = halves(decay)
    state, o = torch.zeros(1, 1, device=DEV), torch.zeros(T + 1, 1, device=DEV)
    ops.gated_scan(ops.SCAN_FIXED_DECAY, dev(q), dev(k), d, dev(v), None, rest, None, state, i32([0, T + 1]), i32([0]), o, 1, 1, 1, 1)
    silu2 = float(plain.silu(torch.tensor(2.0, dtype=torch.float64)))
    assert abs(float(o[-1]) / (silu2 ** 3 * decay[0] ** T) - 1) < 5e-6


@pytest.mark.parametrize("rows, width", [(3, 24), (70, 300), (5, 1024), (2, 1030), (3, 5000)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_of_all_heads_as_one_row_with_a_sigmoid_gate(rows, width, dtype):
    g = torch.Generator().manual_seed(width)
    o, gate, w = torch.randn(rows, width, generator=g) * 3, torch.randn(rows, width + 4, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    want = plain.unit_rms(o.double(), 1e-5) * w.double() * plain.sigmoid(gate[:, :width].double())
    y = torch.zeros(rows, width, dtype=dtype, device=DEV)
    ops.head_rmsnorm_gate(dev(o), dev(w), 0, dev(gate)[:, :width], y, 1, width, 1e-5, gate_sigmoid=True)
    assert (y.double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("H, K, V, decay", [(3, 16, 24, [0.2, 0.97, 0.9999]), (2, 44, 100, [0.0, 1.0]), (1, 256, 40, [0.995]),
                                            (2, 128, 128, [0.9, 0.9995]), (1, 64, 8, [0.5])])
@pytest.mark.parametrize("cuts", [[300], [64, 1, 63, 65, 107], [17, 283], [2, 3, 128, 167]])
@pytest.mark.parametrize("at_once", [1, 3, 100])
def test_chunks_on_the_tensor_cores_over_any_cutting(H, K, V, decay, cuts, at_once):
    """Three sequences in slots 3, 0 and 2 (the second brings a tenth of the tokens of the others, down to one), every cutting,
    with room for one chunk's states, three and all of them.  What the state holds is made of values rounded to 8 bits and of
    keys that are not; the outputs of rounded queries, keys and values."""
    g = torch.Generator().manual_seed(K + V)
    shares = [[n, max(1, n // 10), n] for n in cuts]
    totals = [sum(s[i] for s in shares) for i in range(3)]
    seqs = [lightning_inputs(t, H, K, V, g) for t in totals]
    start = torch.randn(3, H, K, V, generator=g, dtype=torch.float64) * 3
    state, slots = torch.zeros(5, H * V * K + 4, device=DEV), [3, 0, 2]
    for slot, s0 in zip(slots, start):
        state[slot, :H * V * K] = dev(s0.transpose(1, 2).reshape(-1).float())
    powers = dev(torch.from_numpy((np.asarray(decay)[:, None] ** np.arange(ops.LINEAR_CHUNK + 1)).astype(np.float32)))
    scratch = torch.full((at_once * H * K * V,), float("nan"), device=DEV)
    outs, at = [[], [], []], [0, 0, 0]
    for news in shares:
        starts = [0, news[0], news[0] + news[1], sum(news)]
        rows = torch.cat([torch.cat([seqs[i][j][at[i]:at[i] + news[i]] for i in range(3)]) for j in range(3)], dim=1)
        rows = dev(torch.cat([rows, torch.full((starts[-1], 4), 7.0)], dim=1))
        chunks = [(i, f) for i, t in enumerate(news) for f in range(0, t, ops.LINEAR_CHUNK)]
        ranges = np.concatenate([[0], np.cumsum([-(-t // ops.LINEAR_CHUNK) for t in news])])
        o = torch.full((starts[-1], H * V), float("nan"), device=DEV)
        ops.linear_attn_chunks(rows[:, :H * K], rows[:, H * K:2 * H * K], rows[:, 2 * H * K:2 * H * K + H * V], i32([c[0] for c in chunks]),
                               i32([c[1] for c in chunks]), i32(ranges), i32(starts), i32(slots), powers, scratch, state, o, 3, H, K, V)
        for i in range(3):
            outs[i].append(o[starts[i]:starts[i + 1]].cpu())
            at[i] += news[i]
    rounded = lambda t: t.to(torch.bfloat16).double()
    for i, slot in enumerate(slots):
        q, k, v = (plain.silu(t.double()).view(totals[i], H, -1) for t in seqs[i])
        d = torch.tensor(decay, dtype=torch.float64)
        _, S = plain.decayed_sums(q, k, rounded(v), d, start[i])
        end = state[slot, :H * V * K].cpu().double().view(H, V, K).transpose(1, 2)
        for h in range(H):
            assert (end[h] - S[h]).abs().max() < 3e-5 * S[h].abs().max(), h
        want, _ = plain.decayed_sums(rounded(q), k, rounded(v), d, start[i])
        got = torch.cat(outs[i]).double().view(totals[i], H, V)
        for h in range(H):
            assert (got[:, h] - want[:, h]).abs().max() < 6e-3 * want[:, h].abs().max(), h
    assert float(state[1].abs().max()) == 0 and float(state[:, H * V * K:].abs().max()) == 0


def test_a_key_far_back_is_read_through_the_chunks():
    """One token among 1,500 has a key that the last query alone points at: it is read through twenty-three chunks' states."""
    H, K, V, T, decay = 1, 64, 64, 1500, [0.9995]
    g = torch.Generator().manual_seed(4)
    q, k, v = (torch.randn(T, n, generator=g) * 0.2 for n in (K, K, V))
    k[3], q[-1] = torch.where(torch.rand(K, generator=g) < 0.5, 8.0, -30.0), 0.0
    q[-1] = torch.where(k[3] > 0, 8.0, -30.0)
    v[3] = 10 * torch.rand(V, generator=g)
    rows = dev(torch.cat([q, k, v], dim=1))
    firsts = list(range(0, T, ops.LINEAR_CHUNK))
    powers = dev(torch.from_numpy((np.asarray(decay)[:, None] ** np.arange(ops.LINEAR_CHUNK + 1)).astype(np.float32)))
    state, o = torch.zeros(1, K * V, device=DEV), torch.zeros(T, V, device=DEV)
    ops.linear_attn_chunks(rows[:, :K], rows[:, K:2 * K], rows[:, 2 * K:], i32([0] * len(firsts)), i32(firsts), i32([0, len(firsts)]),
                           i32([0, T]), i32([0]), powers, torch.zeros(len(firsts) * K * V, device=DEV), state, o, 1, H, K, V)
    want, _ = lightning_want(q, k, v, H, decay, None)
    alone, _ = lightning_want(q[-1:], k[3:4], v[3:4], H, [1.0], None)
    assert (want[-1] - alone[0] * decay[0] ** (T - 4)).abs().max() < 0.2 * want[-1].abs().max()      # the probe stands out
    assert (o[-1].double().cpu() - want[-1]).abs().max() < 6e-3 * want[-1].abs().max()
