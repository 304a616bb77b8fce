"""The kernels behind the Satavik design, each alone against a float64 statement of the same mechanism, at sizes the
model tests do not have, with inputs made so that a fault shows: one key whose score stands out just inside and just
outside a block of positions, in one map and not in the other; scores far beyond the soft cap and scores on both sides
of where its evaluation changes; routers whose logits differ by hundreds; gates and up branches beyond their limits."""
import math

import numpy as np
import pytest
import torch

import plain_satavik as plain

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
        pool[table[p // PAGE], :, p % PAGE] = rows[p].to(dtype)
    return pool


# ------------------------------------------------------------------------------------------------ attention
KERNELS = ["plain32", "plain16", "tmem16", "split16"]


def takes(kernel, K, V):
    return kernel.startswith("plain") or (K % 8 == 0 and V % 8 == 0 and K <= 128)


def run_attention(kernel, q, k_pool, v_pool, tables, rows, starts, pasts, H, G, K, V, scale, cap, chunk, lam, eps, out_scale, gate,
                  split=128):
    """``rows``: (sequence, position) of every query row; returns [N, H, V]."""
    st, n, dtype = status(), len(rows), q.dtype
    out = torch.zeros(n, H, V, dtype=dtype, device=DEV)
    maps = torch.full((n, 2 * H, V), float("nan"), device=DEV)
    tok_seq, tok_pos = i32([r[0] for r in rows]), i32([r[1] for r in rows])
    args = dict(softcap=cap, chunk=chunk)
    if kernel == "tmem16":
        news = [b - a for a, b in zip(starts, starts[1:])]
        tiles = [(s, f) for s, t in enumerate(news) for f in range(0, t, ops.ATTN_TC05_TILE_ROWS)]
        ops.attn_diff_tc05(q, k_pool, v_pool, out, maps, i32([t[0] for t in tiles]), i32([t[1] for t in tiles]), i32(starts),
                           i32(pasts), tables, PAGE, H, G, K, V, scale, st, lam, eps, out_scale, gate=gate, **args)
        if V > ops.ATTN_DIFF_FUSED_VALUES:
            ops.diff_combine(maps, lam, eps, out_scale, gate, out)
    elif kernel == "split16":
        n_splits = (tables.shape[1] * PAGE + split - 1) // split
        part_o = torch.zeros(n, 2 * H, n_splits, ops.attn_diff_tile(V), device=DEV)
        part_ml = torch.zeros(n, 2 * H, n_splits, 2, device=DEV)
        counters = torch.zeros(ops.ATTN_DECODE_COUNTERS, dtype=torch.int32, device=DEV)
        ops.attn_decode_diff(q, k_pool, v_pool, out, part_o, part_ml, counters, tok_seq, tok_pos, tables, PAGE, H, G, K, V, scale,
                             split, n_splits, st, lam, eps, out_scale, gate=gate, **args)
        assert int(counters.abs().sum().item()) == 0
    else:
        ops.attn_simt(q, k_pool, v_pool, maps, tok_seq, tok_pos, tables, PAGE, 2 * H, G, K, None, st, vd=V, scale=scale, maps=2,
                      **args)
        ops.diff_combine(maps, lam, eps, out_scale, gate, out)
    assert int(st.item()) == 0
    return out.double().cpu()


def difference(q, k, v, first, chunk, scale, cap, lam, eps, out_scale, gate):
    """float64: new rows first .. of one sequence; q [n, H, 2, K], k [T, G, 2, K], v [T, G, V]."""
    n, H = q.shape[0], q.shape[1]
    T = k.shape[0]
    seen = plain.visible_keys(T, chunk)[first:first + n]
    vals = v.repeat_interleave(H // v.shape[1], dim=1)
    a = [torch.einsum("hts,shv->thv", plain.map_weights(q[:, :, m], k[:, :, m], scale, cap, seen), vals) for m in (0, 1)]
    return plain.unit_rms(a[0] - lam * a[1], eps) * out_scale * plain.sigmoid(gate)[:, :, None]


BOUND16 = 0.02          # of the largest output; weights and outputs are rounded to 8 bits


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("H, G, K, V, chunk, cap", [
    (4, 2, 24, 40, 37, 6.0), (3, 1, 56, 88, 100, 50.0), (2, 2, 64, 128, 70, 30.0), (8, 2, 64, 64, 64, None),
    (6, 3, 128, 128, 129, 20.0), (2, 1, 64, 128, 1, 30.0), (2, 2, 32, 64, None, 15.0), (20, 1, 16, 32, 200, 90.0),
    (2, 1, 128, 256, 150, 25.0), (1, 1, 72, 136, None, None), (10, 2, 8, 8, 128, 4.0), (2, 2, 96, 72, 64, 61.0)])
@pytest.mark.parametrize("new", [200, 3])
def test_block_edges_from_prompt_rows_and_from_single_rows(kernel, H, G, K, V, chunk, cap, new):
    """460 cached positions in pages handed out in no order; the new tokens are the last 200 (a prompt's portion) or the
    last 3 (decoding).  For probed queries one key of one map gets a large score: the block's first position (just
    inside), the one before it (just outside: it must not count), the query itself, its predecessor, a page's first."""
    if not takes(kernel, K, V):
        pytest.skip("the tensor-core kernels want multiples of 8, keys up to 128")
    dtype = torch.float32 if kernel == "plain32" else torch.bfloat16
    g = torch.Generator().manual_seed((chunk or 7) * 3 + new + K)
    T, first = 460, 460 - new
    q, k = torch.randn(new, H, 2, K, generator=g) * 0.3, torch.randn(T, G, 2, K, generator=g) * 0.3
    v = torch.randn(T, G, V, generator=g)
    kinds = set()
    for n, row in enumerate(sorted(set([0, 1, 2, new - 1, new // 2, new // 3, new // 4, new // 5, new - 2, new // 7]))):
        pos = first + row
        start = pos - pos % chunk if chunk else 0
        key = [start, start - 1, pos, pos - 1, pos - pos % PAGE][n % 5]
        if key < 0 or key > pos:
            continue
        kinds.add(n % 5)
        head, m = row % H, (row // 2) % 2
        direction = torch.randn(K, generator=g)
        direction /= direction.norm()
        k[key, head // (H // G), m] = direction * 6
        q[row, head, m] = direction * 6
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    gate = torch.randn(new, H, generator=g)
    lam, eps, out_scale, scale = 0.6, 1e-5, 0.7, 0.5
    want = difference(q, k, v, first, chunk, scale, cap, lam, eps, out_scale, gate.double())
    big = want.abs().max()
    # the probes tell blocks that begin one position off
    if chunk not in (None, 1) and 1 in kinds and (new > 3 or chunk < 30):
        seen = plain.visible_keys

        def shifted(T_, c):
            t = torch.arange(T_)
            return (t[None, :] <= t[:, None]) & ((t[None, :] + 1) // c >= t[:, None] // c)
        plain.visible_keys = shifted
        try:
            assert (difference(q, k, v, first, chunk, scale, cap, lam, eps, out_scale, gate.double()) - want).abs().max() > 0.1 * big
        finally:
            plain.visible_keys = seen
    need = (first - first % chunk) if chunk else 0
    order = [7, 2, 11, 0, 5, 13, 1, 9]
    table = [order[i] if (i + 1) * PAGE > need else -1 for i in range((T + PAGE - 1) // PAGE)]
    at = [max(t, 0) for t in table]
    rows_of_gate = torch.zeros(new, 3 * H + 5)
    rows_of_gate[:, H:2 * H] = gate
    got = run_attention(kernel, dev(q.reshape(new, -1), dtype), dev(paged(k.reshape(T, G, 2 * K), at, 16, dtype)),
                        dev(paged(v, at, 16, dtype)), i32([table]), [(0, first + i) for i in range(new)], [0, new], [first], H, G, K, V,
                        scale, cap, chunk, lam, eps, out_scale, dev(rows_of_gate)[:, H:2 * H])
    err = (got - want).abs().amax((1, 2))
    bound = (2e-5 if dtype == torch.float32 else BOUND16) * big
    assert float(err.max()) <= bound, (int(err.argmax()), float(err.max()), float(big))


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("cap", [3.0, 40.0, 60.0, 70.0, 200.0])
def test_soft_cap_from_small_scores_to_scores_far_beyond_it(kernel, cap):
    """Scores from a fiftieth of the cap to ten times the cap, both signs, some rows all small (the polynomial), some all
    large (the exponential form), some both; with scores that large the cap decides every weight."""
    dtype = torch.float32 if kernel == "plain32" else torch.bfloat16
    g = torch.Generator().manual_seed(int(cap))
    T, H, G, K, V = 200, 2, 1, 32, 64
    q, k = torch.randn(T, H, 2, K, generator=g), torch.randn(T, G, 2, K, generator=g)
    target = cap * torch.logspace(math.log10(0.02), math.log10(10.0), T)
    q = q * (target / math.sqrt(K))[torch.randperm(T, generator=g), None, None, None]
    q, k, v = (t.to(dtype).double() for t in (q, k, torch.randn(T, G, V, generator=g)))
    gate = torch.randn(T, H, generator=g)
    want = difference(q, k, v, 0, None, 1.0, cap, 0.4, 1e-6, 0.6, gate.double())
    table = [3, 0, 2, 1]
    got = run_attention(kernel, dev(q.reshape(T, -1), dtype), dev(paged(k.reshape(T, G, 2 * K), table, 4, dtype)),
                        dev(paged(v, table, 4, dtype)), i32([table]), [(0, i) for i in range(T)], [0, T], [0], H, G, K, V, 1.0, cap,
                        None, 0.4, 1e-6, 0.6, dev(gate))
    err = (got - want).abs().amax((1, 2))
    # a row's difference may nearly cancel, and its norm then magnifies what rounding leaves of it: the bulk is held tightly
    rel = err / want.abs().amax()
    assert float(rel.median()) <= (1e-5 if dtype == torch.float32 else 0.01)
    assert float(rel.quantile(0.95)) <= (1e-4 if dtype == torch.float32 else 0.04), (float(rel.quantile(0.95)), int(rel.argmax()))


@pytest.mark.parametrize("kernel", KERNELS)
def test_what_is_left_of_two_maps_that_nearly_cancel(kernel):
    """A second map's weight of 0.998: rows with one visible key leave 0.002 of its value, whose direction must survive
    (both maps return the value itself, whatever their weights); with a weight of 1.002 it turns around."""
    dtype = torch.float32 if kernel == "plain32" else torch.bfloat16
    g = torch.Generator().manual_seed(8)
    T, H, G, K, V, cap = 160, 2, 1, 24, 40, 11.0
    q, k, v = (t.to(dtype).double() for t in (torch.randn(T, H, 2, K, generator=g), torch.randn(T, G, 2, K, generator=g),
                                              torch.randn(T, G, V, generator=g)))
    for lam in (0.998, 1.002):
        got = run_attention(kernel, dev(q.reshape(T, -1), dtype), dev(paged(k.reshape(T, G, 2 * K), [1, 0, 2], 3, dtype)),
                            dev(paged(v, [1, 0, 2], 3, dtype)), i32([[1, 0, 2]]), [(0, i) for i in range(T)], [0, T], [0], H, G, K, V, 0.5,
                            cap, 16, lam, 1e-9, 1.0, None)
        want = plain.unit_rms(v, 1e-12) * math.copysign(1, 1 - lam)
        first = torch.arange(0, T, 16)
        assert (got[first] - want[first]).abs().max() < (2e-3 if dtype == torch.float32 else 0.03)


@pytest.mark.parametrize("H, G, K, V, chunk, cap", [(4, 2, 64, 128, 96, 30.0), (2, 1, 128, 64, None, None), (3, 3, 40, 200, 300, 12.0)])
def test_unequal_runs_through_the_tensor_memory_kernel(H, G, K, V, chunk, cap):
    """Five sequences of unequal lengths with unequal pasts in one launch, more items than the device has SMs."""
    g = torch.Generator().manual_seed(H * 100 + V)
    news, pasts = [400, 7, 129, 256, 500], [0, 70, 333, 64, 1]
    starts = [0] + list(np.cumsum(news))
    n, perm = sum(news), torch.randperm(64, generator=g).tolist()
    tables, ks, vs, qs, want = [], [], [], [], []
    k_pool, v_pool = torch.zeros(64, G, PAGE, 2 * K, dtype=torch.bfloat16), torch.zeros(64, G, PAGE, V, dtype=torch.bfloat16)
    gate = torch.randn(n, H, generator=g)
    for s, (new, past) in enumerate(zip(news, pasts)):
        T = new + past
        q = (torch.randn(new, H, 2, K, generator=g) * 0.6).bfloat16()
        k = (torch.randn(T, G, 2, K, generator=g) * 0.6).bfloat16()
        v = torch.randn(T, G, V, generator=g).bfloat16()
        table = [perm.pop() for _ in range((T + PAGE - 1) // PAGE)]
        for p in range(T):
            k_pool[table[p // PAGE], :, p % PAGE] = k[p].reshape(G, 2 * K)
            v_pool[table[p // PAGE], :, p % PAGE] = v[p]
        tables.append(table + [-1] * (12 - len(table)))
        qs.append(q.reshape(new, -1))
        want.append(difference(q.double(), k.double(), v.double(), past, chunk, 0.35, cap, 0.5, 1e-5, 0.5,
                               gate[starts[s]:starts[s + 1]].double()))
    rows = [(s, past + i) for s, (new, past) in enumerate(zip(news, pasts)) for i in range(new)]
    got = run_attention("tmem16", dev(torch.cat(qs)), dev(k_pool), dev(v_pool), i32(tables), rows, starts, pasts, H, G, K, V, 0.35,
                        cap, chunk, 0.5, 1e-5, 0.5, dev(gate))
    want = torch.cat(want)
    err = (got - want).abs().amax((1, 2))
    assert float(err.max()) <= 0.03 * float(want.abs().max()), (rows[int(err.argmax())], float(err.max()))


def test_splits_do_not_show(capsys):
    """The split-key kernel with splits of 64, 128 and the whole row: the same row to within rounding."""
    g = torch.Generator().manual_seed(3)
    T, H, G, K, V = 700, 4, 2, 48, 96
    q = torch.randn(2, H * 2 * K, generator=g).bfloat16()
    k, v = torch.randn(T, G, 2 * K, generator=g).bfloat16(), torch.randn(T, G, V, generator=g).bfloat16()
    table = list(range(11))
    outs = [run_attention("split16", dev(q), dev(paged(k, table, 11, torch.bfloat16)), dev(paged(v, table, 11, torch.bfloat16)),
                          i32([table]), [(0, T - 1), (0, T - 2)], [0, 2], [T - 2], H, G, K, V, 0.2, 25.0, None, 0.5, 1e-5, 0.5, None,
                          split=s) for s in (64, 128, 768)]
    assert float((outs[0] - outs[2]).abs().max()) <= 0.01 and float((outs[1] - outs[2]).abs().max()) <= 0.01


# ------------------------------------------------------------------------------------------------ ahead of the attention
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, hd, vd, rot, own", [(4, 2, 64, 128, 64, True), (3, 1, 20, 13, 6, True), (5, 5, 24, 40, 8, True),
                                                       (2, 1, 48, 96, 0, True), (8, 2, 128, 8, 32, False), (40, 8, 128, 64, 128, True)])
def test_norm_rotation_and_cache_write(dtype, nh, nkv, hd, vd, rot, own):
    g = torch.Generator().manual_seed(nh * 31 + hd)
    n, extra, eps, base = 9, 7 if hd % 8 else 8, 1e-5, 3000.0
    q_width, k_width = nh * 2 * hd, nkv * 2 * hd
    width = q_width + (k_width + nkv * vd if own else 0) + extra
    rows = torch.randn(n, width, generator=g) * 2
    qw, kw = 1 + 0.5 * torch.randn(hd, generator=g), 1 + 0.5 * torch.randn(hd, generator=g)
    pos = [0, 1, 63, 64, 65, 200, 517, 700, 1023]      # (a 32-bit angle alone would be off by 6e-5 at the last)
    table = torch.randperm(20, generator=g)[:16].tolist()
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    hi, lo = freq.float(), (freq - freq.float().double()).float()
    k_pool, v_pool = (torch.full((20, nkv, PAGE, w), 7.0, dtype=dtype, device=DEV) for w in (2 * hd, vd))
    q_out, st = torch.zeros(n, q_width, dtype=dtype, device=DEV), status()
    ops.headnorm_rope_kvwrite(dev(rows), dev(qw), dev(kw) if own else None, eps, dev(hi) if rot else None,
                              dev(lo) if rot else None, rot, i32([0] * n), i32(pos),
                              q_out, k_pool, v_pool, i32([table]), PAGE, nh, nkv, 2, hd, vd, own, st)
    assert int(st.item()) == 0
    r, p = rows.double(), torch.tensor(pos)

    def made(x, w):
        x = plain.rms_norm(x, w.double(), eps)
        return plain.rotate_halves(x, p, rot, base) if rot else x
    tol = 1e-5 if dtype == torch.float32 else 0.04
    assert (q_out.double().cpu().view(n, nh, 2, hd) - made(r[:, :q_width].view(n, nh, 2, hd), qw)).abs().max() < tol
    if not own:
        assert bool((k_pool == 7).all()) and bool((v_pool == 7).all())
        return
    k = made(r[:, q_width:q_width + k_width].view(n, nkv, 2, hd), kw)
    v = r[:, q_width + k_width:q_width + k_width + nkv * vd].view(n, nkv, vd)
    kc, vc = k_pool.double().cpu(), v_pool.double().cpu()
    written = set()
    for i, q in enumerate(pos):
        page, at = table[q // PAGE], q % PAGE
        written.add((page, at))
        assert (kc[page, :, at].view(nkv, 2, hd) - k[i]).abs().max() < tol
        assert (vc[page, :, at] - v[i]).abs().max() < tol
    assert int((vc == 7).all(-1).all(1).sum()) == 20 * PAGE - len(written)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, V", [(3, 40), (1, 7), (16, 128), (5, 256)])
def test_difference_norm_and_gate(dtype, H, V):
    g = torch.Generator().manual_seed(H + V)
    a, gate = torch.randn(11, 2 * H, V, generator=g) * 3, torch.randn(11, H, generator=g) * 2
    a[3, 0] = a[3, 1] * 0.8 + 1e-3                      # nearly nothing is left of this head's difference
    for use in (True, False):
        y = torch.zeros(11, H, V, dtype=dtype, device=DEV)
        ops.diff_combine(dev(a), 0.8, 1e-6, 0.55, dev(gate) if use else None, y)
        ad = a.double().view(11, H, 2, V)
        want = plain.unit_rms(ad[:, :, 0] - 0.8 * ad[:, :, 1], 1e-6) * 0.55
        if use:
            want = want * plain.sigmoid(gate.double())[:, :, None]
        d = (y.double().cpu() - want).abs()
        d[3, 0] *= 1e-3                                  # the norm magnifies the inputs' own rounding there
        assert float(d.max()) < (1e-5 if dtype == torch.float32 else 0.02)


# ------------------------------------------------------------------------------------------------ norms on the results
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 100, 30, 2048])
@pytest.mark.parametrize("rows", [3, 300])
def test_norm_of_the_result_is_added_and_the_stream_is_read_as_it_is(dtype, width, rows):
    g = torch.Generator().manual_seed(width + rows)
    x, y, w = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g) * 5, torch.randn(width, generator=g)
    xd, h = dev(x), torch.zeros(rows, width, dtype=dtype, device=DEV)
    ops.norm_add_rmsnorm(xd, dev(y), dev(w), 1e-5, None, h, 0.0)
    want = x.double() + plain.rms_norm(y.double(), w.double(), 1e-5)
    assert (xd.double().cpu() - want).abs().max() < 2e-5
    assert torch.equal(h.float(), xd.to(dtype).float())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("has_shared, last", [(True, False), (False, False), (True, True)])
def test_combine_with_a_norm_of_its_result(dtype, has_shared, last):
    """The experts' rows of a token are summed (in ascending id), normalised and added to the stream; what follows is the
    stream itself or (``last``) the model's last norm on a few rows."""
    g = torch.Generator().manual_seed(5)
    n, k, width = 37, 3, 96
    ids = torch.stack([torch.randperm(9, generator=g)[:k] for _ in range(n)]).to(torch.int32)
    inverse = torch.randperm(n * k, generator=g).view(n, k).to(torch.int32)
    rows, shared = torch.randn(n * k, width, generator=g), torch.randn(n, width, generator=g)
    x, w, wf = torch.randn(n, width, generator=g), torch.randn(width, generator=g), torch.randn(width, generator=g)
    y = rows.double()[inverse.long()].sum(1) + (shared.double() if has_shared else 0)
    want = x.double() + plain.rms_norm(y, w.double(), 1e-5)
    xd = dev(x)
    sel = [36, 0, 5] if last else None
    h = torch.zeros(3 if last else n, width, dtype=dtype, device=DEV)
    ops.moe_combine_add_rmsnorm(dev(rows), dev(ids), dev(inverse), None, dev(shared) if has_shared else None, xd,
                                dev(wf) if last else None, h, 1e-6, rows=i32(sel) if last else None, write_x=not last,
                                gamma_y=dev(w), eps_y=1e-5)
    if last:
        assert torch.equal(xd.cpu(), x)
        ref = plain.rms_norm(want[sel], wf.double(), 1e-6)
        assert (h.double().cpu() - ref).abs().max() < (2e-5 if dtype == torch.float32 else 0.05)
    else:
        assert (xd.double().cpu() - want).abs().max() < 2e-5
        assert torch.equal(h.float(), xd.to(dtype).float())
    bare = dev(x)
    ops.moe_combine_add_rmsnorm(dev(rows), dev(ids), dev(inverse), None, dev(shared) if has_shared else None, bare, None, None, 0.0,
                                gamma_y=dev(w), eps_y=1e-5)
    assert (bare.double().cpu() - want).abs().max() < 2e-5


# ------------------------------------------------------------------------------------------------ routers
@pytest.mark.parametrize("n", [1, 5, 70, 300])
@pytest.mark.parametrize("weights", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E, top, width, spread", [(9, 3, 128, 1.0), (60, 4, 256, 120.0), (5, 5, 72, 3.0), (33, 1, 100, 300.0), (1, 1, 64, 1.0)])
def test_biased_router_weights_the_chosen_logits(n, weights, E, top, width, spread):
    """Logits that differ by hundreds: a softmax over all experts would leave zeros to choose among.  The bias decides
    choices: without it most tokens would choose otherwise."""
    g = torch.Generator().manual_seed(n * 7 + E)
    h = torch.randn(n, width, generator=g)
    wr = (torch.randn(E, width, generator=g) * (spread / math.sqrt(width))).to(weights)
    bias = torch.randn(E, generator=g) * spread * 1.5
    z = h.double() @ wr.double().T + bias.double()
    ids, wts, gap = torch.zeros(n, top, dtype=torch.int32, device=DEV), torch.zeros(n, top, device=DEV), torch.sort(z, -1, True).values
    st, logits = status(), torch.zeros(n, E + 1, device=DEV)
    if n <= ops.ROUTE_SMALL_TOKENS:
        offsets, perm = torch.zeros(E + 1, dtype=torch.int32, device=DEV), torch.zeros(n * top, dtype=torch.int32, device=DEV)
        pw, inv = torch.zeros(n * top, device=DEV), torch.zeros(n, top, dtype=torch.int32, device=DEV)
        ops.route_small(dev(h), dev(wr), None, logits, ids, wts, None, top, False, offsets, perm, pw, inv, st, bias=dev(bias),
                        chosen_softmax=True)
        assert torch.equal(pw[inv.long().view(-1)].view(n, top), wts)
        assert torch.equal(perm[inv.long().view(-1)].view(n, top), torch.arange(n, device=DEV, dtype=torch.int32)[:, None].expand(n, top))
        assert int(offsets[-1]) == n * top
    else:
        ops.router_topk(dev(h), dev(wr), None, ids, wts, None, top, False, st, logits=logits, bias=dev(bias), chosen_softmax=True)
    assert int(st.item()) == 0
    own = torch.topk(z, top, -1).indices
    clear = torch.ones(n, dtype=torch.bool) if E == top else (gap[:, top - 1] - gap[:, top]) > 1e-3 * max(1.0, spread)
    got = ids.cpu().long()
    assert torch.equal(torch.sort(got[clear], -1).values, torch.sort(own[clear], -1).values)
    want = plain.chosen_weights(z, got)
    assert (wts.double().cpu() - want).abs().max() < 2e-3 * (spread / 100 + 0.01)
    if spread == 1.0 and E > top and n > 5:
        bare = torch.topk(h.double() @ wr.double().T, top, -1).indices
        assert not torch.equal(torch.sort(bare, -1).values, torch.sort(own, -1).values)


# ------------------------------------------------------------------------------------------------ gated units
def unit(a, w, limit):
    g, u = (a.double() @ w.double().T).chunk(2, -1)
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * plain.sigmoid(1.702 * g) * (u + 1)


@pytest.mark.parametrize("form", ["few", "many"])
@pytest.mark.parametrize("rows, inter, width, limit", [(5, 72, 128, 0.9), (8, 256, 64, 2.0), (1, 2048, 512, 1.2)])
def test_clamped_unit_in_the_products_epilogue(form, rows, inter, width, limit):
    """Gates and up branches lie on both sides of the limits (a limit that is not applied, or applied to one side only,
    is off by more than the bound)."""
    g = torch.Generator().manual_seed(inter)
    rows = rows if form == "few" else rows * 50 + 3
    a, w = torch.randn(rows, width, generator=g).bfloat16(), (torch.randn(2 * inter, width, generator=g) * (2 / math.sqrt(width))).bfloat16()
    act = torch.zeros(rows, inter, dtype=torch.bfloat16, device=DEV)
    if form == "few":
        ops.gemm_skinny(dev(a), dev(w), act, swiglu=True, glu=(limit, 1.702, 1.0))
    else:
        st = status()
        ops.gemm_tc05(dev(a), dev(w), act, st, swiglu=True, glu=(limit, 1.702, 1.0))
        assert int(st.item()) == 0
    want = unit(a, w, limit)
    assert (act.double().cpu() - want).abs().max() < 0.02 * float(want.abs().max())
    assert (unit(a, w, 2 * limit) - want).abs().max() > 0.1 * float(want.abs().max())


@pytest.mark.parametrize("rows", [6, 400])
def test_clamped_unit_of_grouped_rows(rows):
    """The grouped forms: a permutation of (token, expert) rows through the weight-streaming kernel (few rows) and through
    the tensor-memory kernel's tile list (many)."""
    from esp_b200.parts.linear import grouped_swiglu_linear
    g = torch.Generator().manual_seed(rows)
    E, inter, width, top, limit = 5, 48, 64, 2, 1.1
    h = torch.randn(rows, width, generator=g).bfloat16()
    w = (torch.randn(E, 2 * inter, width, generator=g) * (2 / math.sqrt(width))).bfloat16()
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(rows)]).to(torch.int32)
    st, n = status(), rows * top
    offsets, perm = torch.zeros(E + 1, dtype=torch.int32, device=DEV), torch.zeros(n, dtype=torch.int32, device=DEV)
    pw, inv = torch.zeros(n, device=DEV), torch.zeros(rows, top, dtype=torch.int32, device=DEV)
    tiles = None
    if rows > 100:
        most = (n + ops.TC05_TILE_ROWS - 1) // ops.TC05_TILE_ROWS + E
        tiles = tuple(torch.zeros(s, dtype=torch.int32, device=DEV) for s in (most, most, most, 1))
    ops.moe_permute(dev(ids), torch.ones(rows, top, device=DEV), E, offsets, perm, pw, inv, st, tiles=tiles)

    class Rt:
        class ws:
            @staticmethod
            def get(name, shape, dtype):
                return torch.empty(shape, dtype=dtype, device=DEV)
        status = st
    act = torch.zeros(n, inter, dtype=torch.bfloat16, device=DEV)
    grouped_swiglu_linear(Rt, dev(h), dev(w), act, offsets, perm, n, rows, "t", tiles, glu=(limit, 1.702, 1.0))
    assert int(st.item()) == 0
    got = act.double().cpu()[inv.cpu().long()]
    want = torch.stack([torch.stack([unit(h[t:t + 1], w[e], limit)[0] for e in ids[t].tolist()]) for t in range(rows)])
    assert (got - want).abs().max() < 0.02 * float(want.abs().max())
