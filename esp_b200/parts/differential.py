"""Attention with two maps per head whose outputs are subtracted (see ``DifferentialAttentionSpec``)."""
from __future__ import annotations

import torch

from ..cache import KvLayout
from ..cache.book import PAGE
from ..csrc import ops
from ..errors import Unsupported
from .attention import DECODE_ROWS, scaled_tiles
from .base import ParamSpec, Part, build, register
from .linear import linear

ROW_ALIGN = 16         # the packed projection's rows are a multiple of this; the last ones are zeros that nothing reads


class DifferentialAttention(Part):
    """One packed product gives queries, keys, values and the heads' gates of a token (a layer that reads another's
    cache: queries and gates); one kernel norms and rotates every map of every head and stores keys and values in the
    cache, whose key rows hold both maps of a head side by side; the attention kernels for bfloat16 carry both maps
    over the same pages, and end with the difference, its norm and the gate; the plain kernel (32-bit, and sizes that
    the others do not take) leaves both maps' outputs in 32-bit to a kernel of its own for that.  Query head i reads
    key/value head i // (num_heads / num_kv_heads)."""

    graph_safe = True

    def __init__(self, spec, rt):
        self.spec, self.rt = spec, rt
        s = spec
        if s.key_dim > 256 or s.value_dim > 256:
            raise Unsupported("dim", f"{s.key_dim} / {s.value_dim}; the attention kernels take head sizes up to 256")
        if s.num_heads % s.num_kv_heads != 0:
            raise Unsupported("kv_heads", f"{s.num_kv_heads} does not divide {s.num_heads} heads")
        if not s.scale > 0:
            raise Unsupported("scale", f"{s.scale}; the attention kernels take a positive scale")
        self.q_width = s.num_heads * 2 * s.key_dim
        self.k_width = s.num_kv_heads * 2 * s.key_dim if s.own_kv else 0
        self.v_width = s.num_kv_heads * s.value_dim if s.own_kv else 0
        self.o_width = s.num_heads * s.value_dim
        self.gate_at = self.q_width + self.k_width + self.v_width
        used = self.gate_at + (s.num_heads if s.head_gate else 0)
        self.row_width = (used + ROW_ALIGN - 1) // ROW_ALIGN * ROW_ALIGN
        self.position = None
        if s.position is not None:
            if getattr(s.position, "factor", None) is not None:
                raise Unsupported("rot", "interpolated frequencies on an attention layer with two maps")
            key = ("position", s.position)            # layers with the same encoding share one part (and its frequencies)
            if key not in rt.shared_parts:
                rt.shared_parts[key] = build("position", s.position, rt)
            self.position = rt.shared_parts[key]
        self.w_in = self.w_o = self.q_norm = self.k_norm = self.lambda_parts = None
        self.lam = None                               # the second map's weight: a number, known once the weights are in

    def children(self):
        return [self.position] if self.position is not None else []

    # -- parameters ----------------------------------------------------------
    def _n(self, which):
        return self.spec.prefix + getattr(self.spec.names, which)

    def _lambda_names(self):
        return [self.spec.prefix + n for n in self.spec.names.lambda_parts]

    def param_specs(self):
        s = self.spec
        specs = [ParamSpec(self._n("q"), (self.q_width, s.hidden), "matrix"),
                 ParamSpec(self._n("o"), (s.hidden, self.o_width), "matrix"),
                 ParamSpec(self._n("q_norm"), (s.key_dim,), "norm_scale")]
        if s.own_kv:
            specs += [ParamSpec(self._n("k"), (self.k_width, s.hidden), "matrix"),
                      ParamSpec(self._n("v"), (self.v_width, s.hidden), "matrix"),
                      ParamSpec(self._n("k_norm"), (s.key_dim,), "norm_scale")]
        if s.head_gate:
            specs.append(ParamSpec(self._n("head_gate"), (s.num_heads, s.hidden), "matrix"))
        specs += [ParamSpec(n, (s.key_dim,), "map_weight", init=(0.0, 0.1)) for n in self._lambda_names()]
        return specs

    def allocate(self, stored, rt):
        s, dev = self.spec, rt.device
        places = {self._n("q"): (0, self.q_width)}
        if s.own_kv:
            places[self._n("k")] = (self.q_width, self.q_width + self.k_width)
            places[self._n("v")] = (self.q_width + self.k_width, self.gate_at)
        if s.head_gate:
            places[self._n("head_gate")] = (self.gate_at, self.gate_at + s.num_heads)
        self.w_in = torch.zeros((self.row_width, s.hidden), dtype=rt.matrix_dtype([stored[n] for n in places]), device=dev)
        self.w_o = torch.empty((s.hidden, self.o_width), dtype=rt.matrix_dtype([stored[self._n("o")]]), device=dev)
        f32 = lambda: torch.empty(s.key_dim, dtype=torch.float32, device=dev)
        self.q_norm = f32()
        views = {n: self.w_in[a:b] for n, (a, b) in places.items()}
        views.update({self._n("o"): self.w_o, self._n("q_norm"): self.q_norm})
        if s.own_kv:
            self.k_norm = f32()
            views[self._n("k_norm")] = self.k_norm
        self.lambda_parts = torch.empty((4, s.key_dim), dtype=torch.float32, device=dev)
        views.update({n: self.lambda_parts[i] for i, n in enumerate(self._lambda_names())})
        return views

    def finalize(self):
        if self.lambda_parts is not None and self.lam is None:
            a = self.lambda_parts.double()
            dots = (a[0::2] * a[1::2]).sum(-1)
            self.lam = float(torch.exp(dots[0]) - torch.exp(dots[1])) + self.spec.diff

    # -- what it keeps per sequence ------------------------------------------------
    def kv_layout(self):
        s = self.spec
        vd = s.value_dim if s.value_dim != 2 * s.key_dim else None
        return KvLayout(s.num_kv_heads, 2 * s.key_dim, s.keep_window, value_dim=vd, chunk=s.keep_chunk)

    def state_spec(self):
        return None

    # -- which kernel a step of n token rows gets, and the index lists it needs ----------
    def kernel_for(self, n: int, page: int = PAGE) -> str:
        s = self.spec
        if self.rt.dtype == torch.bfloat16:
            if (n <= DECODE_ROWS and ops.attn_decode_diff_fits(s.key_dim, s.value_dim, page)
                    and n * 2 * s.num_heads <= ops.ATTN_DECODE_COUNTERS):
                return "split"         # few rows: the keys are split over blocks
            if ops.attn_diff_tc05_fits(s.key_dim, s.value_dim, page):
                return "tc05"          # many rows: both maps' scores and weighted values in tensor memory
        return "plain"

    def step_arrays_key(self):
        s = self.spec
        return ("attention_differential", self.rt.dtype, s.key_dim, s.value_dim)

    def step_arrays(self, step):
        return scaled_tiles(self.kernel_for(step.n_tokens), step)

    # -- running ---------------------------------------------------------------
    def forward(self, h, ctx, layer):
        s, rt = self.spec, self.rt
        n = h.shape[0]
        table = ctx.block_tables[layer.group]
        rows = rt.ws.get(f"diff_rows_{self.row_width}", (n, self.row_width), torch.float32)
        linear(rt, h, self.w_in, rows)
        q = rt.ws.get("attn_q", (n, self.q_width), rt.dtype)
        pos = self.position
        freq = (pos.inv_freq, pos.inv_freq_lo, pos.spec.rotary_dim) if pos is not None else (None, None, 0)
        ops.headnorm_rope_kvwrite(rows, self.q_norm, self.k_norm, s.eps, *freq, ctx.tok_seq, ctx.tok_pos, q, layer.k, layer.v,
                                  table, layer.page, s.num_heads, s.num_kv_heads, 2, s.key_dim, s.value_dim, s.own_kv, rt.status)
        o = rt.ws.get("attn_o", (n, self.o_width), rt.dtype)
        gate = rows[:, self.gate_at:self.gate_at + s.num_heads] if s.head_gate else None
        self.attend(q, gate, o, ctx, layer)
        y = rt.ws.get("mixer_out", (n, s.hidden), torch.float32)
        linear(rt, o, self.w_o, y)
        return y

    def attend(self, q, gate, o, ctx, layer):
        s, rt = self.spec, self.rt
        n = q.shape[0]
        table = ctx.block_tables[layer.group]
        kind = self.kernel_for(n, layer.page)
        out_scale = 1.0 - s.diff
        if kind == "split":
            positions = table.shape[1] * layer.page
            group = 2 * s.num_heads // s.num_kv_heads
            kv_blocks = s.num_kv_heads * ((group + 15) // 16)
            span = min(positions, s.chunk + layer.page) if s.chunk else positions
            vd = ops.attn_diff_tile(s.value_dim)
            split = ops.attn_decode_split(n, kv_blocks, span, max(ops.attn_diff_tile(2 * s.key_dim), vd), rt.sm_count)
            n_splits = (positions + split - 1) // split
            part_o = rt.ws.get("attn_part_o", (n, 2 * s.num_heads, n_splits, vd), torch.float32)
            part_ml = rt.ws.get("attn_part_ml", (n, 2 * s.num_heads, n_splits, 2), torch.float32)
            if getattr(rt, "attn_counters", None) is None:
                rt.attn_counters = torch.zeros(ops.ATTN_DECODE_COUNTERS, dtype=torch.int32, device=rt.device)
            ops.attn_decode_diff(q, layer.k, layer.v, o, part_o, part_ml, rt.attn_counters, ctx.tok_seq, ctx.tok_pos, table,
                                 layer.page, s.num_heads, s.num_kv_heads, s.key_dim, s.value_dim, s.scale, split, n_splits,
                                 rt.status, self.lam, s.eps, out_scale, gate=gate, softcap=s.softcap, chunk=s.chunk,
                                 seq_past=ctx.seq_past if layer.writes else None)
            return
        tile_seq = None
        if kind == "tc05":
            rows = ops.ATTN_TC05_TILE_ROWS
            tile_seq, tile_first = ctx.arrays.get(f"attention.tiles{rows}.seq"), ctx.arrays.get(f"attention.tiles{rows}.first")
        fused = tile_seq is not None and s.value_dim <= ops.ATTN_DIFF_FUSED_VALUES
        maps = None if fused else rt.ws.get("diff_maps", (n, 2 * s.num_heads, s.value_dim), torch.float32)
        if tile_seq is not None:
            ops.attn_diff_tc05(q, layer.k, layer.v, o if fused else None, maps, tile_seq, tile_first, ctx.seq_start, ctx.seq_past,
                               table, layer.page, s.num_heads, s.num_kv_heads, s.key_dim, s.value_dim, s.scale, rt.status,
                               self.lam, s.eps, out_scale, gate=gate, softcap=s.softcap, chunk=s.chunk)
            if fused:
                return
        else:                              # (a step made without this part's lists takes the plain kernel as well)
            ops.attn_simt(q, layer.k, layer.v, maps, ctx.tok_seq, ctx.tok_pos, table, layer.page, 2 * s.num_heads,
                          s.num_kv_heads, s.key_dim, None, rt.status, vd=s.value_dim, scale=s.scale, chunk=s.chunk,
                          softcap=s.softcap, maps=2)
        ops.diff_combine(maps, self.lam, s.eps, out_scale, gate, o.view(n, s.num_heads, s.value_dim))


register("mixer", "attention_differential", DifferentialAttention)
