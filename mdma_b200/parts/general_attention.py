"""Grouped-query attention over the cache with options on every step of it (`general_attention`).

q = Wq h, k = Wk h, v = Wv h, no biases; `values` "keys": the values are the keys' projections themselves (v = k before the
norm and the rotation; there is no Wv and `v_dim` is `head_dim`).  `qk_norm`: every query and key head is divided by its
root mean square and multiplied by a weight of `head_dim` numbers that all heads share (tensors `q.norm`, `k.norm`),
before the rotation; `position`, a rotation by a frequency table, turns q and k; `v_norm`: every value head is divided by
its root mean square, without a weight, and cached so.

A query at position i sees the keys j <= i of its own sequence: all of them; with `window` n those with i - j < n, and with
`keep_first` m also those with j < m; with `chunk` n those of its own chunk, j // n == i // n, counted from the sequence's
start.  Kept tokens keep their true positions.  Scores (q . k) * scale; `softcap` c > 0: c tanh(score / c); then
`slope_power` p > 0: minus slope_h (i - j), slope_h = 2^(-p (h + 1) / heads).  Softmax in float; `sink`: exp of a learned
number per head (tensor `sink`) joins the denominator once.

`differential` d (absent: one map): every head has two maps, q and k laid out head by head as [map 1, map 2], each a
softmax of its own over the same values; with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + d (tensors of `head_dim` numbers)
o = a_1 - lambda a_2, divided by its root mean square over the head (no weight), times 1 - d.

`gate`: the concatenated heads are multiplied element by element by sigmoid(Wg h).  `out_scale`: a constant on the result.
Then Wo, added to the residual stream.

Kernels.  One product makes q, k, v and the gate; one kernel norms, turns and caches (adding up what a K-split product
left); attention runs on the tensor cores in the serving engine (tcgen05 for many rows, mma.sync for few, a tile kernel
for single tokens) where both head sizes are multiples of 16 up to 128, else, and always in the 32-bit engine, a warp per
(token, head) visits the keys in position order; one kernel merges runs of keys, takes the maps apart, norms and gates.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import KVNeed
from ..registry import MIXERS, POSITIONS
from ..spec import TensorSpec
from .base import Part
from .linear import Linear

LOG2E = 1.4426950408889634


@MIXERS.register("general_attention")
class GeneralAttention(Part):
    graph_safe = True          # forward reads no host-side per-step values
    takes_out_scale = True
    MAX_HEAD_DIM = 256         # the kernels' limit for keys and for values

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.n_heads, self.n_kv_heads = int(p["num_heads"]), int(p["num_kv_heads"])
        self.head_dim = int(p["head_dim"])
        self.v_dim = int(p.get("v_dim") or self.head_dim)
        self.scale, self.eps = float(p["scale"]), float(p.get("eps", 0.0))
        self.window, self.chunk = int(p.get("window", 0) or 0), int(p.get("chunk", 0) or 0)
        self.keep_first = int(p.get("keep_first", 0) or 0) if self.window else 0
        self.softcap, self.slope_power = float(p.get("softcap", 0.0) or 0.0), float(p.get("slope_power", 0.0) or 0.0)
        self.sink, self.gate = bool(p.get("sink", False)), bool(p.get("gate", False))
        self.qk_norm, self.v_norm = bool(p.get("qk_norm", False)), bool(p.get("v_norm", False))
        self.differential = p.get("differential")
        self.maps = 1 if self.differential is None else 2
        self.keys_as_values = p.get("values", "own") == "keys"
        self.out_scale = float(p.get("out_scale", 1.0))
        if p.get("values", "own") not in ("own", "keys"):
            raise ValueError(f"values {p['values']!r}: have 'own' and 'keys'")
        if self.n_heads % self.n_kv_heads:
            raise ValueError(f"{self.n_heads} heads do not divide over {self.n_kv_heads} kv heads")
        if self.window and self.chunk:
            raise ValueError("a window and chunks do not go together")
        if self.scale <= 0 or self.softcap < 0:
            raise ValueError("the scores' scale must be positive, the soft cap positive or absent")
        if self.keys_as_values and (self.v_dim != self.head_dim or self.maps > 1):
            raise ValueError("values that are the keys' projections have the keys' size, and go with one map per head")
        pos = p.get("position")
        self.position = POSITIONS.get(pos.kind)(pos) if pos is not None else None
        if self.position is not None and not hasattr(self.position, "rotary_table"):
            raise ValueError("this attention takes a rotation by a frequency table, or no position encoding")
        self.q_width, self.k_width = self.n_heads * self.maps * self.head_dim, self.n_kv_heads * self.maps * self.head_dim
        self.v_width, self.out_width = self.n_kv_heads * self.v_dim, self.n_heads * self.v_dim
        self.k_col = self.q_width
        self.v_col = self.k_col if self.keys_as_values else self.k_col + self.k_width
        self.g_col = self.v_col + (self.k_width if self.keys_as_values else self.v_width)
        self.row_width = self.g_col + (self.out_width if self.gate else 0)
        self.row_pitch = -(-self.row_width // 8) * 8       # the attention kernels read query rows 16 bytes at a time

    def children(self):
        return [self.position] if self.position is not None else []

    def check_limits(self, rt):
        if max(self.head_dim, self.v_dim) > self.MAX_HEAD_DIM:
            raise ValueError(f"head sizes {self.head_dim} / {self.v_dim} are beyond the attention kernels' limit of {self.MAX_HEAD_DIM}")

    def attention_shapes(self):
        return [(self.n_heads * self.maps, self.n_kv_heads * self.maps, max(self.head_dim, self.v_dim))]

    def _projections(self):
        return ["q", "k"] + ([] if self.keys_as_values else ["v"]) + (["g"] if self.gate else [])

    def tensor_specs(self):
        W = self.hidden
        rows = {"q": self.q_width, "k": self.k_width, "v": self.v_width, "g": self.out_width}
        specs = {n: TensorSpec((rows[n], W)) for n in self._projections()}
        if self.qk_norm:
            specs["q.norm"] = TensorSpec((self.head_dim,), "vector")
            specs["k.norm"] = TensorSpec((self.head_dim,), "vector")
        if self.sink:
            specs["sink"] = TensorSpec((self.n_heads,), "vector", "normal")
        if self.maps == 2:
            for n in ("lq1", "lk1", "lq2", "lk2"):
                specs[n] = TensorSpec((self.head_dim,), "vector", "normal")
        specs["o"] = TensorSpec((W, self.out_width))
        return specs

    def fused_tensors(self):
        return {"proj": tuple(self._projections())}          # one product for all projections of h

    def device_tensors(self):
        out = {}
        for name, used in (("slopes", self.slope_power > 0), ("sinks", self.sink)):
            if used:
                out[name] = ((self.n_heads,), torch.float32)
                out[name + "_log2"] = ((self.n_heads,), torch.float32)
        return out

    def kv_need(self):
        return KVNeed(self.n_kv_heads * self.maps, self.head_dim, self.window, v_dim=0 if self.v_dim == self.head_dim else self.v_dim,
                      keep_first=self.keep_first, chunk=self.chunk, n_v_heads=self.n_kv_heads if self.maps > 1 else 0)

    def state_need(self):
        return None

    def workspace(self):
        out = {f"gproj_{self.row_pitch}": (self.row_pitch, "act"), f"gattn_{self.out_width}": (self.out_width, "act")}
        if self.maps == 2:
            out[f"gmaps_{self.maps * self.out_width}"] = (self.maps * self.out_width, "f32")
        return out

    def slope_values(self) -> torch.Tensor:
        """slope_h = 2^(-slope_power (h + 1) / heads) in double."""
        h = torch.arange(1, self.n_heads + 1, dtype=torch.float64)
        return torch.pow(torch.tensor(2.0, dtype=torch.float64), -self.slope_power * h / self.n_heads)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        if self.position is not None:
            self.position.bind({}, rt)
        fused = tensors.get("proj")
        if fused is None:
            fused = torch.cat([tensors[n] for n in self._projections()], dim=0).contiguous()
        self.proj, self.o = Linear(fused, rt), Linear(tensors["o"], rt)
        self.q_weight, self.k_weight = tensors.get("q.norm"), tensors.get("k.norm")
        self.sink_values = tensors.get("sink")
        self.slopes = self.slopes_log2 = self.sinks = self.sinks_log2 = None
        if self.slope_power > 0:
            self.slopes = rt.derived(self.slope_values().to(torch.float32))
            self.slopes_log2 = rt.derived((self.slope_values() * LOG2E).to(torch.float32))      # the tensor-core kernels work in powers of two
        if self.sink:
            values = self.sink_values.detach().cpu().double()
            self.sinks, self.sinks_log2 = rt.derived(values.to(torch.float32)), rt.derived((values * LOG2E).to(torch.float32))
        self.lam, self.l_vectors = 0.0, []
        if self.maps == 2:
            self.l_vectors = [tensors[n] for n in ("lq1", "lk1", "lq2", "lk2")]
            lq1, lk1, lq2, lk2 = (t.detach().cpu().double() for t in self.l_vectors)
            self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + float(self.differential)
        self._fast_ok = False
        if rt.attention == "fast" and rt.dtype == torch.bfloat16:
            from .. import ops_tensor
            self._fast_ok = ops_tensor.attention_general_supported(self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim)

    def _prepare(self, ctx, h, row, view, write):
        """row = the projections of h; q and k normed and turned, keys and values in the cache."""
        n = ctx.n_tokens
        self.proj.store(h, row, n, defer=True)
        partial, splits, stride = None, 0, 0
        if self.rt.gemm == "tensor":
            from .. import ops_tensor
            pend = ops_tensor.take_pending(row, ops.GEMM_STORE, n, self.rt.tc, any_pitch=True)
            if pend is not None:
                partial, splits, stride = pend
            else:
                ops_tensor.flush_pending(row.device, self.rt.tc)
        inv_freq, rotary_dim, interleaved = self.position.rotary_table() if self.position is not None else (None, 0, False)
        # query heads that are neither normed nor turned stay as the product left them
        q_heads = self.n_heads * self.maps if (self.qk_norm or rotary_dim or partial is not None) else 0
        ops.qk_norm_rotate(row, self.k_col, self.v_col, ctx.tok_seq, ctx.tok_pos, ctx.seq_slot, inv_freq,
                           float(getattr(self.position, "magnitude", 1.0)), self.q_weight, self.k_weight, self.qk_norm, self.eps,
                           view.k, view.v, view.page_table, view.max_pages, view.page_size, n, q_heads, self.n_kv_heads * self.maps,
                           self.head_dim, self.v_dim, rotary_dim, interleaved, write, n_v_heads=self.n_kv_heads, v_norm=self.v_norm,
                           partial=partial, splits=splits, split_stride=stride, row_width=self.row_width, tail_col=self.g_col)

    def _run(self, ctx, h, view, owns_cache):
        n = ctx.n_tokens
        whole = ctx.buf(f"gproj_{self.row_pitch}", self.row_pitch)
        row = whole[:, :self.row_width]
        out = ctx.buf(f"gattn_{self.out_width}", self.out_width)
        self._prepare(ctx, h, row, view, owns_cache)
        gate = row[:, self.g_col:] if self.gate else None
        maps = ctx.buf(f"gmaps_{self.maps * self.out_width}", self.maps * self.out_width, torch.float32) if self.maps == 2 else None
        finish = dict(gate=gate, out_scale=self.out_scale)
        if self.maps == 2:
            d = float(self.differential)
            finish.update(maps=2, lam=self.lam, norm_scale=1.0 - d, eps=self.eps)
        if self._fast_ok:
            from .. import ops_tensor
            partial = ops_tensor.attention_general(
                ctx, whole, view, self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim, self.scale,
                out=out if self.maps == 1 else None, out_f32=maps, maps=self.maps, window=self.window, keep_first=self.keep_first,
                chunk=self.chunk, softcap=self.softcap, sink_log2=self.sinks_log2, slope_log2=self.slopes_log2, st=self.rt.tc)
            if partial is not None:
                ops.attention_finish(out, n, self.n_heads, self.v_dim, partial=partial, sink_log2=self.sinks_log2, **finish)
            elif self.maps == 2 or gate is not None or self.out_scale != 1.0:
                ops.attention_finish(out, n, self.n_heads, self.v_dim, rows=maps if self.maps == 2 else out, **finish)
            return out
        plain = dict(sinks=self.sinks, keep_first=self.keep_first, chunk=self.chunk, softcap=self.softcap)
        args = (whole, view.k, view.v, ctx, view.page_table, view.max_pages, view.page_size, self.slopes)
        sizes = (self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim, self.window, self.scale)
        if self.maps == 1:
            ops.attention_distance(*args, gate, out, *sizes, out_scale=self.out_scale, **plain)
        else:
            ops.attention_distance(*args, None, maps, *sizes, maps=2, **plain)
            ops.attention_finish(out, n, self.n_heads, self.v_dim, rows=maps, **finish)
        return out

    def forward(self, ctx, h, x, view, owns_cache=True):
        self.o.accumulate(self._run(ctx, h, view, owns_cache), x, ctx.n_tokens)

    def produce(self, ctx, h, out, view, owns_cache=True, defer=False):
        """The result as float rows; `defer`: the last product may leave K-split partial sums of `out`."""
        self.o.store(self._run(ctx, h, view, owns_cache), out, ctx.n_tokens, defer=defer)

    def resident_tensors(self):
        return [t for t in (self.proj.w, self.o.w, self.q_weight, self.k_weight, self.sink_values, *self.l_vectors) if t is not None]
