"""A matrix memory with exponential gates (`matrix_memory`, the mLSTM of the xLSTM paper).

q = Wq h * dim^(-1/2), k = Wk h [heads x dim], v = Wv h [heads x v_dim]; per head the logarithms of an input and a forget gate,
i = cap tanh((Wi h + bi) / cap), f = log sigmoid(cap tanh((Wf h + bf) / cap)), and with a running maximum m from 0

    m_t = max(f + m_(t-1), i),    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,    n_t likewise with k alone,
    o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6).

S, n and m start at zero, are float, and live in the site's state row per sequence.  Every head's o is divided by its root
mean square; the heads side by side are multiplied by the weight `norm` (of all heads' size), by sigmoid(Wg h), by the
constant `out_scale`, and projected by Wo.  The projections are one product in the compute dtype with float rows; everything
behind them up to the gated heads is float in both engines.

The 32-bit engine and short portions walk row by row in one fixed order; single tokens of the serving engine go from the
projection (its K-split partial sums included) to the gated heads in one kernel; portions of `CHUNKS_FROM` rows or more go
a chunk at a time, long ones in runs of `RUN_ROWS` rows side by side if the scratch holds the runs' states.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateNeed
from ..registry import MIXERS
from ..spec import TensorSpec
from .base import Part
from .linear import Linear


@MIXERS.register("matrix_memory")
class MatrixMemory(Part):
    graph_safe = True
    takes_out_scale = True
    CHUNKS_FROM = 16          # rows of a sequence in a step from which the serving engine walks chunk by chunk
    RUN_ROWS = 128            # rows of a run; sequences of two runs and more are walked as runs side by side
    MAX_RUNS, MAX_DIM = 256, 256          # the kernels' limits

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.dim = int(p["num_heads"]), int(p["head_dim"])
        self.v_dim = int(p.get("v_dim") or self.dim)
        self.cap, self.eps = float(p["gate_cap"]), float(p["eps"])
        self.out_scale = float(p.get("out_scale", 1.0))
        if self.cap <= 0:
            raise ValueError(f"the gates' cap must be positive, got {self.cap}")
        self.qk_width, self.v_width = self.heads * self.dim, self.heads * self.v_dim
        self.k_col, self.v_col = self.qk_width, 2 * self.qk_width
        self.g_col = self.v_col + self.v_width
        self.i_col = self.g_col + self.v_width
        self.f_col = self.i_col + self.heads
        self.row_width = self.f_col + self.heads
        self.row_pitch = -(-self.row_width // 4) * 4
        self.floats = ops.matrix_memory_state_floats(self.heads, self.dim, self.v_dim)
        self.cols = (0, self.k_col, self.v_col, self.i_col, self.f_col)

    def check_limits(self, rt):
        if max(self.dim, self.v_dim) > self.MAX_DIM:
            raise ValueError(f"matrix memory heads of {self.dim} x {self.v_dim} are beyond the kernels' limit of {self.MAX_DIM}")

    def tensor_specs(self):
        W = self.hidden
        return {"q": TensorSpec((self.qk_width, W)), "k": TensorSpec((self.qk_width, W)), "v": TensorSpec((self.v_width, W)),
                "g": TensorSpec((self.v_width, W)), "i": TensorSpec((self.heads, W)), "f": TensorSpec((self.heads, W)),
                "i.b": TensorSpec((self.heads,), "vector", "normal"), "f.b": TensorSpec((self.heads,), "vector", "normal"),
                "norm": TensorSpec((self.v_width,), "vector"), "o": TensorSpec((W, self.v_width))}

    def fused_tensors(self):
        return {"proj": ("q", "k", "v", "g", "i", "f")}

    def kv_need(self):
        return None

    def state_need(self):
        return StateNeed((self.floats,), torch.float32)

    def _names(self):
        tag = f"{self.heads}_{self.dim}_{self.v_dim}"
        return {n: f"mem_{n}_{tag}" for n in ("proj", "sum", "out", "runs")}

    def workspace(self):
        n = self._names()
        return {n["proj"]: (self.row_pitch, "f32"), n["sum"]: (self.v_width, "f32"), n["out"]: (self.v_width, "act"),
                n["runs"]: (self._run_columns(), "f32")}

    def _run_columns(self) -> int:
        # scratch for the runs side by side: room for two runs' states per RUN_ROWS rows of a step
        return -(-2 * self.floats // self.RUN_ROWS)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        fused = tensors.get("proj")
        if fused is None:
            fused = torch.cat([tensors[n] for n in ("q", "k", "v", "g", "i", "f")], dim=0).contiguous()
        self.proj, self.o = Linear(fused, rt), Linear(tensors["o"], rt)
        self.norm, self.i_bias, self.f_bias = tensors["norm"], tensors["i.b"], tensors["f.b"]
        self._token_ok = rt.dtype == torch.bfloat16 and ops.matrix_memory_token_fits(self.dim, self.v_dim)

    def _run(self, ctx, h, view):
        n, names, f32 = ctx.n_tokens, self._names(), torch.float32
        proj = ctx.buf(names["proj"], self.row_pitch, f32)[:, :self.row_width]
        out = ctx.buf(names["out"], self.v_width)
        q_scale = self.dim ** -0.5
        single = ctx.max_new == 1 and self._token_ok
        self.proj.store(h, proj, n, defer=single)
        partial, splits, stride = None, 0, 0
        if self.rt.gemm == "tensor":
            from .. import ops_tensor
            pend = ops_tensor.take_pending(proj, ops.GEMM_STORE, n, self.rt.tc, any_pitch=True) if single else None
            if pend is not None:
                partial, splits, stride = pend
            else:
                ops_tensor.flush_pending(proj.device, self.rt.tc)
        if single:
            ops.matrix_memory_token(proj, self.cols, self.g_col, self.i_bias, self.f_bias, self.cap, q_scale, self.norm, ctx, view.state,
                                    out, self.heads, self.dim, self.v_dim, self.eps, self.out_scale, partial, splits, stride)
            return out
        sums = ctx.buf(names["sum"], self.v_width, f32)
        chunked = self.rt.dtype != f32 and ctx.max_new >= self.CHUNKS_FROM
        run_rows, max_runs, scratch = 0, 1, None
        if chunked and ctx.max_new >= 2 * self.RUN_ROWS:
            # (room for them all, unless one long prompt comes with many short ones)
            runs = ctx.buf(names["runs"], self._run_columns(), f32).view(-1)
            most = -(-ctx.max_new // self.RUN_ROWS)
            if most <= self.MAX_RUNS and ctx.n_seqs * most * self.floats <= runs.numel():
                run_rows, max_runs, scratch = self.RUN_ROWS, most, runs
        ops.matrix_memory(proj, self.cols, self.i_bias, self.f_bias, self.cap, q_scale, ctx, view.state, sums, self.heads, self.dim,
                          self.v_dim, chunked, run_rows, max_runs, scratch)
        ops.gated_head_rmsnorm(sums, proj[:, self.g_col:], self.norm, out, n, self.heads, self.v_dim, self.eps, scale=self.out_scale)
        return out

    def forward(self, ctx, h, x, view, owns_cache=True):
        self.o.accumulate(self._run(ctx, h, view), x, ctx.n_tokens)

    def produce(self, ctx, h, out, view, owns_cache=True, defer=False):
        """The result as float rows; `defer`: the last product may leave K-split partial sums of `out`."""
        self.o.store(self._run(ctx, h, view), out, ctx.n_tokens, defer=defer)

    def resident_tensors(self):
        return [self.proj.w, self.o.w, self.norm, self.i_bias, self.f_bias]
