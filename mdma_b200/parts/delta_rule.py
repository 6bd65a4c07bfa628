"""The gated delta rule with a decay per key channel (`channel_delta`).

Projections of a row h: q, k = Wq h, Wk h (kv_heads heads of dim numbers, every one serving heads / kv_heads neighbouring
heads), v = Wv h (heads of v_dim).  y_t[c] = SiLU(sum_j C[c, taps-1-j] x_(t-j)[c]) replaces every channel c of the three,
C the stacked `q.conv`, `k.conv`, `v.conv` and x_t = 0 for t < 0.  Then, head by head,

    q' = dim^-1/2 q / |q|,   k' = k / |k|   with |x|^2 = unit_eps + sum x^2,
    b = sigmoid(Wb h),   log g = -e^A_log softplus(A2 A1 h + dt_bias)      (a number a head; a number a head and channel),
    S <- diag(g) S,   u = b (v - S^T k'),   S <- S + k' u^T,   o = S^T q'          S [dim, v_dim],
    result = Wo [rms_unit(o) * norm * sigmoid(G2 G1 h)]      (`norm` has v_dim numbers for all heads).

State per sequence: S (floats) and the convolutions' last taps-1 inputs.  Everything that enters the recurrence is float
in both engines (the projections write float rows); A1 h and G1 h go into their second products in the compute dtype.
The 32-bit engine and short portions walk row by row in one fixed order; the serving engine walks portions of
`CHUNKS_FROM` rows or more a chunk of rows at a time (csrc/delta_chunk.cu), and its single tokens take one kernel from
the projection to the gated norm where its sizes fit (one q/k head per head).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateNeed
from ..registry import MIXERS
from ..spec import TensorSpec
from .base import Part
from .linear import Linear


@MIXERS.register("channel_delta")
class ChannelDelta(Part):
    graph_safe = True
    MAX_DIM, MAX_TAPS = 256, 16          # the kernels' limits
    CHUNKS_FROM = 16                     # rows of a sequence in a step from which the serving engine walks chunk by chunk

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.kv_heads = int(p["num_heads"]), int(p.get("num_kv_heads") or p["num_heads"])
        self.dim = int(p["head_dim"])
        self.v_dim = int(p.get("v_dim") or self.dim)
        self.taps = int(p["conv"])
        self.decay_rank, self.gate_rank = int(p["decay_rank"]), int(p["gate_rank"])
        self.eps, self.unit_eps = float(p["eps"]), float(p.get("unit_eps", 1e-6))
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads do not divide over {self.kv_heads} kv heads")
        self.qk_width, self.k_width, self.v_width = self.kv_heads * self.dim, self.heads * self.dim, self.heads * self.v_dim
        self.channels = 2 * self.qk_width + self.v_width            # what the convolutions see
        # a projection row: q, k, v, the step sizes' logits, the inner rows of the decays and of the gate
        self.inner_col = self.channels + self.heads
        self.row_width = self.inner_col + self.decay_rank + self.gate_rank
        self.row_pitch = -(-self.row_width // 8) * 8
        self.state_floats = self.heads * self.dim * self.v_dim
        self.conv_at = -(-self.state_floats // 4) * 4
        self.chunks_fit = self.dim % 4 == 0 and self.v_dim % 4 == 0 and self.v_dim <= 512
        self.conv_floats = (self.taps - 1) * self.channels

    def check_limits(self, rt):
        if self.dim > self.MAX_DIM:
            raise ValueError(f"delta-rule heads of {self.dim} are beyond the kernels' limit of {self.MAX_DIM}")
        if not 1 <= self.taps <= self.MAX_TAPS:
            raise ValueError(f"a convolution of {self.taps} taps is outside the kernel's 1..{self.MAX_TAPS}")

    def tensor_specs(self):
        W = self.hidden
        return {"q": TensorSpec((self.qk_width, W)), "q.conv": TensorSpec((self.qk_width, self.taps)),
                "k": TensorSpec((self.qk_width, W)), "k.conv": TensorSpec((self.qk_width, self.taps)),
                "v": TensorSpec((self.v_width, W)), "v.conv": TensorSpec((self.v_width, self.taps)),
                "b": TensorSpec((self.heads, W)), "A_log": TensorSpec((self.heads,), "vector", "normal"),
                "norm": TensorSpec((self.v_dim,), "vector"),
                "a1": TensorSpec((self.decay_rank, W)), "a2": TensorSpec((self.k_width, self.decay_rank)),
                "dt_bias": TensorSpec((self.k_width,), "vector", "normal"),
                "g1": TensorSpec((self.gate_rank, W)), "g2": TensorSpec((self.v_width, self.gate_rank)),
                "o": TensorSpec((W, self.v_width))}

    def fused_tensors(self):
        return {"qkvbag": ("q", "k", "v", "b", "a1", "g1"), "conv": ("q.conv", "k.conv", "v.conv")}

    def kv_need(self):
        return None

    def state_need(self):
        return StateNeed((self.conv_at + self.conv_floats,), torch.float32)

    def _names(self):
        tag = f"{self.heads}_{self.kv_heads}_{self.dim}_{self.v_dim}"
        return {n: f"delta_{n}_{tag}" for n in ("proj", "q", "k", "v", "lg", "beta", "raw", "gate", "sum", "out", "chunks")}

    def workspace(self):
        n = self._names()
        ws = {n["proj"]: (self.row_pitch, "f32"), n["q"]: (self.qk_width, "f32"), n["k"]: (self.qk_width, "f32"),
              n["v"]: (self.v_width, "f32"), n["lg"]: (self.k_width, "f32"), n["beta"]: (self.heads, "f32"),
              n["raw"]: (self.k_width, "f32"), n["gate"]: (self.v_width, "act"), n["sum"]: (self.v_width, "f32"),
              n["out"]: (self.v_width, "act")}
        if self.chunks_fit:
            ws[n["chunks"]] = (self._chunk_columns(), "f32")
        ws[f"delta_a1_{self.decay_rank}"] = (-(-self.decay_rank // 8) * 8, "act")
        ws[f"delta_g1_{self.gate_rank}"] = (-(-self.gate_rank // 8) * 8, "act")
        return ws

    def _chunk_columns(self) -> int:
        # scratch of the chunks side by side: a row's share, and an eighth more for sequences' last, partial chunks
        return -(-9 * ops.delta_chunk_floats(self.heads, self.dim, self.v_dim) // 128)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)

        def whole(name, pieces):
            t = tensors.get(name)
            return t if t is not None else torch.cat([tensors[n] for n in pieces], dim=0).contiguous()
        self.proj = Linear(whole("qkvbag", ("q", "k", "v", "b", "a1", "g1")), rt)
        self.conv = whole("conv", ("q.conv", "k.conv", "v.conv"))
        self.a2, self.g2, self.o = Linear(tensors["a2"], rt), Linear(tensors["g2"], rt), Linear(tensors["o"], rt)
        self.a_log, self.dt_bias, self.norm = tensors["A_log"], tensors["dt_bias"], tensors["norm"]
        self._token_ok = (rt.dtype != torch.float32 and self.conv.dtype == torch.bfloat16
                          and self.a_log.dtype == self.dt_bias.dtype == self.norm.dtype
                          and ops.delta_token_fits(self.heads, self.kv_heads, self.dim, self.v_dim, self.decay_rank, self.gate_rank, self.taps))

    def _low_rank(self, ctx, proj, raw, gate):
        """raw = a2 a1 h (float rows), gate = g2 g1 h."""
        n, c = ctx.n_tokens, self.inner_col
        if proj.dtype == gate.dtype:
            a, g = proj[:, c:c + self.decay_rank], proj[:, c + self.decay_rank:self.row_width]
        else:
            a = ctx.buf(f"delta_a1_{self.decay_rank}", -(-self.decay_rank // 8) * 8)[:, :self.decay_rank]
            g = ctx.buf(f"delta_g1_{self.gate_rank}", -(-self.gate_rank // 8) * 8)[:, :self.gate_rank]
            ops.delta_inner(proj, c, self.decay_rank, self.gate_rank, a, g, n)
        self.a2.store(a, raw, n)
        self.g2.store(g, gate, n)

    def _run(self, ctx, h, view):
        n = ctx.n_tokens
        names = self._names()
        f32 = torch.float32
        proj = ctx.buf(names["proj"], self.row_pitch, f32)[:, :self.row_width]
        out = ctx.buf(names["out"], self.v_width)
        state = view.state[:, :self.state_floats]
        conv_state = view.state[:, self.conv_at:self.conv_at + self.conv_floats] if self.taps > 1 else None
        q_scale = self.dim ** -0.5
        single = ctx.max_new == 1 and self._token_ok
        self.proj.store(h, proj, n, defer=single)
        if single:
            partial, splits, stride = None, 0, 0
            if self.rt.gemm == "tensor":
                from .. import ops_tensor
                pend = ops_tensor.take_pending(proj, ops.GEMM_STORE, n, self.rt.tc, any_pitch=True)
                if pend is not None:
                    partial, splits, stride = pend
                else:
                    ops_tensor.flush_pending(proj.device, self.rt.tc)
            ops.delta_token(proj, self.a2.w, self.g2.w, self.conv, self.taps, self.a_log, self.dt_bias, self.norm, ctx, view.state,
                            self.conv_at, out, self.heads, self.dim, self.v_dim, self.unit_eps, q_scale, self.eps, partial, splits,
                            stride)
            return out
        raw, gate = ctx.buf(names["raw"], self.k_width, f32), ctx.buf(names["gate"], self.v_width)
        sums = ctx.buf(names["sum"], self.v_width, f32)
        self._low_rank(ctx, proj, raw, gate)
        if self.rt.gemm == "tensor":
            from .. import ops_tensor
            ops_tensor.flush_pending(proj.device, self.rt.tc)
        chunks = None
        if self.chunks_fit and self.rt.dtype != f32 and ctx.max_new >= self.CHUNKS_FROM:
            # (room for them all, unless very many short sequences come with a long one)
            chunks = ctx.buf(names["chunks"], self._chunk_columns(), f32).view(-1)
            if (n // 16 + ctx.n_seqs + 1) * ops.delta_chunk_floats(self.heads, self.dim, self.v_dim) > chunks.numel():
                chunks = None
        if chunks is not None:
            ops.delta_chunks(proj, raw, self.conv, self.taps, self.a_log, self.dt_bias, conv_state, chunks, ctx, state, sums,
                             self.heads, self.kv_heads, self.dim, self.v_dim, self.unit_eps, q_scale)
        else:
            q, k = ctx.buf(names["q"], self.qk_width, f32), ctx.buf(names["k"], self.qk_width, f32)
            v, lg = ctx.buf(names["v"], self.v_width, f32), ctx.buf(names["lg"], self.k_width, f32)
            beta = ctx.buf(names["beta"], self.heads, f32)
            ops.delta_prepare(proj, raw, self.conv, self.taps, self.a_log, self.dt_bias, ctx, conv_state, q, k, v, lg, beta,
                              self.heads, self.kv_heads, self.dim, self.v_dim, self.unit_eps, q_scale)
            ops.delta_scan(q, k, v, lg, beta, ctx, state, sums, self.heads, self.kv_heads, self.dim, self.v_dim)
        ops.delta_conv_keep(proj, self.taps, self.channels, ctx, conv_state)
        ops.gated_head_rmsnorm(sums, gate, self.norm, out, n, self.heads, self.v_dim, self.eps)
        return out

    def forward(self, ctx, h, x, view, owns_cache=True):
        self.o.accumulate(self._run(ctx, h, view), x, ctx.n_tokens, defer=False)

    def produce(self, ctx, h, out, view, owns_cache=True, defer=False):
        self.o.store(self._run(ctx, h, view), out, ctx.n_tokens, defer=defer)

    def resident_tensors(self):
        return [self.proj.w, self.conv, self.a2.w, self.g2.w, self.o.w, self.a_log, self.dt_bias, self.norm]
