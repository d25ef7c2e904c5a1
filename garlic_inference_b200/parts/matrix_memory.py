"""A matrix memory with exponential gates (the mLSTM cell of xLSTM), as a mixer with a matrix of state per head.

    q = Wq x * key_dim^-1/2,  k = Wk x  (n_heads x key_dim),   v = Wv x  (n_heads x value_dim)
    i = cap tanh((Wi x + bi) / cap),   f = logsigmoid(cap tanh((Wf x + bf) / cap))        log gates, one per head
    m_t = max(f + m_(t-1), i)                                                              0 before the first token
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,   n_t the same with k alone
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)
    y   = Wo( o / rms(o over value_dim) * w * sigmoid(Wg x) )

The projections of q, k, v and the output gate are one packed product; those of the two log gates are a second one
whose result stays float32.  S, n and m are float32 in a slot's state row (n and m once per slice of 32 value columns,
csrc/matrix_memory.cu says why) and are walked by one kernel for prompts, portions and single tokens alike, from zero
at a sequence's start.  Upstream has no recurrent mixer.
"""
from __future__ import annotations

import torch

from ..cache import StateRequirement
from ..ops import kernels, linear
from ..weights.loader import TensorWant
from .base import Mixer, register_part, seq_spans_array
from .linear_attention import pack_rows, scan_state_floats


def matrix_memory_floats(key_dim: int, value_dim: int) -> int:
    """Floats of one head's state: the matrix, then n and m per slice of 32 value columns (the kernel's rule)."""
    slices = -(-value_dim // 32)
    return scan_state_floats(key_dim, value_dim) + slices * scan_state_floats(key_dim, 1) + -(-slices // 4) * 4


class MatrixMemory(Mixer):
    kind = "matrix_memory"
    graph_safe = True

    @classmethod
    def wanted(cls, params):
        hid, H, d, dv = (int(params[k]) for k in ("hidden_size", "n_heads", "key_dim", "value_dim"))
        gate = lambda: TensorWant((H, hid))
        return {"q": TensorWant((H * d, hid)), "k": TensorWant((H * d, hid)), "v": TensorWant((H * dv, hid)),
                "g": TensorWant((H * dv, hid)), "i": gate(), "f": gate(), "i.b": TensorWant((H,), std_scale=10.0),
                "f.b": TensorWant((H,), std_scale=10.0), "norm": TensorWant((H * dv,), "norm"), "o": TensorWant((hid, H * dv))}

    def __init__(self, params, load, rt):
        super().__init__(params, load, rt)
        self.hidden, self.H = int(params["hidden_size"]), int(params["n_heads"])
        self.d, self.dv = int(params["key_dim"]), int(params["value_dim"])
        self.cap, self.eps = float(params["gate_cap"]), float(params["eps"])
        if not self.cap > 0:
            raise ValueError(f"gate_cap must be positive, found {self.cap}")
        self.w_in, (self.q_off, self.k_off, self.v_off, self.g_off) = pack_rows(
            load, (("q", self.H * self.d), ("k", self.H * self.d), ("v", self.H * self.dv), ("g", self.H * self.dv)),
            self.hidden, rt)
        self.w_gates, (self.i_off, self.f_off) = pack_rows(load, (("i", self.H), ("f", self.H)), self.hidden, rt)
        self.i_bias, self.f_bias = (load(n).to(torch.float32).contiguous() for n in ("i.b", "f.b"))
        self.w_o, self.norm = load("o"), load("norm")
        self.state_floats = self.H * matrix_memory_floats(self.d, self.dv)

    def cache_requirement(self):
        return StateRequirement((self.state_floats,), torch.float32)

    def step_arrays(self, shape, cache):
        return {} if shape.all_single else {"seq_spans": lambda: seq_spans_array(shape)}

    def pre_output(self, x, ctx, cache, position, writes_cache=True, out=None, out_mul=1.0):
        """Everything before the output projection: [n, n_heads * value_dim] in the activation type, times
        `out_mul`, written into `out` (columns of a wider matrix) when given."""
        if not writes_cache:
            raise ValueError("a mixer with state of its own cannot read another layer's")
        proj = linear(x, self.w_in)
        gates = linear(x, self.w_gates, out_dtype=torch.float32)
        o = kernels.matrix_memory_scan(proj, (self.q_off, self.k_off, self.v_off), gates, (self.i_off, self.f_off),
                                       self.i_bias, self.f_bias, self.cap, cache.state, ctx.seq_spans(), ctx.tok_slot,
                                       self.H, self.d, self.dv)
        return kernels.gated_group_rmsnorm(o, proj[:, self.g_off:self.g_off + self.H * self.dv], self.norm, self.eps,
                                           groups=self.H, gate_kind="sigmoid", mul=out_mul, out=out)

    def step(self, x, ctx, cache, position, writes_cache=True):
        return linear(self.pre_output(x, ctx, cache, position, writes_cache), self.w_o)


register_part(MatrixMemory.kind, MatrixMemory)
