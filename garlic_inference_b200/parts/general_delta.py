"""The generalized delta rule, as a mixer with a matrix of state per head: a decay and a removal rate per head and key
channel, both made from the input.

    r = Wr x,  k = Wk x,  v = Wv x                       n_heads x head_dim each
    w = exp(-exp(-1/2) sigmoid(W2 tanh(W1 x) + w0))       decay
    a = sigmoid(Wa x + a0)                                removal rate
    u = k / sqrt(|k|^2 + unit_eps)                        per head
    S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T    (the old S in both);   o_t = S_t^T r
    y = Wo( o / rms(o over head_dim) * norm * sigmoid(Wg x) )

The projections of r, k, v and the output gate are one packed product; those of the removal rate and the thin first
factor of the decay are a second one whose result stays float32, as does the second thin product's.  The state is
float32 in a slot's state row and is walked by one kernel for prompts, portions and single tokens alike, from zero at a
sequence's start.  Upstream has no recurrent mixer.
"""
from __future__ import annotations

import torch

from ..cache import StateRequirement
from ..ops import kernels, linear
from ..weights.loader import TensorWant
from .base import Mixer, register_part, seq_spans_array
from .linear_attention import pack_rows, scan_state_floats


class GeneralDeltaRule(Mixer):
    kind = "general_delta_rule"
    graph_safe = True

    @classmethod
    def wanted(cls, params):
        hid, H, d, r = (int(params[k]) for k in ("hidden_size", "n_heads", "head_dim", "decay_rank"))
        wide = lambda: TensorWant((H * d, hid))
        return {"r": wide(), "k": wide(), "v": wide(), "g": wide(), "a": wide(), "a.b": TensorWant((H * d,), std_scale=10.0),
                "w1": TensorWant((r, hid)), "w2": TensorWant((H * d, r), std_scale=4.0),
                "w0": TensorWant((H * d,), std_scale=10.0), "norm": TensorWant((H * d,), "norm"), "o": TensorWant((hid, H * d))}

    def __init__(self, params, load, rt):
        super().__init__(params, load, rt)
        self.hidden, self.H, self.d = int(params["hidden_size"]), int(params["n_heads"]), int(params["head_dim"])
        self.rank, self.eps = int(params["decay_rank"]), float(params["eps"])
        self.unit_eps = float(params.get("unit_eps", 1e-6))
        C = self.C = self.H * self.d
        self.w_in, (self.r_off, self.k_off, self.v_off, self.g_off) = pack_rows(
            load, (("r", C), ("k", C), ("v", C), ("g", C)), self.hidden, rt)
        self.w_aw, (self.a_off, self.w1_off) = pack_rows(load, (("a", C), ("w1", self.rank)), self.hidden, rt)
        self.w2 = load("w2")
        self.decay_bias, self.removal_bias = (load(n).to(torch.float32).contiguous() for n in ("w0", "a.b"))
        self.w_o, self.norm = load("o"), load("norm")
        self.state_floats = self.H * scan_state_floats(self.d, self.d)

    def cache_requirement(self):
        return StateRequirement((self.state_floats,), torch.float32)

    def step_arrays(self, shape, cache):
        return {} if shape.all_single else {"seq_spans": lambda: seq_spans_array(shape)}

    def pre_output(self, x, ctx, cache, position, writes_cache=True, out=None, out_mul=1.0):
        """Everything before the output projection: [n, n_heads * head_dim] in the activation type, times `out_mul`,
        written into `out` (columns of a wider matrix) when given."""
        if not writes_cache:
            raise ValueError("a mixer with state of its own cannot read another layer's")
        proj = linear(x, self.w_in)
        aw = linear(x, self.w_aw, out_dtype=torch.float32)
        thin = kernels.tanh_rows(aw[:, self.w1_off:self.w1_off + self.rank], self.rt.dtype)
        decay = linear(thin, self.w2, out_dtype=torch.float32)
        removal = aw[:, self.a_off:self.a_off + self.C]
        if not ctx.all_single:                       # many tokens: the exponentials once, not in every slice of the scan
            kernels.general_delta_rates(decay, self.decay_bias, removal, self.removal_bias, self.rt.dtype)
        o = kernels.general_delta_scan(proj, (self.r_off, self.k_off, self.v_off), decay, self.decay_bias, removal,
                                       self.removal_bias, cache.state, ctx.seq_spans(), ctx.tok_slot, self.H, self.d,
                                       self.d, self.unit_eps, ready=not ctx.all_single)
        return kernels.gated_group_rmsnorm(o, proj[:, self.g_off:self.g_off + self.C], self.norm, self.eps, groups=self.H,
                                           gate_kind="sigmoid", mul=out_mul, out=out)

    def step(self, x, ctx, cache, position, writes_cache=True):
        return linear(self.pre_output(x, ctx, cache, position, writes_cache), self.w_o)


register_part(GeneralDeltaRule.kind, GeneralDeltaRule)
