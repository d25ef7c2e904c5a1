"""Attention whose keys and values are expanded from a cached low-rank latent, as a mixer.

    q = Wq x = per head [ plain_dim unrotated | rot_dim rotated ]
        with `q_rank`:  q = Wuq ( rmsnorm(Wdq x) * w ), the queries through a normed latent of their own
    [c | kr] = Wdkv x;  c <- rmsnorm(c) * w  (kv_rank);  kr (rot_dim): one rotated key part shared by all heads
    head h:  key = [ Wuk,h c | rot(kr) ],  value = Wuv,h c
    score = (q_plain . Wuk,h c + rot(q_rot) . rot(kr)) * softmax_scale,  causal; with `window` w the query at position i
            sees the keys with i - j < w only, and pages that fall out of it go back
    rot_dim 0: no rotated part; both latents are then normed (and c cached) in one kernel, and with rows of just the
            latent the queries are what the per-head product leaves
    softmax whose denominator also holds exp(sink_h) (optional, one learned number per head)
    o_h = sum_j p_j Wuv,h c_j;  with `head_gate`:  o_h <- o_h * sigmoid(Wg x)_h, one number per head from the mixer's input
    y = Wo concat_h( o_h )

With `own_kv` False the layer has no Wdkv: the schedule points it at another layer's cache entry, whose rows (the
normed latent and the rotated key part as that layer cached them) it reads with its own Wuk, Wuv and queries.

Only c and rot(kr) are cached: one row per position in a single-plane paged entry.  The expansion is not
materialised, but for long portions (below): q'_h = Wuk,h^T q_plain,h is made by a per-head product, attention runs over the cached rows for
all heads (score q'_h . c_j + rot(q_rot) . rot(kr_j), values c_j), and Wuv,h is applied to the result.

Which attention runs.  Everything under float32, and short portions: the exact-order kernel (scores, softmax
and weighted sum float32, one block per token and head).  Decode steps in bfloat16: the shared-rows kernel,
which stages the cached rows in shared memory once for 32 heads (asynchronous copies, a chunk ahead), cuts the
keys into slices and does both products on tensor cores (mma.sync; float32 scores, softmax and sums, the
weights rounded to bfloat16 as the second product's operand).  Portions of `PRODUCT_MIN_ROWS`
tokens and more in bfloat16: because all heads share the cached rows, the scores of a block of tokens are one
matrix product [tokens x heads, row] . [row, keys] with float32 results, the softmax (causal, with the sink,
float32) is this package's kernel, and the weighted sum is a second product [tokens x heads, keys] . [keys,
kv_rank]; the sequence's rows are gathered from its pages once per step and the tokens are cut into blocks
whose scores fit `SCORE_BYTES`.  Tensor cores do both products; the weights are rounded to bfloat16 only as
the second product's operand.
Without a rotated part, portions of plain_dim + value_dim tokens and more in bfloat16 (sizes that the flash kernels take)
expand the keys and values they see, [heads, keys, plain_dim] and [heads, keys, value_dim] by two batched products of the
gathered rows, and run the flash kernel for prompts over them as one large page (tcgen05 for sizes of 128, mma.sync
otherwise; window, sink and gate inside it): an expanded key costs kv_rank (plain_dim + value_dim) once and saves about
kv_rank per new token, and no scores are written to memory.
The rotation is the position part's (its frequencies, magnitude and layout: pairs (2i, 2i+1), or halves (i,
i + n/2)).  Upstream has grouped-query attention only (src/models/qwen3/qwen3.cpp:140-179).
"""
from __future__ import annotations

import torch

from ..cache import KVRequirement
from ..ops import kernels, linear, per_head_linear
from ..weights.loader import TensorWant
from .attention import query_runs
from .base import Mixer, StepShape, register_part
from .linear_attention import pack_rows


# From how many new tokens of a sequence on a bfloat16 step runs attention as product - softmax - product.
PRODUCT_MIN_ROWS = 32
SCORE_BYTES = 256 << 20        # float32 scores of one block of tokens (all heads, all keys)
WINDOW_BLOCK = 256             # tokens of a block when a window cuts the keys
EXPAND_BYTES = 2 << 30         # keys and values of one sequence expanded for a portion


class LatentAttention(Mixer):
    kind = "latent_attention"
    graph_safe = True

    @classmethod
    def wanted(cls, params):
        hid, H, d, dr, dv, r = (params[k] for k in ("hidden_size", "n_heads", "plain_dim", "rot_dim", "value_dim",
                                                    "kv_rank"))
        w = {"uk": TensorWant((H * d, r)), "uv": TensorWant((H * dv, r)), "o": TensorWant((hid, H * dv))}
        if params.get("q_rank"):
            qr = params["q_rank"]
            w.update({"dq": TensorWant((qr, hid)), "dq.norm": TensorWant((qr,), "norm"), "uq": TensorWant((H * (d + dr), qr))})
        else:
            w["q"] = TensorWant((H * (d + dr), hid))
        if params.get("own_kv", True):
            w.update({"dkv": TensorWant((r + dr, hid)), "dkv.norm": TensorWant((r,), "norm")})
        if params.get("head_gate", False):
            w["g"] = TensorWant((H, hid))
        if params.get("sink", False):
            w["sink"] = TensorWant((H,), std_scale=20.0)
        return w

    def __init__(self, params, load, rt):
        super().__init__(params, load, rt)
        self.hidden, self.H = int(params["hidden_size"]), int(params["n_heads"])
        self.d, self.dr, self.dv, self.rank = (int(params[k]) for k in ("plain_dim", "rot_dim", "value_dim", "kv_rank"))
        self.scale, self.eps = float(params["softmax_scale"]), float(params["eps"])
        self.window = int(params.get("window") or 0)
        self.q_rank = int(params.get("q_rank") or 0)
        self.own_kv, self.head_gate = bool(params.get("own_kv", True)), bool(params.get("head_gate", False))
        self.row = -(-(self.rank + self.dr) // 8) * 8             # a cache row, padded for the kernel's 16-byte loads
        # everything that reads the mixer's input is one product: [queries or their latent | latent and key part | gates]
        packed = [("dq", self.q_rank) if self.q_rank else ("q", self.H * (self.d + self.dr))]
        packed += [("dkv", self.rank + self.dr)] if self.own_kv else []
        packed += [("g", self.H)] if self.head_gate else []
        self.w_in, offs = pack_rows(load, packed, self.hidden, rt)
        self.q_off = offs[0]
        self.c_off = offs[1] if self.own_kv else None
        self.g_off = offs[-1] if self.head_gate else None
        self.q_norm, self.w_uq = (load("dq.norm"), load("uq")) if self.q_rank else (None, None)
        self.c_norm = load("dkv.norm") if self.own_kv else None
        # Wuk per head as [rank, plain_dim]: the product q'_h = Wuk,h^T q_h in the [out, in] form of the others
        self.w_uk_t = load("uk").view(self.H, self.d, self.rank).transpose(1, 2).contiguous()
        self.w_uv = load("uv").view(self.H, self.dv, self.rank)
        self.w_o = load("o")
        self.sink = load("sink") if params.get("sink", False) else None
        self.sink_f32 = self.sink.to(torch.float32).contiguous() if self.sink is not None else None
        self._one_page = None
        self._no_rotation = None

    def cache_requirement(self):
        return KVRequirement(1, self.row, self.window or None, planes=1)

    def _rotation(self, position, device):
        if position is not None:
            freq, magnitude, n_rot, layout = position.rotary_frequencies()
            if n_rot > self.dr:
                raise ValueError(f"{n_rot} rotated dimensions of a key part of {self.dr}")
            return freq, magnitude, n_rot, layout == "half"
        if self._no_rotation is None:
            self._no_rotation = torch.zeros(0, dtype=torch.float32, device=device)
        return self._no_rotation, 1.0, 0, False

    # ---- portions whose keys and values are expanded ------------------------------------------------
    def _first_seen(self, p: int) -> int:
        """First position that the query at position p sees."""
        return max(0, p - self.window + 1) if self.window else 0

    def _first_page(self, past: int, page: int) -> int:
        """Logical page of the first position that a portion behind `past` positions sees (those before may be gone)."""
        return self._first_seen(past) // page

    def _expands(self, n_new: int, past: int, page: int) -> bool:
        keys = (-(-(past + n_new) // page) - self._first_page(past, page)) * page
        return (self.rt.dtype == torch.bfloat16 and self.dr == 0 and n_new >= max(PRODUCT_MIN_ROWS, self.d + self.dv)
                and self.w_uv.dtype == torch.bfloat16 and self.w_uk_t.dtype == torch.bfloat16
                and kernels.mma_attention_takes(self.rt.dtype, self.d, self.dv)
                and self.H * keys * (self.d + self.dv) * 2 <= EXPAND_BYTES)

    def _run_rows(self, keys: int) -> int:
        """Rows of a run of the flash kernel that takes a page of `keys` expanded keys."""
        return 128 if self.d == self.dv and kernels.tcgen05_attention_takes(self.rt.dtype, self.d, keys) else 64

    def _runs_of(self, shape, page: int):
        """[(sequence, first page, keys, rows of a run)] of the step's portions that are expanded, and all their runs one
        after the other; slot 0 and positions counted from the first page, as the expanded page holds them."""
        import numpy as np
        which, runs = [], []
        for i, (start, n_new, past) in enumerate(zip(shape.seq_starts, shape.seq_lens, shape.seq_past)):
            if not self._expands(n_new, past, page):
                continue
            p0 = self._first_page(past, page)
            keys = (-(-(past + n_new) // page) - p0) * page
            which.append((i, p0, keys, self._run_rows(keys)))
            runs.append(query_runs(StepShape([0], [start], [n_new], [past - p0 * page], False), which[-1][3]))
        return which, np.concatenate(runs) if runs else np.zeros((0, 4), dtype=np.int32)

    def _runs_name(self, page: int) -> str:
        return f"latent_runs_{self.window}_{page}_{self.d}_{self.dv}_{self.H}"

    def step_arrays(self, shape, cache):
        page = cache.kv.page_size
        if shape.all_single or not any(self._expands(m, p, page) for m, p in zip(shape.seq_lens, shape.seq_past)):
            return {}
        return {self._runs_name(page): lambda: self._runs_of(shape, page)[1]}

    def _attend_expanded(self, q, kv, ctx, which, gate, out):
        """Attention of the expanded portions of q [n, H, plain_dim], gated, into their rows of `out` [n, H * value_dim]."""
        page = kv.page_size
        pool = kv.k_pool.view(kv.k_pool.shape[0], page, self.row)
        runs = ctx.arrays.get(self._runs_name(page))
        if runs is None:                           # a context put together by hand: cut and copy here
            runs = ctx.arrays[self._runs_name(page)] = torch.from_numpy(self._runs_of(ctx, page)[1]).to(q.device)
        if self._one_page is None:
            self._one_page = torch.zeros((1, 1), dtype=torch.int32, device=q.device)
        at = 0
        for i, p0, keys, rows in which:
            n_runs = -(-ctx.seq_lens[i] // rows)
            c = pool.index_select(0, kv.block_table[ctx.seq_slots[i], p0:p0 + keys // page].long()).view(1, keys, self.row)
            c = c[:, :, :self.rank].expand(self.H, keys, self.rank)
            k, v = torch.bmm(c, self.w_uk_t), torch.bmm(c, self.w_uv.transpose(1, 2))
            args = (q, k.unsqueeze(0), v.unsqueeze(0), self._one_page, runs[at:at + n_runs], self.scale)
            if rows == 128:
                kernels.attention_prefill_tcgen05(*args, self.window, sinks=self.sink_f32, gate=gate, out=out)
            else:
                kernels.attention_prefill_masked_bf16(*args, window=self.window, sinks=self.sink_f32, gate=gate, out=out)
            at += n_runs

    def step(self, x, ctx, cache, position, writes_cache=True):
        return linear(self.pre_output(x, ctx, cache, position, writes_cache), self.w_o)

    def pre_output(self, x, ctx, cache, position, writes_cache=True, out=None, out_mul=1.0):
        """Everything before the output projection: [n, n_heads * value_dim] in the activation type, times
        `out_mul`, written into `out` (columns of a wider matrix) when given."""
        kv = cache.kv
        if self.own_kv != bool(writes_cache):
            raise ValueError("a layer with a latent of its own writes its cache entry, and one without reads another "
                             "layer's: the schedule says otherwise")
        n = x.shape[0]
        freq, magnitude, n_rot, half = self._rotation(position, x.device)
        proj = linear(x, self.w_in)
        # without a rotated part the latents depend on nothing but this product: one kernel norms both and caches c
        both = self.dr == 0 and self.q_rank and self.own_kv and self.q_norm.dtype == self.c_norm.dtype
        if both:
            q_src, q_off = linear(kernels.latent_norms(proj, self.q_off, self.c_off, self.q_norm, self.c_norm, self.eps, ctx.tok_pos,
                                                       ctx.tok_slot, kv.block_table, kv.k_pool, ctx.status), self.w_uq), 0
        elif self.q_rank:
            q_src, q_off = linear(kernels.rmsnorm_rows(proj[:, self.q_off:self.q_off + self.q_rank], self.q_norm, self.eps),
                                  self.w_uq), 0
        else:
            q_src, q_off = proj, self.q_off
        q = q_src[:, q_off:q_off + self.H * (self.d + self.dr)].view(n, self.H, self.d + self.dr)
        plain = not self.head_gate and out is None and out_mul == 1.0
        gate = proj[:, self.g_off:self.g_off + self.H] if self.head_gate else None
        # portions whose keys and values are expanded (the latents above are in the cache by now)
        which = []
        if both and out is None and out_mul == 1.0 and not ctx.all_single and not ctx.captured and ctx.seq_lens:
            which, _ = self._runs_of(ctx, kv.page_size)
        if len(which) == len(ctx.seq_lens) > 0 and n == sum(ctx.seq_lens):
            done = torch.empty((n, self.H * self.dv), dtype=self.rt.dtype, device=x.device)
            self._attend_expanded(q.contiguous(), kv, ctx, which, gate, done)
            return done
        q_lat = per_head_linear(q[:, :, :self.d], self.w_uk_t)                       # [n, H, rank]
        q_rows = q_lat if both and self.row == self.rank else \
            kernels.latent_prepare(q_src, q_off, proj if self.own_kv and not both else None, self.c_off or 0, q_lat,
                                   self.c_norm, self.eps, freq, magnitude, n_rot, ctx.tok_pos, ctx.tok_slot, kv.block_table,
                                   kv.k_pool, self.H, self.d, self.dr, self.rank, ctx.status,
                                   append=writes_cache and not both, half_layout=half)
        o_lat = self.attend(q_rows, kv, ctx, skip={w[0] for w in which})
        # with a gate (or a factor, or columns to write into) the values leave their product in float32 and are
        # rounded once, after the gate
        o = per_head_linear(o_lat.view(n, self.H, self.rank), self.w_uv,
                            out_dtype=None if plain else torch.float32)             # [n, H, value_dim]
        done = o.view(n, self.H * self.dv)
        if not plain:
            done = kernels.attn_finish(done, self.H, 1, None, None, out_mul, gate, self.rt.dtype, out=out)
        if which:
            self._attend_expanded(q.contiguous(), kv, ctx, which, gate, done)
        return done

    def attend(self, q_rows, kv, ctx, skip=frozenset()):
        """Attention of q_rows [n, H, row] over the cached rows; returns [n, H * kv_rank].  The rows of sequences in `skip`
        may be left as they are."""
        by_products = (q_rows.dtype == torch.bfloat16 and not ctx.all_single and not ctx.captured and ctx.seq_lens
                       and max(ctx.seq_lens) >= PRODUCT_MIN_ROWS)
        if ctx.all_single and kernels.latent_decode_takes(q_rows.dtype, q_rows.shape[2], self.rank, self.H):
            return kernels.latent_decode(q_rows, kv.k_pool, kv.block_table, ctx.tok_pos, ctx.tok_slot, self.scale,
                                         self.sink, self.rank, ctx.status, window=self.window)
        if not by_products:
            return kernels.attention_generic(q_rows, kv.k_pool, kv.k_pool, kv.block_table, ctx.tok_pos, ctx.tok_slot,
                                             self.scale, self.window, ctx.status, sinks=self.sink, value_dim=self.rank)
        n, H, row = q_rows.shape
        out = torch.empty((n, H * self.rank), dtype=q_rows.dtype, device=q_rows.device)
        page = kv.page_size
        pool = kv.k_pool.view(kv.k_pool.shape[0], page, row)
        short = [(s, st, m, p) for s, st, m, p in zip(ctx.seq_slots, ctx.seq_starts, ctx.seq_lens, ctx.seq_past)
                 if m < PRODUCT_MIN_ROWS]
        for i, (slot, start, n_new, past) in enumerate(zip(ctx.seq_slots, ctx.seq_starts, ctx.seq_lens, ctx.seq_past)):
            if n_new < PRODUCT_MIN_ROWS or i in skip:
                continue
            n_pages = -(-(past + n_new) // page)
            p0 = self._first_page(past, page)
            rows = pool.index_select(0, kv.block_table[slot, p0:n_pages].long()).view((n_pages - p0) * page, row)
            block = max(1, min(n_new, SCORE_BYTES // (4 * H * (n_pages - p0) * page)))
            if self.window:                            # a block sees its window and itself: a short block wastes less
                block = min(block, WINDOW_BLOCK)
            for q0 in range(0, n_new, block):
                tq = min(block, n_new - q0)
                k0 = max(p0 * page, self._first_seen(past + q0) // 8 * 8)       # first key of the block's products
                # what this block sees, padded to 8
                r0, r1 = k0 - p0 * page, min(-(-(past + q0 + tq) // 8) * 8, n_pages * page) - p0 * page
                q = q_rows[start + q0:start + q0 + tq].view(tq * H, row)
                scores = torch.mm(q, rows[r0:r1].t(), out_dtype=torch.float32)
                weights = kernels.causal_sink_softmax(scores, H, past + q0, self.scale, self.sink, q_rows.dtype,
                                                      window=self.window, first_key=k0)
                out[start + q0:start + q0 + tq] = torch.mm(weights, rows[r0:r1, :self.rank]).view(tq, H * self.rank)
        if short:                                  # sequences that bring a few tokens: the exact-order kernel
            idx = torch.cat([torch.arange(st, st + m) for _, st, m, _ in short]).to(q_rows.device)
            part = kernels.attention_generic(q_rows.index_select(0, idx).contiguous(), kv.k_pool, kv.k_pool,
                                             kv.block_table, ctx.tok_pos.index_select(0, idx).contiguous(),
                                             ctx.tok_slot.index_select(0, idx).contiguous(), self.scale, self.window,
                                             ctx.status, sinks=self.sink, value_dim=self.rank)
            out.index_copy_(0, idx, part)
        return out


register_part(LatentAttention.kind, LatentAttention)
