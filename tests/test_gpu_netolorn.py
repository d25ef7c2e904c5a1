"""Netolorn through the engine against the plain implementation: each mechanism alone, prompts against token-by-token
decoding, portions, batches, slots and pages used again, keys just inside and just outside windows and kept first tokens,
the first tokens, long decoding, generation, the two programs, and the kernels alone."""
import math

import numpy as np
import pytest
import torch

import plain_netolorn as plain
import tiny
import tiny_netolorn as tk

pytestmark = pytest.mark.gpu

_DIRS, _MODELS = {}, {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    def get(name):
        if name not in _DIRS:
            _DIRS[name] = tk.write_model(name, tmp_path_factory.mktemp(f"netolorn_{name}"))
        return _DIRS[name]
    return get


@pytest.fixture(scope="module")
def model(folder):
    def get(name, dtype, max_tokens=4096, page_size=16, **kw):
        key = (name, dtype, max_tokens, page_size, tuple(sorted(kw.items())))
        if key not in _MODELS:
            from garlic_inference_b200 import AutoModel
            _MODELS[key] = AutoModel.from_pretrained(folder(name), device=0, dtype=dtype, max_tokens=max_tokens,
                                                     page_size=page_size, **kw)
        return _MODELS[key]
    return get


def _requests(name, lengths, seed):
    return tiny.random_requests(tk.TINY[name]["vocab"], lengths, seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["window", "causal", "latent", "dense", "moe", "mix", "tc", "odd", "ones"])
def test_prompts_decoding_portions_and_batches_agree_with_the_plain_model(name, dtype, model, folder):
    """Every way of cutting the same requests gives the plain logits: whole prompts; all but 40 tokens, then one at a
    time; portions of 2, 7, 33 and 3 tokens; portions with all requests in one batch; unequal requests that start
    together and decode together.  The cache has room for one batch only, so slots and pages are given back and used
    again by later requests; windows pass over prompts and over decoded tokens."""
    m = model(name, dtype, max_tokens=512, page_size=16, max_slots=4)
    reqs = _requests(name, [70, 1, 37, 150], seed=5)
    want, own = tk.plain_pair(folder(name), reqs)
    for what, steps in (("whole", tiny.trace_whole(reqs)),
                        ("tail", tiny.trace_tail_by_one(reqs, tail=40)),
                        ("portions", tk.trace_portions(reqs, [2, 7, 33, 3])),
                        ("portions together", tk.trace_portions(reqs, [5, 2, 64], together=True)),
                        ("batched", tiny.trace_batched(reqs, [["r3", "r1"], ["r0", "r2", "r1"]], prompt_frac=0.6))):
        got = tiny.run_trace_in_process(m, steps)
        tiny.assert_covers(got, reqs)
        tk.judge_routed(got, want, own, dtype, f"{name} {dtype} {what}", folder(name), reqs)
    assert m.engine.cache.slots.n_free == 4, "every slot came back"
    assert all(g.host.pool.n_free == g.host.pool.n_pages for g in m.engine.cache.groups), "every page came back"


def test_tensor_core_kernels_on_pages_of_64(model, folder):
    """The same on pages of 64 tokens, where prompts of the heads of 128 run the tcgen05 kernel and the other tensor-core
    head sizes the mma.sync kernels, with window, kept tokens, sinks and gates inside them."""
    m = model("tc", "bfloat16", max_tokens=2048, page_size=64, max_slots=4)
    reqs = _requests("tc", [300, 3, 129, 64], seed=15)
    want, own = tk.plain_pair(folder("tc"), reqs)
    for steps in (tiny.trace_whole(reqs), tiny.trace_tail_by_one(reqs, tail=70), tk.trace_portions(reqs, [65, 2, 30]),
                  tiny.trace_batched(reqs, [list(reqs)], prompt_frac=0.5)):
        got = tiny.run_trace_in_process(m, steps)
        tiny.assert_covers(got, reqs)
        tk.judge_routed(got, want, own, "bfloat16", "tc on pages of 64", folder("tc"), reqs)


@pytest.mark.parametrize("name,page,sizes", [("long", 64, [300, 140, 290, 20]), ("long", 48, [270, 31, 300, 2]),
                                             ("tc", 16, [60, 5, 33, 90])])
def test_long_portions_expand_the_latent_rows_they_see(name, page, sizes, model, folder, monkeypatch):
    """Latent attention in portions long enough that keys and values are expanded, behind windows whose pages are gone,
    beside sequences of the same step that bring a few tokens; pages of 64 (the tcgen05 kernel for heads of 128), of 48
    and of 16 (mma.sync).  The same rows without the expansion differ by rounding alone."""
    from garlic_inference_b200.parts import LatentAttention
    seen = []
    whole = LatentAttention._attend_expanded
    monkeypatch.setattr(LatentAttention, "_attend_expanded",
                        lambda self, q, kv, ctx, which, gate, out: (seen.append((len(which), len(ctx.seq_lens), which)),
                                                                    whole(self, q, kv, ctx, which, gate, out))[1])
    m = model(name, "bfloat16", max_tokens=4096, page_size=page, max_slots=4)
    reqs = _requests(name, [900, 760, 30] if name == "long" else [200, 150, 9], seed=23)
    want, own = tk.plain_pair(folder(name), reqs)
    steps = tk.trace_portions(reqs, sizes, together=True)
    got = tiny.run_trace_in_process(m, steps)
    tiny.assert_covers(got, reqs)
    tk.judge_routed(got, want, own, "bfloat16", f"expanded {name} {page}", folder(name), reqs)
    assert any(a == b for a, b, _ in seen) and any(a < b for a, b, _ in seen), "whole steps and parts of steps"
    assert any(w[1] > 0 for _, _, which in seen for w in which), "a portion whose first page is gone"
    kinds = {w[3] for _, _, which in seen for w in which}
    assert kinds == ({64} if name == "tc" or page == 48 else {128})
    count = len(seen)
    monkeypatch.setattr(LatentAttention, "_expands", lambda self, n_new, past, page: False)
    other = tiny.run_trace_in_process(m, steps)
    tk.judge_routed(other, want, own, "bfloat16", f"not expanded {name} {page}", folder(name), reqs)
    assert len(seen) == count


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_of_a_thousand_tokens_through_the_trace_program(dtype, folder, tmp_path):
    """Requests of 1,100, 425, 97 and 1 tokens through bin/trace_run on its default pages of 64: whole, and started
    together with their last 40 % decoded together."""
    reqs = _requests("long", [1100, 425, 97, 1], seed=17)
    want, own = tk.plain_pair(folder("long"), reqs)
    steps = tiny.trace_whole(reqs) + [dict(s, step=s["step"] + 4, entries=[dict(e, id=e["id"] + "b") for e in s["entries"]],
                                           end=[r + "b" for r in s["end"]])
                                      for s in tiny.trace_batched(reqs, [list(reqs)], prompt_frac=0.6)]
    got = tiny.run_trace_program(folder("long"), dtype, steps, tmp_path / "out", 2048, tk.TINY["long"]["vocab"])
    first = {rid: rows for rid, rows in got.items() if not rid.endswith("b")}
    second = {rid[:-1]: rows for rid, rows in got.items() if rid.endswith("b")}
    for part, what in ((first, "whole"), (second, "together")):
        tiny.assert_covers(part, reqs)
        tk.judge_routed(part, want, own, dtype, f"long {dtype} {what}", folder("long"), reqs)


def test_float32_logits_do_not_depend_on_the_cut_or_the_batch(model):
    """Without routed experts (whose few-row and many-row paths sum in different orders) the same position gives the
    same bits whole, in portions, decoded, alone or in a batch."""
    for name in ("window", "causal", "latent", "dense"):
        m = model(name, "float32", max_tokens=1024, page_size=16)
        reqs = _requests(name, [90, 33], seed=6)
        base = tiny.run_trace_in_process(m, tiny.trace_whole(reqs))
        for steps in (tk.trace_portions(reqs, [2, 31, 8]), tiny.trace_tail_by_one(reqs, tail=20),
                      tk.trace_portions(reqs, [16, 3], together=True)):
            got = tiny.run_trace_in_process(m, steps)
            for rid in reqs:
                for p in range(len(reqs[rid])):
                    assert np.array_equal(got[rid][p], base[rid][p]), f"{name}: request {rid} position {p} differs in its bits"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "tc"])
def test_long_decoding(name, dtype, model, folder):
    """300 tokens decoded one at a time after a prompt of 5, two requests together, through the recorded decode step:
    cache pages taken and given back one by one while the kept first tokens' pages stay."""
    m = model(name, dtype, max_tokens=1024, page_size=16)
    reqs = _requests(name, [305, 280], seed=9)
    want, own = tk.plain_pair(folder(name), reqs)
    got = tiny.run_trace_in_process(m, tiny.trace_batched(reqs, [["r0", "r1"]], prompt_frac=5 / 305))
    tiny.assert_covers(got, reqs)
    tk.judge_routed(got, want, own, dtype, f"long decoding {name} {dtype}", folder(name), reqs)
    assert m.engine.graphs is not None and 2 in m.engine.graphs._graphs, "decode steps ran from a recorded graph"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["moe", "mix", "tc"])
def test_a_dozen_requests_decode_together(name, dtype, model, folder):
    """Twelve unequal requests start together and decode together through a recorded step of 16 rows (four of them
    padding), and leave one after the other."""
    m = model(name, dtype, max_tokens=2048, page_size=16, max_slots=12)
    reqs = _requests(name, [31 + 3 * i for i in range(12)], seed=21)
    want, own = tk.plain_pair(folder(name), reqs)
    got = tiny.run_trace_in_process(m, tiny.trace_batched(reqs, [list(reqs)], prompt_frac=0.5))
    tiny.assert_covers(got, reqs)
    tk.judge_routed(got, want, own, dtype, f"twelve together {name} {dtype}", folder(name), reqs)
    assert m.engine.graphs is not None and 16 in m.engine.graphs._graphs


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(dtype, model, folder):
    m = model("mix", dtype, max_tokens=512, page_size=16, max_slots=3)
    prompts = list(_requests("mix", [9, 1, 30, 17, 5], seed=10).values())
    got = m.generate(prompts, max_new_tokens=10)
    assert m.last_stats.batches == 2
    cfg, w = plain.read_model_dir(folder("mix"))
    for prompt, new in zip(prompts, got):
        ids = list(prompt)
        assert len(new) == 10
        for k, tok in enumerate(new):
            logits = plain.forward(cfg, w, ids)[-1]
            best = int(logits.argmax())
            if tok != best:
                gap = float(logits[best] - logits[tok]) / float(logits.abs().max())
                assert dtype == "bfloat16" and gap <= 0.1, \
                    f"prompt of {len(prompt)}, new token {k}: engine chose {tok}, plain {best} (gap {gap:.2e})"
                break
            ids.append(tok)


def test_trace_program_and_command_line_serve_the_design(folder, tmp_path):
    import subprocess
    import sys
    reqs = _requests("odd", [20, 3], seed=12)
    want, own = tk.plain_pair(folder("odd"), reqs)
    steps = tiny.trace_batched(reqs, [["r0", "r1"]])
    got = tiny.run_trace_program(folder("odd"), "float32", steps, tmp_path / "out", 256, tk.TINY["odd"]["vocab"])
    tk.judge(got, want, own, "float32", "trace program")
    r = subprocess.run([sys.executable, str(tiny.REPO / "bin" / "runner"), str(folder("odd")), "--prompt-ids", "5,6,7",
                        "--max-new-tokens", "4", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    ids = [int(t) for t in r.stdout.splitlines()[0].split()]
    cfg, w = plain.read_model_dir(folder("odd"))
    seq = [5, 6, 7]
    for tok in ids:
        assert tok == int(plain.forward(cfg, w, seq)[-1].argmax())
        seq.append(tok)


# ---- kernels alone -----------------------------------------------------------------------------
def _paged(keys, values, page, spare=3):
    """Pools and a block table (slot 1) that hold keys [T, G, d] and values [T, G, dv] on pages out of order."""
    T, G, d = keys.shape
    dv = values.shape[2]
    n_pages = -(-T // page)
    order = torch.randperm(n_pages + spare)[:n_pages]
    k_pool = torch.zeros(n_pages + spare, G, page, d, dtype=keys.dtype, device="cuda")
    v_pool = torch.zeros(n_pages + spare, G, page, dv, dtype=keys.dtype, device="cuda")
    for j in range(T):
        k_pool[order[j // page], :, j % page] = keys[j]
        v_pool[order[j // page], :, j % page] = values[j]
    table = torch.full((2, n_pages + 1), -1, dtype=torch.int32, device="cuda")
    table[1, :n_pages] = order.to(torch.int32)
    return k_pool, v_pool, table


def _plain_attention(q, k, v, scale, sink, size, keep, gate=None):
    T, H, _ = q.shape
    G = k.shape[1]
    seen = plain.window_mask(T, size, keep)
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h].double() @ k[:, g].double().T) * scale
        out[:, h] = plain.softmax_sink(s, seen, sink[h].double()) @ v[:, g].double()
    return out if gate is None else out * torch.sigmoid(gate.double())


def _dropped(table, page, size, keep, T):
    """The table of a sequence of T positions whose pages out of sight of the last query have gone back."""
    out = table.clone()
    for lp in range(max(0, T - size) // page):
        if lp * page >= keep:
            out[1, lp] = -1
    return out


@pytest.mark.parametrize("shape", [(6, 2, 32, 64, 16, torch.float32), (6, 2, 32, 64, 16, torch.bfloat16), (4, 2, 64, 64, 16, torch.bfloat16),
                                   (4, 1, 128, 128, 64, torch.bfloat16), (3, 3, 10, 6, 16, torch.float32)])
def test_windows_with_kept_first_tokens_sinks_and_gates(shape):
    """One key is made to stand out so far that every query which sees it reads its value alone and every other does not,
    at places just inside and just outside the window's far edge and the kept tokens' last position.  Exact-order kernel,
    mma.sync prompt kernel, tcgen05 prompt kernel (heads of 128 on pages of 64), split-KV decode kernel on a table whose
    pages out of sight are gone."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.parts import StepShape
    from garlic_inference_b200.parts.attention import query_runs
    H, G, d, dv, page, dtype = shape
    torch.manual_seed(d)
    T, scale = 300, 0.4
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    slot = torch.ones(T, dtype=torch.int32, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    sink = torch.randn(H)
    runs = {n: torch.from_numpy(query_runs(StepShape([1], [0], [T], [0], False), n)).cuda() for n in (64, 128)}
    for size, keep in ((72, 20), (40, 0), (64, 64), (70, 65), (33, 130), (1, 1), (129, 3), (400, 7)):
        for far in sorted({0, max(keep - 1, 0), keep, 100, 127, 128}):
            k, v, q = torch.randn(T, G, d) * 0.3, torch.randn(T, G, dv), torch.randn(T, H, d) * 0.3
            k[far, :, :4] = 8.0
            q[:, :, :4] = 2.0
            gate = torch.randn(T, H * dv)
            q, k, v, gate = q.to(dtype), k.to(dtype), v.to(dtype), gate.to(dtype)
            g3 = gate.float().view(T, H, dv)
            want = _plain_attention(q.float(), k.float(), v.float(), scale, sink, size, keep, g3)
            # what the comparison rests on: the far key decides where it is seen, and only there
            alone = v[far].float().repeat_interleave(H // G, 0).double() * torch.sigmoid(g3.double())
            last = far + size - 1
            if far + 1 < T:
                assert float((want[min(last, T - 1)] - alone[min(last, T - 1)]).abs().max()) < 1e-2
            if last + 1 < T and far >= keep:
                assert float((want[last + 1] - alone[last + 1]).abs().max()) > 1e-2, "out of the window"
            if far < keep:
                assert float((want[T - 1] - alone[T - 1]).abs().max()) < 1e-2, "a kept token is seen to the end"
            kp, vp, table = _paged(k.cuda(), v.cuda(), page)
            qc, gc, sc = q.cuda(), gate.cuda(), sink.cuda()
            got = kernels.attention_masked(qc, kp, vp, table, pos, slot, scale, status, window=size, sinks=sc, keep_first=keep,
                                           out_float32=True)
            got = kernels.attn_finish(got, H, 1, None, None, 1.0, gc, dtype)
            torch.testing.assert_close(got.cpu().double().view(T, H, dv), want, **tol)
            if dtype == torch.float32:
                continue
            got = kernels.attention_prefill_masked_bf16(qc, kp, vp, table, runs[64], scale, window=size, sinks=sc, keep_first=keep,
                                                        gate=gc, rows_covered=True)
            torch.testing.assert_close(got.cpu().double().view(T, H, dv), want, **tol)
            if d == 128:
                got = kernels.attention_prefill_tcgen05(qc, kp, vp, table, runs[128], scale, size, rows_covered=True, sinks=sc,
                                                        keep_first=keep, gate=gc)
                torch.testing.assert_close(got.cpu().double().view(T, H, dv), want, **tol)
            for t in sorted({far, min(last, T - 1), min(last + 1, T - 1), T - 1}):
                gone = _dropped(table, page, size, keep, t + 1)
                at = torch.tensor([t], device="cuda")
                for n_splits in (1, 3):
                    one = kernels.attention_decode_masked_bf16(qc[at].contiguous(), kp, vp, gone, pos[at].contiguous(),
                                                               slot[at].contiguous(), scale, n_splits=n_splits, window=size,
                                                               sinks=sc, keep_first=keep, gate=gc[at])
                    torch.testing.assert_close(one.cpu().double().view(1, H, dv), want[t:t + 1], **tol)
                one = kernels.attention_masked(qc[at].contiguous(), kp, vp, gone, pos[at].contiguous(), slot[at].contiguous(),
                                               scale, status, window=size, sinks=sc, keep_first=keep, out_float32=True)
                one = one.cpu().double().view(1, H, dv) * torch.sigmoid(g3[t:t + 1].double())
                torch.testing.assert_close(one, want[t:t + 1], **tol)
    assert int(status.item()) == 0
    kernels.check_bounded_waits(torch.device("cuda", 0))


def test_prompt_portions_that_continue_behind_a_window(shape=(4, 2, 128)):
    """A portion of a prompt whose earlier pages are gone but for the kept tokens': rows 230 .. 362 of a sequence, on
    the tcgen05 and the mma.sync kernel."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.parts import StepShape
    from garlic_inference_b200.parts.attention import query_runs
    H, G, d = shape
    torch.manual_seed(12)
    T, past, size, keep, page, scale = 363, 230, 50, 40, 64, 0.1
    k, v, q = torch.randn(T, G, d).bfloat16(), torch.randn(T, G, d).bfloat16(), torch.randn(T, H, d).bfloat16()
    sink, gate = torch.randn(H), torch.randn(T, H * d).bfloat16()
    want = _plain_attention(q.float(), k.float(), v.float(), scale, sink, size, keep, gate.float().view(T, H, d))
    kp, vp, table = _paged(k.cuda(), v.cuda(), page)
    gone = _dropped(table, page, size, keep, past + 1)
    assert int(gone[1, 0]) >= 0 and int(gone[1, 1]) < 0 and int(gone[1, 2]) >= 0, "page 1 is gone, page 0 is kept"
    for rows in (64, 128):
        runs = torch.from_numpy(query_runs(StepShape([1], [0], [T - past], [past], False), rows)).cuda()
        args = (q[past:].contiguous().cuda(), kp, vp, gone, runs, scale)
        kw = dict(rows_covered=True, sinks=sink.cuda(), keep_first=keep, gate=gate[past:].contiguous().cuda())
        got = kernels.attention_prefill_tcgen05(*args, size, **kw) if rows == 128 else \
            kernels.attention_prefill_masked_bf16(*args, window=size, **kw)
        torch.testing.assert_close(got.cpu().double().view(T - past, H, d), want[past:], rtol=3e-2, atol=3e-2)
    kernels.check_bounded_waits(torch.device("cuda", 0))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(3, 1, 16, 12, 8, True), (40, 8, 128, 128, 128, True), (5, 5, 64, 32, 24, True),
                                   (3, 1, 10, 6, 6, True), (2, 2, 8, 8, 0, True), (6, 2, 24, 16, 8, False), (2, 1, 272, 8, 16, True)])
def test_queries_and_keys_over_their_root_mean_square_after_the_rotation(sizes, dtype):
    """Biases, scaled rotation with its factor on cosine and sine, each head over its own root mean square, keys and
    values into pages out of order: the kernel with a group of lanes per head, and the general one for widths that are no
    words of four, pairs (2i, 2i+1) and wide heads.  A large eps shows where it stands; few and many tokens.  (The kernel's
    angles are float32 products: up to 300 radians here, 2e-5 of them rounding.)"""
    from garlic_inference_b200.ops import kernels
    H, G, d, dv, dims, half = sizes
    page = 16
    tol = dict(rtol=1e-5, atol=1e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    cols = H * d + G * d + G * dv
    for T in (7, 301):
        torch.manual_seed(d + T)
        src = torch.randn(T, cols + 8, device="cuda").to(dtype)[:, 8:]
        bias = torch.randn(cols, device="cuda")
        pos = torch.arange(T, dtype=torch.int32, device="cuda")
        slot = torch.ones(T, dtype=torch.int32, device="cuda")
        slot[3] = -1                                     # a padding row: nothing goes into the cache
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        f, mag = plain.turn_frequencies(dims, 300.0, tk.YARN) if dims else (None, 1.0)
        kp, vp, table = _paged(torch.zeros(T, G, d, device="cuda", dtype=dtype), torch.zeros(T, G, dv, device="cuda", dtype=dtype), page)
        q = kernels.attn_prepare(src, 0, H * d, H * d + G * d, f.float().cuda() if dims else None, dims, half, pos, slot, table,
                                 kp, vp, H, d, dtype, status, bias=bias, magnitude=mag, head_eps=0.5)
        x = src.float().cpu() + bias.cpu()

        def turned(y):
            if half or not dims:
                return plain.rotate_halves(y, torch.arange(T), dims, 300.0, tk.YARN)
            order = [*range(0, dims, 2), *range(1, dims, 2), *range(dims, d)]          # pairs (2i, 2i + 1) as halves
            out = torch.empty_like(y)
            out[..., order] = plain.rotate_halves(y[..., order], torch.arange(T), dims, 300.0, tk.YARN)
            return out

        want_q = plain.rms(turned(x[:, :H * d].reshape(T, H, d)), 0.5)
        want_k = plain.rms(turned(x[:, H * d:H * d + G * d].reshape(T, G, d)), 0.5)
        want_v = x[:, H * d + G * d:].reshape(T, G, dv).clone()
        want_k[3] = want_v[3] = 0.0
        cached = lambda pool, w: pool[table[1, :table.shape[1] - 1].long()].permute(0, 2, 1, 3).reshape(-1, G, w)[:T].float().cpu()
        torch.testing.assert_close(q.float().cpu(), want_q, **tol)
        torch.testing.assert_close(cached(kp, d), want_k, **tol)
        torch.testing.assert_close(cached(vp, dv), want_v, **tol)
        assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_results_that_join_the_stream_through_a_norm(dtype):
    """Every way a result joins (as it is, Dynamic Tanh, RMS, none pending) with every way the stream goes on (nothing,
    rounded, Dynamic Tanh, RMS), narrow, odd and wide rows, few and many of them, gathered rows, an output that is columns
    of a wider matrix, results and alphas large enough to saturate the tanh."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.ops.kernels import NormVecs
    torch.manual_seed(8)
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.5e-2, atol=1.5e-2)
    for n, dim in ((1, 7), (5, 50), (3, 192), (700, 260), (9, 2048), (2, 4100), (150, 8192), (2, 9000)):
        mk = lambda kind: NormVecs(kind, *(torch.randn(dim, device="cuda").to(torch.bfloat16) for _ in range(2 if kind == "dyt" else 1)),
                                   **({"alpha": torch.tensor([0.8], device="cuda").to(torch.bfloat16)} if kind == "dyt" else {"eps": 0.3}))
        vecs = {"dyt": mk("dyt"), "rms": mk("rms")}
        last = {"dyt": mk("dyt"), "rms": mk("rms")}

        def apply(v, z):
            if v.kind == "dyt":
                return plain.tanh_norm(z, v.alpha.double().cpu(), v.weight.double().cpu(), v.bias.double().cpu())
            return plain.rms(z, 0.3) * v.weight.double().cpu()

        for join in (None, "plain", "dyt", "rms"):
            for out in (None, "cast", "dyt", "rms"):
                res = torch.randn(n, dim, device="cuda") * 2
                delta = (torch.randn(n, dim, device="cuda") * torch.logspace(-2, 2, n, device="cuda")[:, None]).to(dtype)
                want = res.double().cpu()
                if join is not None:
                    d = delta.double().cpu()
                    want = want + (d if join == "plain" else apply(vecs[join], d))
                want_out = want if out in (None, "cast") else apply(last[out], want)
                args = (None if join is None else delta, vecs.get(join), None, dtype)
                rows = torch.tensor([n - 1, 0], dtype=torch.int32, device="cuda")
                if out is not None:
                    before = res.clone()
                    got = kernels.join_norm(*args[:2], res, dtype, last=last.get(out, "cast"), rows=rows)
                    torch.testing.assert_close(got.double().cpu(), want_out[rows.cpu().long()], **tol)
                    assert torch.equal(res, before), "gathered rows are not written back"
                    wide = torch.full((n, dim + 12), 7.0, device="cuda").to(dtype)
                    kernels.join_norm(*args[:2], res, dtype, last=last.get(out, "cast"), out=wide[:, 8:8 + dim], write_residual=False)
                    torch.testing.assert_close(wide[:, 8:8 + dim].double().cpu(), want_out, **tol)
                    assert torch.equal(res, before) and (wide[:, :8] == 7.0).all() and (wide[:, 8 + dim:] == 7.0).all()
                got = kernels.join_norm(*args[:2], res, dtype, last=last.get(out, "cast") if out else None)
                torch.testing.assert_close(res.double().cpu(), want, rtol=1e-5, atol=2e-5)
                if out is not None:
                    torch.testing.assert_close(got.double().cpu(), want_out, **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_side_gate_and_both_latents(dtype):
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(9)
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    for n, dim, layers, vocab in ((1, 1, 3, 5), (9, 24, 4, 60), (400, 36, 2, 33)):
        table = torch.randn(vocab, dim * layers, device="cuda").to(torch.bfloat16)
        tokens = torch.randint(0, vocab, (n,), dtype=torch.int32, device="cuda")
        z = (3 * torch.randn(n, dim, device="cuda")).to(dtype)
        for i in range(layers):
            got = kernels.token_side_gate(z, tokens, table, i * dim)
            want = plain.gelu_tanh(z.double().cpu()) * table.double().cpu()[tokens.cpu().long(), i * dim:(i + 1) * dim]
            torch.testing.assert_close(got.double().cpu(), want, **tol)
    for n, q_rank, rank, row, page in ((5, 40, 24, 24, 16), (70, 10, 14, 16, 16), (3, 1536, 512, 512, 64), (33, 72, 64, 64, 8)):
        src = torch.randn(n, 8 + q_rank + rank, device="cuda").to(dtype)
        qw, cw = torch.randn(q_rank, device="cuda").to(torch.bfloat16), torch.randn(rank, device="cuda").to(torch.bfloat16)
        pos, slot = torch.arange(n, dtype=torch.int32, device="cuda"), torch.ones(n, dtype=torch.int32, device="cuda")
        slot[n - 1] = -1
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        pool, _, table = _paged(torch.full((n, 1, row), 5.0, device="cuda", dtype=dtype), torch.zeros(n, 1, 2, device="cuda", dtype=dtype), page)
        got = kernels.latent_norms(src, 8, 8 + q_rank, qw, cw, 0.2, pos, slot, table, pool, status)
        x = src.double().cpu()
        torch.testing.assert_close(got.double().cpu(), plain.rms(x[:, 8:8 + q_rank], 0.2) * qw.double().cpu(), **tol)
        held = pool[table[1, :table.shape[1] - 1].long()].reshape(-1, row)[:n].double().cpu()
        torch.testing.assert_close(held[:n - 1, :rank], (plain.rms(x[:, 8 + q_rank:], 0.2) * cw.double().cpu())[:n - 1], **tol)
        assert (held[:n - 1, rank:] == 0).all() and (held[n - 1] == 5.0).all() and int(status.item()) == 0


def test_attention_over_latent_rows_in_a_window():
    """Single tokens over shared rows, and the softmax of score rows, with a row made to stand out just inside and just
    outside the window; pages out of sight are gone."""
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(11)
    for H, row, rank, page, size in ((5, 40, 40, 16, 33), (36, 64, 64, 64, 70), (16, 72, 64, 16, 1), (40, 512, 512, 64, 96)):
        T, scale = 260, 0.5
        c = (torch.randn(T, 1, row) * 0.2).bfloat16()
        far = 130
        c[far, 0, :4] = 6.0
        q = (torch.randn(T, H, row) * 0.2).bfloat16()
        q[:, :, :4] = 3.0
        seen = plain.window_mask(T, size)
        s = torch.einsum("thr,jr->htj", q.double(), c[:, 0].double()) * scale
        w = plain.softmax_sink(s, seen[None])
        want = torch.einsum("htj,jr->thr", w, c[:, 0, :rank].double())
        pool, _, table = _paged(c.cuda(), torch.zeros(T, 1, 2), page)
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        for t in (0, 31, 32, far, far + size - 1, far + size, T - 1):
            gone = _dropped(table, page, size, 0, t + 1)
            for n_splits in (1, 4, None):
                got = kernels.latent_decode(q[t:t + 1].contiguous().cuda(), pool, gone, torch.tensor([t], dtype=torch.int32, device="cuda"),
                                            torch.ones(1, dtype=torch.int32, device="cuda"), scale, None, rank, status,
                                            n_splits=n_splits, window=size)
                torch.testing.assert_close(got.cpu().double().view(H, rank), want[t], rtol=3e-2, atol=3e-2)
        assert int(status.item()) == 0
        edge = want[far + size - 1] - c[far, 0, :rank].double()
        assert float(edge.abs().max()) < 2e-2 and float((want[far + size] - c[far, 0, :rank].double()).abs().max()) > 0.5
        # rows of scores: tokens 100 .. 149 against keys from 24 on (or from the first the window needs)
        first_key = max(0, 100 - size + 1) // 8 * 8
        scores = s[:, 100:150, first_key:152].permute(1, 0, 2).reshape(50 * H, -1).float().contiguous().cuda()
        for out_dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
            got = kernels.causal_sink_softmax(scores, H, 100, 1.0, None, out_dtype, window=size, first_key=first_key)
            ref = w[:, 100:150, first_key:152].permute(1, 0, 2).reshape(50 * H, -1)
            torch.testing.assert_close(got.double().cpu(), ref, rtol=tol, atol=tol)


def test_biased_router_and_an_addend_with_a_gate():
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(13)
    for n, E, top in ((45, 12, 5), (7, 6, 6), (300, 64, 8), (5, 1, 1), (9, 40, 2)):
        z = torch.randn(n, E + 1, device="cuda") * 2
        b = torch.randn(E, device="cuda") * 3
        idx, wt = kernels.router_topk(z[:, :E], top, b)
        ri, rw = plain.route(z[:, :E].cpu(), {"router": torch.eye(E), "router.b": b.cpu()}, {"experts": E, "top": top})
        assert torch.equal(idx.cpu().long(), ri)
        torch.testing.assert_close(wt.cpu(), rw, rtol=1e-5, atol=1e-7)
        if 1 < top < E:
            assert not torch.equal(idx, kernels.router_topk(z[:, :E], top)[0]), "the bias chooses"
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
            buf, add = torch.randn(n * top, 72, device="cuda").to(dtype), torch.randn(n, 72, device="cuda").to(dtype)
            got = kernels.moe_combine(buf, None, wt, add, z[:, E:])
            want = (buf.view(n, top, 72).double() * wt[:, :, None].double()).sum(1) + torch.sigmoid(z[:, E:].double()) * add.double()
            torch.testing.assert_close(got.double(), want, rtol=tol, atol=tol)
