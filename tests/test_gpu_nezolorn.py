"""Nezolorn through the engine against the plain implementation: each mechanism alone, prompts against token-by-token
decoding, portions, batches, slots, pages and states used again, keys just inside and just outside every window and
block, far keys, the first tokens, long decoding, generation, the two programs, and the kernels alone."""
import math

import numpy as np
import pytest
import torch

import plain_nezolorn as plain
import tiny
import tiny_nezolorn as tk

pytestmark = pytest.mark.gpu

_DIRS, _MODELS = {}, {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    def get(name):
        if name not in _DIRS:
            _DIRS[name] = tk.write_model(name, tmp_path_factory.mktemp(f"nezolorn_{name}"))
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
@pytest.mark.parametrize("name", ["window", "blocks", "memory", "delta", "dense", "mix", "tc", "odd", "ones"])
def test_prompts_decoding_portions_and_batches_agree_with_the_plain_model(name, dtype, model, folder):
    """Every way of cutting the same requests gives the plain logits: whole prompts; all but 40 tokens, then one
    at a time; portions of 2, 7, 33 and 3 tokens; portions with all requests in one batch; unequal requests that
    start together and decode together.  The cache has room for one batch only, so slots, pages, block rows, last
    tokens and state rows are given back and used again by later requests."""
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
        tk.judge(got, want, own, dtype, f"{name} {dtype} {what}")
    cache = m.engine.cache
    assert cache.slots.n_free == 4, "every slot came back"
    assert all(g.host.pool.n_free == g.host.pool.n_pages for g in cache.groups), "every page came back"


def test_tensor_core_kernels_on_pages_of_64(model, folder):
    """The same on pages of 64 tokens, where prompts of the layers with heads of 128 run the tcgen05 kernel and the
    others the mma.sync one, with the block rows inside them."""
    m = model("tc", "bfloat16", max_tokens=2048, page_size=64, max_slots=4)
    reqs = _requests("tc", [200, 3, 129, 64], seed=15)
    want, own = tk.plain_pair(folder("tc"), reqs)
    for steps in (tiny.trace_whole(reqs), tiny.trace_tail_by_one(reqs, tail=70), tk.trace_portions(reqs, [65, 2, 30]),
                  tiny.trace_batched(reqs, [list(reqs)], prompt_frac=0.5)):
        got = tiny.run_trace_in_process(m, steps)
        tiny.assert_covers(got, reqs)
        tk.judge(got, want, own, "bfloat16", "tc on pages of 64")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_of_a_thousand_tokens_through_the_trace_program(dtype, folder, tmp_path):
    """Requests of 1,100, 425, 97 and 1 tokens through bin/trace_run on its default pages of 64: whole, and started
    together with their last 40 % decoded together.  Hundreds of block rows, pages that left the window, states carried a
    thousand tokens."""
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
        tk.judge(part, want, own, dtype, f"long {dtype} {what}")


def test_float32_logits_do_not_depend_on_the_cut_or_the_batch(model):
    """The same position gives the same bits whole, in portions, decoded, alone or in a batch: attention in the
    exact-order kernel, block rows summed in one order whoever makes them, both recurrences walked token by token."""
    for name in ("window", "blocks", "memory", "delta", "mix"):
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
    """300 tokens decoded one at a time after a prompt of 5, two requests together, through the recorded decode
    step: pages taken and given back one by one, a block row made at every block's last token, states carried 300
    times."""
    m = model(name, dtype, max_tokens=1024, page_size=16)
    reqs = _requests(name, [305, 280], seed=9)
    want, own = tk.plain_pair(folder(name), reqs)
    steps = tiny.trace_batched(reqs, [["r0", "r1"]], prompt_frac=5 / 305)
    got = tiny.run_trace_in_process(m, steps)
    tiny.assert_covers(got, reqs)
    tk.judge(got, want, own, dtype, f"long decoding {name} {dtype}")
    assert m.engine.graphs is not None and 2 in m.engine.graphs._graphs, "decode steps ran from a recorded graph"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_a_dozen_requests_decode_together(name, dtype, model, folder):
    """Twelve unequal requests start together and decode together through a recorded step of 16 rows (four of them
    padding): the kernels see padding rows (slot -1: no state, no page, no last token), and requests leave one after
    the other."""
    m = model(name, dtype, max_tokens=2048, page_size=16, max_slots=12)
    reqs = _requests(name, [31 + 3 * i for i in range(12)], seed=21)
    want, own = tk.plain_pair(folder(name), reqs)
    got = tiny.run_trace_in_process(m, tiny.trace_batched(reqs, [list(reqs)], prompt_frac=0.5))
    tiny.assert_covers(got, reqs)
    tk.judge(got, want, own, dtype, f"twelve together {name} {dtype}")
    assert m.engine.graphs is not None and 16 in m.engine.graphs._graphs


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(dtype, model, folder):
    """The scheduler's own loop: the tokens it samples stay on the device, so the pair embedding's last token comes
    from there too."""
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


def test_a_folder_without_the_thin_rank_in_its_config(folder, tmp_path):
    """The inner size of the decay's thin products is no key of the design: a folder whose config.json lacks this
    library's own key gets it from the stored tensor's shape."""
    import json
    from garlic_inference_b200 import AutoModel
    src = folder("delta")
    dst = tmp_path / "bare"
    dst.mkdir()
    cfg = json.loads((src / "config.json").read_text())
    assert cfg["layers"][0]["mixer"].pop("rank") == 6
    (dst / "config.json").write_text(json.dumps(cfg))
    (dst / "model.safetensors").symlink_to(src / "model.safetensors")
    m = AutoModel.from_pretrained(dst, device=0, dtype="float32", max_tokens=256, page_size=16)
    reqs = _requests("delta", [60], seed=2)
    want, own = tk.plain_pair(dst, reqs)
    tk.judge(tiny.run_trace_in_process(m, tiny.trace_whole(reqs)), want, own, "float32", "rank from the tensor")


# ---- kernels alone -----------------------------------------------------------------------------
def _paged(keys, values, page, spare=3, slots=2):
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
    table = torch.full((slots, n_pages + 1), -1, dtype=torch.int32, device="cuda")
    table[1, :n_pages] = order.to(torch.int32)
    return k_pool, v_pool, table


def _empty_means(T, G, d, dv, block, page, dtype, spare=2):
    """Block rows for a sequence of T positions in slot 1, on pages out of order, none filled yet."""
    from garlic_inference_b200.cache import MeansView, mean_page_rows
    rows = mean_page_rows(page, block)
    n_pages = max(1, -(-(T // block) // rows))
    order = torch.randperm(n_pages + spare)[:n_pages]
    table = torch.full((2, n_pages + 1), -1, dtype=torch.int32, device="cuda")
    table[1, :n_pages] = order.to(torch.int32)
    pool = lambda w: torch.zeros(n_pages + spare, G, rows, w, dtype=dtype, device="cuda")
    return MeansView(pool(d), pool(dv), table, block), order, rows


def _block_rows(means, order, rows, n, key=True):
    """Rows 0 .. n - 1 of the sequence as a list of [G, width] float32 on the CPU."""
    pool = means.k_pool if key else means.v_pool
    return [pool[order[b // rows], :, b % rows].float().cpu() for b in range(n)]


def _run_arrays(T):
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    slot = torch.ones(T, dtype=torch.int32, device="cuda")
    return pos, slot, torch.zeros(1, dtype=torch.int32, device="cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,H,G,page,size,block", [(64, 6, 2, 16, 40, 8), (128, 4, 2, 64, 70, 5), (48, 4, 4, 64, 33, 24),
                                                   (16, 34, 2, 16, 17, 1), (12, 3, 1, 16, 5, 9), (128, 2, 1, 128, 1, 2)])
def test_attention_over_a_window_and_block_rows_with_keys_that_stand_out(d, H, G, page, size, block, dtype):
    """One token's key is made so large that it takes nearly all the weight where it is seen alone, and its value has
    numbers of its own.  Every query is compared, so the token is asked for just inside and just outside the window, in
    the gap where its block is not yet behind the window, and as a block row from the block's own edge on (where the
    mean of its block's keys still stands out).  Tokens: the first, page borders, a block's first and last, the middle.
    Exact-order kernel, both prompt kernels, the split-KV decode kernel."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.parts import StepShape
    from garlic_inference_b200.parts.attention import query_runs
    torch.manual_seed(4)
    T, scale = 330, 0.3
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=4e-2)
    pos, slot, status = _run_arrays(T)
    for far in (0, page - 1, page, block * (40 // block), block * (40 // block) + block - 1, 150):
        k = torch.randn(T, G, d) * 0.2
        v = torch.randn(T, G, d)
        q = torch.randn(T, H, d) * 0.2
        k[far, :, :4] = 9.0 * block
        v[far] += 20.0
        q[:, :, :4] = 0.7
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        k_pool, v_pool, table = _paged(k.cuda(), v.cuda(), page)
        means, order, rows = _empty_means(T, G, d, d, block, page, dtype)
        kernels.pool_blocks(k_pool, v_pool, table, pos, slot, status, means)
        for key, src in ((True, k), (False, v)):
            got = _block_rows(means, order, rows, T // block, key)
            for b in range(T // block):
                torch.testing.assert_close(got[b], src[b * block:(b + 1) * block].float().mean(0), rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-5)
        want = plain.pooled_attention_heads(q.double(), k.double(), v.double(), size, block, scale)
        if dtype == torch.bfloat16:          # the rows as the cache holds them: rounded means
            # (their own rounding is the cache's, not the kernel's, so the oracle is given the same rows)
            want = _attention_with_rows(q, k, v, _block_rows(means, order, rows, T // block), _block_rows(means, order, rows, T // block, False), size, block, scale)
        shift = lambda i: float((want[i] - plain.pooled_attention_heads(q[i:i + 1].double(), v[:1].double() * 0, v[:1].double() * 0, 1, 0, 1.0)).mean())
        if far + size < T:
            assert shift(far + size - 1) > 10.0, "just inside the window the key takes nearly all the weight"
            end = (far // block + 1) * block - 1 + size
            if end > far + size:
                assert shift(far + size) < 5.0, "in the gap between window and block it is not seen"
            if end < T and (far // block + 1) * block <= T:
                assert shift(end) > 0.5 * 20.0 / block - 1.0, "from the block's edge on its mean is seen"
        got = kernels.attention_masked(q.cuda(), k_pool, v_pool, table, pos, slot, scale, status, window=size, out_float32=True, means=means)
        torch.testing.assert_close(got.cpu().double().view(T, H, d), want, **tol)
        if dtype == torch.bfloat16 and kernels.mma_attention_takes(dtype, d):
            runs = torch.from_numpy(query_runs(StepShape([1], [0], [T], [0], False), 64)).cuda()
            got = kernels.attention_prefill_masked_bf16(q.cuda(), k_pool, v_pool, table, runs, scale, window=size, rows_covered=True, means=means)
            torch.testing.assert_close(got.cpu().double().view(T, H, d), want, **tol)
            # the last rows as a step that continues a sequence from the cache
            runs = torch.from_numpy(query_runs(StepShape([1], [0], [T - 201], [201], False), 64)).cuda()
            got = kernels.attention_prefill_masked_bf16(q[201:].contiguous().cuda(), k_pool, v_pool, table, runs, scale, window=size, rows_covered=True, means=means)
            torch.testing.assert_close(got.cpu().double().view(T - 201, H, d), want[201:], **tol)
            if H // G <= 16:
                some = sorted({0, 1, size - 1, size, min(T - 1, far + size - 1), min(T - 1, far + size), min(T - 1, (far // block + 1) * block - 1 + size),
                               min(T - 1, (far // block + 1) * block - 2 + size), 257, T - 1})
                idx = torch.tensor(some, device="cuda")
                for n_splits in (1, 3, 16):
                    one = kernels.attention_decode_masked_bf16(q.cuda()[idx].contiguous(), k_pool, v_pool, table, pos[idx].contiguous(),
                                                               slot[idx].contiguous(), scale, window=size, n_splits=n_splits, means=means)
                    torch.testing.assert_close(one.cpu().double().view(len(some), H, d), want[some], **tol)
            if kernels.tcgen05_attention_takes(dtype, d, page):
                runs = torch.from_numpy(query_runs(StepShape([1], [0], [T], [0], False), 128)).cuda()
                got = kernels.attention_prefill_tcgen05(q.cuda(), k_pool, v_pool, table, runs, scale, size, rows_covered=True, means=means)
                torch.testing.assert_close(got.cpu().double().view(T, H, d), want, **tol)
                runs = torch.from_numpy(query_runs(StepShape([1], [0], [T - 201], [201], False), 128)).cuda()
                got = kernels.attention_prefill_tcgen05(q[201:].contiguous().cuda(), k_pool, v_pool, table, runs, scale, size, rows_covered=True, means=means)
                torch.testing.assert_close(got.cpu().double().view(T - 201, H, d), want[201:], **tol)
    assert int(status.item()) == 0
    kernels.check_bounded_waits(torch.device("cuda", 0))


def _attention_with_rows(q, k, v, k_rows, v_rows, size, block, scale):
    """The plain attention with block rows given: o[t, h] over the window's keys and the rows behind it."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    K = torch.cat([k.double(), torch.stack(k_rows).double()]) if k_rows else k.double()
    V = torch.cat([v.double(), torch.stack(v_rows).double()]) if v_rows else v.double()
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = torch.cat([(j <= i) & (i - j < size), (torch.arange(len(k_rows))[None, :] + 1) * block - 1 <= i - size], 1)
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for h in range(H):
        s = (q[:, h].double() @ K[:, h // rep].T) * scale
        out[:, h] = torch.softmax(torch.where(seen, s, torch.full_like(s, -math.inf)), -1) @ V[:, h // rep]
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_cache_rows_values_before_the_rotation_and_block_rows_one_token_at_a_time(dtype):
    """The kernel between projections and attention with values taken from the keys: rotated keys and unrotated values in
    the pages; and a step per token leaves the same block rows, bit for bit, as one step with all tokens and the
    kernel that fills the rows afterwards.  Two sequences and a padding row in every step."""
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(6)
    H, G, d, page, block, T = 4, 2, 12, 16, 5, 43
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    src = torch.randn(T, (H + G) * d + 3, device="cuda").to(dtype)[:, 3:]
    pos, slot, status = _run_arrays(T)
    freq = torch.tensor([plain.rotary_frequency(i, 8, 50.0, tk.BANDS) for i in range(4)], dtype=torch.float32, device="cuda")
    blank = lambda: _paged(torch.zeros(T, G, d, device="cuda", dtype=dtype), torch.zeros(T, G, d, device="cuda", dtype=dtype), page)
    k_pool, v_pool, table = blank()
    means, order, rows = _empty_means(T, G, d, d, block, page, dtype)
    q = kernels.attn_prepare(src, 0, H * d, H * d, freq, 8, True, pos, slot, table, k_pool, v_pool, H, d, dtype, status)
    kernels.pool_blocks(k_pool, v_pool, table, pos, slot, status, means)
    x = src.float().cpu()
    want_q = plain.rotate_halves(x[:, :H * d].reshape(T, H, d), torch.arange(T), 8, 50.0, tk.BANDS)
    want_k = plain.rotate_halves(x[:, H * d:].reshape(T, G, d), torch.arange(T), 8, 50.0, tk.BANDS)
    cached = lambda pool: pool[table[1, :-(-T // page)].long()].permute(0, 2, 1, 3).reshape(-1, G, d)[:T].float().cpu()
    torch.testing.assert_close(q.float().cpu(), want_q, **tol)
    torch.testing.assert_close(cached(k_pool), want_k, **tol)
    torch.testing.assert_close(cached(v_pool), x[:, H * d:].reshape(T, G, d), rtol=0, atol=0)
    for key, src_rows in ((True, cached(k_pool)), (False, cached(v_pool))):
        for b, row in enumerate(_block_rows(means, order, rows, T // block, key)):
            torch.testing.assert_close(row, src_rows[b * block:(b + 1) * block].mean(0), rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-5)
    # token by token, in slot 1 of other pages, beside slot 0 (whose tables stay unmapped: it writes nothing) and padding
    k2, v2, table2 = blank()
    means2, order2, rows2 = _empty_means(T, G, d, d, block, page, dtype)
    for t in range(T):
        step = torch.cat([src[t:t + 1], src[:1]])
        p = torch.tensor([t, 4], dtype=torch.int32, device="cuda")
        s = torch.tensor([1, -1], dtype=torch.int32, device="cuda")
        kernels.attn_prepare(step, 0, H * d, H * d, freq, 8, True, p, s, table2, k2, v2, H, d, dtype, status, means=means2)
    for key in (True, False):
        for a, b in zip(_block_rows(means, order, rows, T // block, key), _block_rows(means2, order2, rows2, T // block, key)):
            assert torch.equal(a, b)
    untouched = [p for p in range(means2.k_pool.shape[0]) if p not in order2.tolist()]
    assert float(means2.k_pool[untouched].abs().max()) == 0.0 and int(status.item()) == 0


def _walk(T, cuts, others, run):
    """Feed `T` rows in steps of the given sizes, each beside 3 rows of another sequence (slot 0) and a padding row;
    `run(rows, slots, spans)` gives the step's outputs.  Rows of the walked sequence, in slot 2."""
    got, at = [], 0
    for n in cuts:
        slots = torch.tensor([0] * 3 + [2] * n + [-1], dtype=torch.int32, device="cuda")
        spans = torch.tensor([[2, 3, n], [0, 0, 3], [-1, 3 + n, 1]], dtype=torch.int32, device="cuda")
        out = run(lambda x, o, pad: torch.cat([o, x[at:at + n], pad]), slots, spans)
        got.append(out[3:3 + n].cpu())
        assert float(out[-1].abs().max()) == 0.0, "a padding row gives zeros"
        at += n
    assert at == T
    return torch.cat(got)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,dv", [(3, 12, 20), (2, 32, 64), (1, 64, 33), (2, 128, 96), (1, 200, 40), (2, 7, 5)])
def test_matrix_memory_scan(H, d, dv, dtype):
    """Against the plain loop, a prompt cut into steps of 1, 2, 9 and the rest with the state in a slot's row, beside a
    second sequence and a padding row.  The logits are large, so the input gate overtakes the running maximum now and
    then (the state is all but replaced) and the forget gate empties it; some keys are zero (the floor of the
    denominator decides)."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.parts.matrix_memory import matrix_memory_floats
    torch.manual_seed(8)
    T, cap = 75, 7.0
    x = torch.randn(T, H * (2 * d + dv)).to(dtype)
    x[20:24, H * d:2 * H * d] = 0.0
    gates = torch.randn(T, 2 * H) * 4.0
    gates[40] = torch.tensor([30.0] * H + [-30.0] * H)
    ib, fb = torch.randn(H), torch.randn(H) + 2.0
    q, k, v = x.double()[:, :H * d].reshape(T, H, d) * d ** -0.5, x.double()[:, H * d:2 * H * d].reshape(T, H, d), x.double()[:, 2 * H * d:].reshape(T, H, dv)
    i = cap * torch.tanh((gates[:, :H].double() + ib.double()) / cap)
    f = plain.logsigmoid(cap * torch.tanh((gates[:, H:].double() + fb.double()) / cap))
    want = torch.stack([plain.matrix_memory_scan(q[:, h], k[:, h], v[:, h], i[:, h], f[:, h]) for h in range(H)], 1).reshape(T, H * dv)
    dx, dg, dib, dfb = x.cuda(), gates.cuda(), ib.cuda(), fb.cuda()
    other, og = torch.randn(3, x.shape[1], device="cuda").to(dtype), torch.randn(3, 2 * H, device="cuda")

    def run_with(state):
        return lambda rows, slots, spans: kernels.matrix_memory_scan(
            rows(dx, other, torch.ones_like(other[:1])), (0, H * d, 2 * H * d), rows(dg, og, og[:1]), (0, H), dib, dfb, cap, state, spans,
            slots, H, d, dv)
    results = []
    for cuts in ([1, 2, 9, T - 12], [T], [1] * T, [33, 32, T - 65]):
        state = torch.zeros(4, H * matrix_memory_floats(d, dv), device="cuda")
        results.append(_walk(T, cuts, other, run_with(state)))
        assert float(state[3].abs().max()) == 0.0 and float(state[1].abs().max()) == 0.0, "no other slot's row was touched"
    scale = want.abs().amax(1, keepdim=True).clamp(min=1e-3)
    assert float(((results[0].double() - want) / scale).abs().max()) < 2e-4
    for r in results[1:]:
        assert torch.equal(r, results[0]), "the bits do not depend on the cut"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d", [(3, 20), (2, 32), (1, 64), (2, 128), (1, 200), (2, 7)])
def test_general_delta_scan(H, d, dtype):
    """Against the plain loop in the same cuts; decays from all but forgetting to all but keeping, removal rates from 0
    to 1, a key of zeros (no direction to remove)."""
    from garlic_inference_b200.ops import kernels
    from garlic_inference_b200.parts.linear_attention import scan_state_floats
    torch.manual_seed(9)
    T, C = 70, H * d
    x = (torch.randn(T, 3 * C) * 0.5).to(dtype)
    x[30, C:2 * C] = 0.0
    zw, za = torch.randn(T, C) * 4, torch.randn(T, C) * 3
    w0, a0 = torch.randn(C), torch.randn(C)
    heads = lambda z: z.double().reshape(T, H, d)
    w = torch.exp(-math.exp(-0.5) * torch.sigmoid(heads(zw + w0)))
    a = torch.sigmoid(heads(za + a0))
    r, k, v = heads(x[:, :C]), heads(x[:, C:2 * C]), heads(x[:, 2 * C:])
    want = torch.stack([plain.general_delta_scan(r[:, h], k[:, h], v[:, h], w[:, h], a[:, h]) for h in range(H)], 1).reshape(T, C)
    dx, dw, da, dw0, da0 = x.cuda(), zw.cuda(), za.cuda(), w0.cuda(), a0.cuda()
    other, og = torch.randn(3, 3 * C, device="cuda").to(dtype), torch.randn(3, C, device="cuda")

    def run_with(state):
        def run(rows, slots, spans):
            zw, za = rows(dw, og, og[:1]), rows(da, og, og[:1])
            ready = len(slots) % 2 == 0              # now and then the rates are made beforehand, as steps with many tokens do
            if ready:
                kernels.general_delta_rates(zw, dw0, za, da0, dtype)
            return kernels.general_delta_scan(rows(dx, other, torch.ones_like(other[:1])), (0, C, 2 * C), zw, dw0, za, da0, state,
                                              spans, slots, H, d, d, 1e-6, ready=ready)
        return run
    results = []
    for cuts in ([1, 2, 9, T - 12], [T], [1] * T, [33, 32, T - 65]):
        state = torch.zeros(4, H * scan_state_floats(d, d), device="cuda")
        results.append(_walk(T, cuts, other, run_with(state)))
        assert float(state[3].abs().max()) == 0.0 and float(state[1].abs().max()) == 0.0, "no other slot's row was touched"
    assert float((results[0].double() - want).abs().max() / want.abs().max()) < 2e-5
    for r2 in results[1:]:
        assert torch.equal(r2, results[0]), "the bits do not depend on the cut"


def test_pair_embedding_reads_the_token_before_across_steps_and_slots():
    """Rows of two sequences and padding in every step; the token before a step's first row comes from the slot's state,
    position 0 reads the last row whatever the state holds, multipliers beyond 32 bits do not overflow."""
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(3)
    vocab, hid, buckets, mp, mc, scale = 5000, 40, 997, 2_000_003, 1_000_033, 1.5
    for dtype in (torch.float32, torch.bfloat16):
        table, pairs = torch.randn(vocab, hid, device="cuda").to(dtype), torch.randn(buckets + 1, hid, device="cuda").to(dtype)
        seqs = {0: torch.randint(vocab, (19,)).tolist(), 3: torch.randint(vocab, (19,)).tolist()}
        want = {s: (table.float().cpu()[ids] * scale + pairs.float().cpu()[plain.bigram_rows(ids, buckets, mp, mc)]) for s, ids in seqs.items()}
        state = torch.full((6, 1), 77, dtype=torch.int32, device="cuda")      # what an earlier sequence left
        at = 0
        for n in (1, 1, 4, 2, 1, 10):
            ids, pos, slot = [], [], []
            for s in seqs:
                ids += seqs[s][at:at + n]
                pos += range(at, at + n)
                slot += [s] * n
            t = lambda xs: torch.tensor(xs, dtype=torch.int32, device="cuda")
            out = kernels.embedding_pairs(t(ids + [9]), table, pairs, mp, mc, t(pos + [0]), t(slot + [-1]), state, renew=n == 1, scale=scale)
            got = out.cpu()
            for k, s in enumerate(seqs):
                torch.testing.assert_close(got[k * n:(k + 1) * n], want[s][at:at + n], rtol=1e-6, atol=1e-6)
                assert int(state[s]) == seqs[s][at + n - 1]
            at += n
        assert state[[1, 2, 4, 5]].flatten().tolist() == [77] * 4, "no other slot's token was touched"


def test_layer_norm_adds_a_scaled_result():
    from garlic_inference_b200.ops import kernels
    torch.manual_seed(9)
    for dim in (100, 50, 2048, 4096):
        res, d1 = torch.randn(37, dim, device="cuda") * 3, torch.randn(37, dim, device="cuda")
        w, f = torch.randn(dim, device="cuda"), torch.randn(dim, device="cuda")
        for factor in (f, torch.full((dim,), 0.3, device="cuda"), f.bfloat16()):
            keep = res.clone()
            out = kernels.add_layernorm(d1, keep, w, None, 1e-5, torch.float32, delta_scale=factor)
            s = res.cpu() + d1.cpu() * factor.float().cpu()
            torch.testing.assert_close(keep.cpu(), s, rtol=1e-6, atol=1e-6)
            torch.testing.assert_close(out.cpu(), plain.layer_norm(s, w.cpu(), 1e-5), rtol=1e-5, atol=1e-5)
            rows = torch.tensor([36, 0, 5], dtype=torch.int32, device="cuda")
            out = kernels.add_layernorm(d1, res.clone(), w, None, 1e-5, torch.float32, rows=rows, delta_scale=factor)
            torch.testing.assert_close(out.cpu(), plain.layer_norm(s, w.cpu(), 1e-5)[rows.cpu().long()], rtol=1e-5, atol=1e-5)
    z = torch.randn(9, 30, device="cuda")
    torch.testing.assert_close(kernels.tanh_rows(z[:, 5:17], torch.bfloat16).float().cpu(), torch.tanh(z[:, 5:17].cpu()), rtol=1e-2, atol=1e-3)
