"""Nezolorn on the CPU: its configuration, plan, tensors and cache, and the plain implementation against closed forms."""
import json
import math

import pytest
import torch

import plain_nezolorn as plain
import tiny_nezolorn as tk


def test_registry_reads_the_architecture_string_and_round_trips(tmp_path):
    from garlic_inference_b200 import load_config
    from garlic_inference_b200.config import NezolornConfig, known_architectures
    assert "Nezolorn" in known_architectures()
    (tmp_path / "config.json").write_text(json.dumps(tk.config_dict("mix")))
    cfg = load_config(tmp_path)
    assert type(cfg) is NezolornConfig and cfg.width == 96 and cfg.vocab == 411 and cfg.embedding_scale == 9.0
    assert cfg.residual_mult == 0.35 and cfg.bigram == {"buckets": 301, "mul_prev": 1009, "mul_cur": 65537}
    for name in tk.TINY:
        c = tk.make_config(name)
        assert NezolornConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    assert tk.make_config("tc").to_dict() == tk.config_dict("tc")


def test_plan_and_tensors():
    from garlic_inference_b200.engine.model import wanted_tensors
    plan = tk.make_config("mix").plan()
    assert [(e.layer, e.cache) for e in plan.schedule] == [(i, i) for i in range(5)]
    assert all(layer.block == "pre_norm_scaled_residual" for layer in plan.layers)
    assert all(g.kind == "constant_scale" and g.params["value"] == 0.35 for layer in plan.layers for g in layer.gates.values())
    assert list(plan.layers[2].norms) == ["input"] and plan.layers[2].feed_forward is None and list(plan.layers[2].gates) == ["mixer"]
    names = wanted_tensors(plan)
    shape = lambda n: tuple(names[n].shape)
    assert shape("embed") == (411, 96) and shape("bigram") == (302, 96) and shape("head") == (411, 96)
    assert shape("l1.mix.left.q") == (96, 96) and shape("l1.mix.left.k") == (32, 96) and shape("l1.mix.left.o") == (96, 96)
    assert "l1.mix.left.v" not in names, "the values are the keys"
    assert shape("l1.mix.right.q") == (80, 96) and shape("l1.mix.right.v") == (200, 96) and shape("l1.mix.right.g") == (200, 96)
    assert shape("l1.mix.right.i") == (5, 96) and shape("l1.mix.right.f.b") == (5,) and shape("l1.mix.right.norm") == (200,)
    assert shape("l0.mix.a") == (96, 96) and shape("l0.mix.a.b") == (96,) and shape("l0.mix.w1") == (10, 96)
    assert shape("l0.mix.w2") == (96, 10) and shape("l0.mix.w0") == (96,) and shape("l0.mix.norm") == (96,)
    assert "l3.norm2" not in names and "l3.norm1" in names and not any(n.startswith("l3.mlp.") for n in names)
    assert shape("l0.mlp.gate") == (128, 96) and shape("final.norm") == (96,) and "l0.norm1.b" not in names
    left = plan.layers[1].mixer.params["left"]["params"]
    assert left["mask"] == {"kind": "window", "size": 24, "pool": 6} and left["values_from_keys"] is True
    assert plan.layers[1].mixer.params["right"]["params"]["gate_cap"] == 9.0
    assert plan.layers[1].mixer.params["left_scale"] == 1.2 and plan.layers[1].mixer.params["right_scale"] == 0.9
    assert len(plan.positions) == 3
    rot = next(p for k, p in plan.positions.items() if "300.0" in k).params
    assert rot["layout"] == "half" and rot["bands"] == {"factor": 8.0, "low": 0.5, "high": 4.0, "original": 96.0} and rot["tables"] is False
    assert "bands" not in next(p for k, p in plan.positions.items() if "5000.0" in k).params
    assert plan.embedding.params["pairs"]["mul_cur"] == 65537 and plan.embedding.weights["pairs"] == "bigram"


def test_the_thin_rank_comes_from_the_tensor():
    from garlic_inference_b200.config import NezolornConfig
    cfg = tk.config_dict("delta")
    del cfg["layers"][0]["mixer"]["rank"]
    bare = NezolornConfig.from_dict(cfg)
    assert bare.plan().layers[0].mixer.params["decay_rank"] == 8                       # this library's own default
    sized = bare.with_shapes({"l0.mix.w1": (6, 48), "l0.mix.w2": (60, 6)})
    assert sized.plan().layers[0].mixer.params["decay_rank"] == 6


def test_refusals_and_warnings():
    from garlic_inference_b200.config import ConfigError, NezolornConfig

    def refused(name, change, match):
        bad = tk.config_dict(name)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            NezolornConfig.from_dict(bad)

    refused("delta", lambda c: c["layers"][0].update(type="convolution"), "convolution")
    refused("dense", lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe")
    refused("window", lambda c: c["layers"][0]["mixer"]["left"].update(vdim=16), "vdim 16")
    refused("window", lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "no multiple")
    refused("window", lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(pool=0), "pool")
    refused("window", lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims 7")
    refused("window", lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(low=9.0), "low")
    refused("memory", lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0.0), "gate_cap")
    refused("memory", lambda c: c.pop("residual_mult"), "residual_mult")
    refused("memory", lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets")
    odd = tk.config_dict("memory")
    odd["layers"][0]["mixer"]["right"]["conv"] = 4
    with pytest.warns(UserWarning, match="conv"):
        NezolornConfig.from_dict(odd)


def test_frequencies_scaled_by_wavelength():
    from garlic_inference_b200.parts import RotaryPositions
    for dims, base, sc in ((16, 300.0, dict(tk.BANDS)), (48, 7000.0, dict(tk.BANDS, original=1000)), (6, 100.0, dict(tk.BANDS, factor=2.5, low=0.25, high=8.0)),
                           (32, 10.0, dict(tk.BANDS, low=2.0, high=2.0))):
        f, magnitude = RotaryPositions.frequencies(dims, base, bands=sc)
        want = [plain.rotary_frequency(i, dims, base, sc) for i in range(dims // 2)]
        torch.testing.assert_close(f, torch.tensor(want, dtype=torch.float64), rtol=1e-14, atol=0.0)
        assert magnitude == 1.0
    plain_f = [7000.0 ** (-2 * i / 48) for i in range(24)]
    f = RotaryPositions.frequencies(48, 7000.0, bands=dict(tk.BANDS, original=1000))[0].tolist()
    kept = [i for i in range(24) if f[i] == plain_f[i]]
    slow = [i for i in range(24) if abs(f[i] * 4 - plain_f[i]) < 1e-12]
    assert kept and slow and len(kept) + len(slow) < 24 and max(kept) < min(slow), "some kept, some blended, some slowed"


def test_cache_of_a_window_with_block_rows():
    """The tokens' pages come back behind the window; the block rows get a page when a block is whole and keep it for the
    sequence's life; everything comes back with the slot; what does not fit is refused before anything changed."""
    from garlic_inference_b200.cache import CacheError, EntryRequirement, KVRequirement, PagedCache, StateRequirement, mean_page_rows
    assert [mean_page_rows(64, p) for p in (1, 2, 5, 8, 100)] == [64, 32, 16, 8, 8]
    req = EntryRequirement(KVRequirement(2, 8, 20, mean_block=4), StateRequirement((8,)))
    c = PagedCache([req, StateRequirement((1,), torch.int32)], max_tokens=256, max_positions=4096, dtype=torch.float32,
                   device="cpu", page_size=16, max_slots=3)
    view = c.view(0)
    tokens, means = c.groups
    assert view.kv.window == 20 and view.kv.means.block == 4 and view.kv.means.k_pool.shape[1:] == (2, 8, 8)
    assert view.kv.means.block_table is means.table and means.stride == 4 and c.view(1).state.dtype == torch.int32
    s = c.alloc_slot()
    free = means.host.pool.n_free
    for n, pages in ((3, 0), (1, 1), (27, 1), (1, 1), (3, 1), (1, 2), (64, 4)):      # a page of 8 rows covers 32 positions
        c.prepare([s], [n]), c.commit([s], [n])
        assert len(means.host.pages_of(s)) == pages and means.host.pool.n_free == free - pages
    assert c.length(s) == 100 and len(tokens.host.pages_of(s)) == 2, "only the pages of the last 20 positions are held"
    # an entry of another slot that would not fit is refused and nothing is taken
    t = c.alloc_slot()
    with pytest.raises(CacheError, match="full"):
        c.prepare([t], [256])
    assert not means.host.pages_of(t) and not tokens.host.pages_of(t)
    c.free_slot(s), c.free_slot(t)
    assert means.host.pool.n_free == means.host.pool.n_pages and tokens.host.pool.n_free == tokens.host.pool.n_pages
    # blocks of one position keep their rows too, while the window's pages come back
    c = PagedCache([KVRequirement(1, 8, 5, mean_block=1)], max_tokens=128, max_positions=256, dtype=torch.float32, device="cpu", page_size=16)
    s = c.alloc_slot()
    c.prepare([s], [100]), c.commit([s], [100])
    assert [len(g.host.pages_of(s)) for g in c.groups] == [1, 7]
    # as many sequences as there are units, each of one unit, always find their block rows' pages
    c = PagedCache([KVRequirement(1, 8, 9, mean_block=3)], max_tokens=640, max_positions=4096, dtype=torch.float32, device="cpu", page_size=16)
    slots = [c.alloc_slot() for _ in range(10)]
    c.prepare(slots, [64] * 10)
    with pytest.raises(CacheError, match="not whole"):
        PagedCache([KVRequirement(1, 8, 5, mean_block=9)], max_tokens=64, max_positions=64, dtype=torch.float32, device="cpu")


def test_plain_functions_against_closed_forms():
    torch.manual_seed(0)
    # layer norm: mean and variance of the squared deviations
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=torch.float64)
    torch.testing.assert_close(plain.layer_norm(x, torch.ones(4).double(), 0.0), (x - 4) / math.sqrt(5))
    # the pair table's row: by both tokens, the last row first
    assert plain.bigram_rows([5, 2, 9], 10, 3, 4) == [10, (15 + 8) % 10, (6 + 36) % 10]
    # rotation of halves: a pair at position p turns by p f, the rest passes
    y = torch.tensor([[[1.0, 0.0, 0.0, 1.0, 5.0]]]).repeat(3, 1, 1)
    r = plain.rotate_halves(y, torch.arange(3), 4, 100.0)
    a0, a1 = 2.0, 2 * 100.0 ** -0.5
    torch.testing.assert_close(r[2, 0], torch.tensor([math.cos(a0), -math.sin(a1), math.sin(a0), math.cos(a1), 5.0]))
    # equal scores: the mean over the tokens of the window and the rows of the blocks behind it
    T, size, pool = 23, 5, 4
    v = torch.randn(T, 1, 3).double()
    o = plain.pooled_attention_heads(torch.zeros(T, 2, 3).double(), torch.randn(T, 1, 3).double(), v, size, pool, 1.0)
    for i in range(T):
        rows = [v[j, 0] for j in range(max(0, i - size + 1), i + 1)]
        rows += [v[b:b + pool, 0].mean(0) for b in range(0, T, pool) if b + pool - 1 <= i - size]
        torch.testing.assert_close(o[i, 0], torch.stack(rows).mean(0))
    ks, vs = plain.pooled_window_keys(v, v, 13, size, pool)
    assert len(ks) == size + 2 and torch.equal(vs[-1], v[4:8].mean(0)), "position 13 sees 9..13 and the blocks 0..3 and 4..7"
    assert len(plain.pooled_window_keys(v, v, 11, size, pool)[0]) == size + 1, "at 11 the block 4..7 is not yet behind the window"
    # matrix memory: one token from zero gives v times q.k over max(|q.k|, ...); gates far apart keep or replace the state
    q, k, w = torch.randn(1, 4).double(), torch.randn(1, 4).double(), torch.randn(1, 3).double()
    qk = float(q @ k.T)
    for i0, f0 in ((0.5, -0.1), (-3.0, -0.2)):
        m = max(f0, i0)
        got = plain.matrix_memory_scan(q, k, w, torch.tensor([i0]).double(), torch.tensor([f0]).double())
        put = math.exp(i0 - m)
        torch.testing.assert_close(got[0], w[0] * (put * qk) / (max(abs(put * qk), math.exp(-m)) + 1e-6))
    # the delta rule: with w = 1 and a = 1 a repeated unit key is replaced by the new value, whatever was there
    u = torch.tensor([[1.0, 0.0], [1.0, 0.0], [0.0, 1.0]]).double()
    vals = torch.randn(3, 2).double()
    ones = torch.ones(3, 2).double()
    o = plain.general_delta_scan(torch.tensor([[1.0, 0.0], [1.0, 0.0], [1.0, 0.0]]).double(), u, vals, ones, ones)
    torch.testing.assert_close(o, torch.stack([vals[0], vals[1], vals[1]]), rtol=1e-5, atol=1e-5)
    z = torch.tensor([-40.0, -1.0, 0.0, 3.0], dtype=torch.float64)
    torch.testing.assert_close(plain.logsigmoid(z), torch.nn.functional.logsigmoid(z))


def test_what_the_comparisons_rest_on_shows_in_the_plain_model(tmp_path):
    """A window or a block's edge moved by one, block rows left out, rotated values, a lost state, the pair embedding
    left out or shifted, the frequencies' scaling left out: each moves the plain logits by far more than the tolerance
    the engine is held to."""
    toks = [(7 * i + i * i) % 250 for i in range(3, 75)]

    def moved(name, cfg_change=None, w_change=None):
        cfg, W = plain.read_model_dir(tk.write_model(name, tmp_path / name))
        base = plain.forward(cfg, W, toks, torch.float64)
        if cfg_change:
            cfg_change(cfg)
        if w_change:
            w_change(W)
        other = plain.forward(cfg, W, toks, torch.float64)
        return float((other - base).abs().max() / base.abs().max())

    left = lambda cfg: cfg["layers"][0]["mixer"]["left"]
    assert moved("window", lambda c: left(c)["mask"].update(size=21)) > 0.01
    assert moved("window", lambda c: left(c)["mask"].update(pool=5)) > 0.01
    assert moved("window", lambda c: left(c)["mask"].update(pool=None)) > 0.01
    assert moved("window", lambda c: left(c)["rot"].pop("scaling")) > 0.001
    assert moved("blocks", lambda c: left(c)["mask"].update(size=4)) > 0.01
    assert moved("memory", lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=60.0)) > 0.001
    assert moved("memory", lambda c: c["embedding"]["bigram"].update(mul_prev=3)) > 0.01
    assert moved("delta", None, lambda W: W.update({"bigram": torch.roll(W["bigram"], 1, 0)})) > 0.01
    assert moved("delta", lambda c: c.update(residual_mult=0.61)) > 0.001
    for name, fn, cut in (("memory", "matrix_memory_scan", None), ("delta", "general_delta_scan", None)):
        saved = getattr(plain, fn)
        try:
            cfg, W = plain.read_model_dir(tmp_path / name)
            base = plain.forward(cfg, W, toks, torch.float64)
            setattr(plain, fn, lambda *a: torch.cat([saved(*(t[:40] for t in a)), saved(*(t[40:] for t in a))]))
            lost = plain.forward(cfg, W, toks, torch.float64)                     # the state starts anew at token 40
        finally:
            setattr(plain, fn, saved)
        assert torch.equal(lost[:40], base[:40]) and float((lost[40:] - base[40:]).abs().max() / base.abs().max()) > 0.01
    saved = plain.pooled_attention
    try:
        cfg, W = plain.read_model_dir(tmp_path / "window")
        base = plain.forward(cfg, W, toks, torch.float64)

        def rotated_values(h, Wm, m, positions):
            q = plain.rotate_halves((h @ Wm["q"].T).reshape(len(h), m["heads"], -1), positions, m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"])
            k = plain.rotate_halves((h @ Wm["k"].T).reshape(len(h), m["kv_heads"], -1), positions, m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"])
            return plain.pooled_attention_heads(q, k, k, m["mask"]["size"], m["mask"]["pool"], m["scale"]).reshape(len(h), -1) @ Wm["o"].T
        plain.pooled_attention = rotated_values
        assert float((plain.forward(cfg, W, toks, torch.float64) - base).abs().max() / base.abs().max()) > 0.01
    finally:
        plain.pooled_attention = saved
