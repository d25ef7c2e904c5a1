"""Netolorn on the CPU: its configuration, plan, tensors and cache, and the plain implementation against closed forms."""
import json
import math

import pytest
import torch

import plain_netolorn as plain
import tiny_netolorn as tk


def test_registry_reads_the_architecture_string_and_round_trips(tmp_path):
    from garlic_inference_b200 import load_config
    from garlic_inference_b200.config import NetolornConfig, known_architectures
    assert "Netolorn" in known_architectures()
    (tmp_path / "config.json").write_text(json.dumps(tk.config_dict("mix")))
    cfg = load_config(tmp_path)
    assert type(cfg) is NetolornConfig and cfg.width == 96 and cfg.vocab == 411 and cfg.norm_eps == 2e-4
    assert cfg.loop == {"start": 1, "stop": 4, "times": 3} and cfg.side_dim == 12
    for name in tk.TINY:
        c = tk.make_config(name)
        assert NetolornConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    assert tk.make_config("tc").to_dict() == tk.config_dict("tc")


def test_plan_schedule_and_tensors():
    from garlic_inference_b200.engine.model import wanted_tensors
    plan = tk.make_config("mix").plan()
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [e.cache for e in plan.schedule] == list(range(11)), "every run of a layer has a cache entry of its own"
    assert [i for i, e in enumerate(plan.schedule) if e.mix == "loop.in"] == [1, 4, 7], "before every pass, the first too"
    assert all(layer.block == "sandwich_residual" for layer in plan.layers)
    assert list(plan.layers[2].norms) == ["input", "mixer_out"] and plan.layers[2].feed_forward is None
    assert [layer.side.params["offset"] for layer in plan.layers] == [0, 12, 24, 36, 48]
    names = wanted_tensors(plan)
    shape = lambda n: tuple(names[n].shape)
    assert shape("embed") == (411, 96) and shape("head") == (411, 96) and shape("loop.in") == (96, 192)
    assert shape("side.embed") == (411, 60) and shape("l4.side.gate") == (12, 96) and shape("l4.side.proj") == (96, 12)
    assert shape("l0.mix.dq") == (40, 96) and shape("l0.mix.uq") == (64, 40) and shape("l0.mix.dkv") == (56, 96)
    assert shape("l0.mix.uk") == (64, 56) and shape("l0.mix.uv") == (96, 56) and shape("l0.mix.g") == (4, 96)
    assert shape("l1.mix.q") == (96, 96) and shape("l1.mix.k") == (48, 96) and shape("l1.mix.v.b") == (48,)
    assert shape("l1.mix.g") == (96, 96) and shape("l1.mix.sink") == (6,) and shape("l2.mix.g") == (48, 96)
    assert shape("l1.mlp.router.b") == (8,) and "l1.mlp.shared.sg" not in names and shape("l3.mlp.shared.sg") == (1, 96)
    assert "l2.norm2" not in names and shape("l2.norm1b.alpha") == () and shape("final.norm.b") == (96,)
    m = plan.layers[1].mixer.params
    assert m["mask"] == {"kind": "window", "size": 30, "keep_first": 18} and m["head_norm_eps"] == 2e-4 and m["learned_sink"]
    assert plan.layers[4].mixer.params["mask"] == {"kind": "causal"} and plan.layers[0].mixer.params["window"] == 33
    rot = next(p for k, p in plan.positions.items() if "300.0" in k).params
    assert rot["layout"] == "half" and rot["yarn"] == {k: float(v) for k, v in tk.YARN.items()} and rot["tables"] is False
    assert len(plan.positions) == 2
    bare = tk.make_config("window").plan()
    assert bare.layers[0].side is None and not bare.mixes and all(e.mix is None for e in bare.schedule)
    unit = plan.layers[3].feed_forward.params["shared"]
    assert unit["gate"] is True and unit["gate_max"] == unit["up_limit"] == 3.0 and unit["up_shift"] == 1.0 and unit["size"] == 24


def test_refusals_and_warnings():
    from garlic_inference_b200.config import ConfigError, NetolornConfig

    def refused(name, change, match):
        bad = tk.config_dict(name)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            NetolornConfig.from_dict(bad)

    mixer = lambda c: c["layers"][0]["mixer"]
    refused("window", lambda c: c["layers"][0].update(type="convolution"), "convolution")
    refused("dense", lambda c: c["layers"][0]["mlp"].update(kind="xielu"), "xielu")
    refused("window", lambda c: mixer(c).update(kv_heads=4), "no multiple")
    refused("window", lambda c: mixer(c)["mask"].update(size=0), "size must be positive")
    refused("window", lambda c: mixer(c)["mask"].update(keep_first=-1), "keep_first")
    refused("window", lambda c: mixer(c)["rot"].update(dims=7), "dims 7")
    refused("window", lambda c: mixer(c)["rot"]["scaling"].update(factor=0.0), "scaling")
    refused("window", lambda c: mixer(c).pop("scale"), "scale")
    refused("latent", lambda c: mixer(c).update(q_rank=0), "q_rank")
    refused("moe", lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top 8 of 7")
    refused("moe", lambda c: c["layers"][0]["mlp"].pop("expert"), "expert")
    refused("moe", lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "ff")
    refused("mix", lambda c: c["loop"].update(stop=9), "does not fit")
    refused("mix", lambda c: c["token_side"].update(dim=0), "token_side")
    refused("window", lambda c: c.pop("norm"), "norm")
    odd = tk.config_dict("moe")
    odd["layers"][0]["mlp"]["router"]["groups"] = 2
    with pytest.warns(UserWarning, match="groups"):
        NetolornConfig.from_dict(odd)


def test_frequencies_of_the_rotary_part():
    from garlic_inference_b200.parts import RotaryPositions
    for dims, base, sc in ((16, 300.0, tk.YARN), (48, 7000.0, dict(tk.YARN, original=1000)), (6, 100.0, dict(tk.YARN, factor=2.5, fast=3.0)),
                           (32, 10.0, dict(tk.YARN, fast=2.0, slow=2.0)), (8, 40.0, None)):
        f, magnitude = RotaryPositions.frequencies(dims, base, yarn=sc)
        want, mag = plain.turn_frequencies(dims, base, sc)
        torch.testing.assert_close(f, want, rtol=1e-14, atol=0.0)
        assert magnitude == mag


def test_cache_of_a_window_with_kept_first_tokens():
    """Pages behind the window come back, but not those of the kept first tokens; everything comes back with the slot."""
    from garlic_inference_b200.cache import KVRequirement, PagedCache
    for keep, kept in ((0, 0), (1, 1), (16, 1), (17, 2), (40, 3)):
        c = PagedCache([KVRequirement(2, 8, 20, keep_first=keep)], max_tokens=512, max_positions=4096, dtype=torch.float32,
                       device="cpu", page_size=16, max_slots=2)
        host = c.groups[0].host
        s, t = c.alloc_slot(), c.alloc_slot()
        for n in (3, 1, 60, 1, 35, 100):
            c.prepare([s, t], [n, 1]), c.commit([s, t], [n, 1])
        assert c.length(s) == 200
        # the last 20 positions of the next query are 181 .. 200: pages 11 and 12
        held = [lp for lp in range(13) if host.table[s, lp] >= 0]
        assert held == [*range(kept), 11, 12] and len(host.pages_of(s)) == kept + 2 and len(set(host.pages_of(s))) == kept + 2
        assert len(host.pages_of(t)) == 1
        c.free_slot(s)
        assert host.pool.n_free == host.pool.n_pages - 1 and (host.table[s] == -1).all()
        c.free_slot(t)
        u = c.alloc_slot()
        c.prepare([u], [250]), c.commit([u], [250])
        assert len(host.pages_of(u)) == kept + 2
        c.free_slot(u)
        assert host.pool.n_free == host.pool.n_pages


def test_plain_functions_against_closed_forms():
    # a window of 3 with two kept first tokens
    seen = plain.window_mask(7, 3, 2)
    assert seen[6].tolist() == [True, True, False, False, True, True, True] and seen[0].tolist() == [True] + [False] * 6
    assert seen[3].tolist() == [True] * 4 + [False] * 3 and plain.window_mask(4, 3)[3].tolist() == [False, True, True, True]
    # a sink that equals the only score takes half the weight; without one the weight is 1
    p = plain.softmax_sink(torch.tensor([[0.7]]), torch.tensor([[True]]), torch.tensor(0.7))
    assert float(p) == pytest.approx(0.5) and float(plain.softmax_sink(torch.tensor([[0.7]]), torch.tensor([[True]]))) == 1.0
    # Dynamic Tanh; a row's elements do not depend on each other
    y = plain.tanh_norm(torch.tensor([0.3, -2.0]), 1.5, torch.tensor([2.0, 1.0]), torch.tensor([0.1, 0.0]))
    assert y.tolist() == pytest.approx([2.0 * math.tanh(0.45) + 0.1, math.tanh(-3.0)], rel=1e-6)
    # a rotated pair keeps its length times the magnitude; position 0 is only scaled; what is not rotated passes
    x = torch.tensor([[[3.0, 1.0, 4.0, 2.0, 9.0]]], dtype=torch.float64)
    mag = 0.1 * math.log(8.0) + 1.0
    turned = plain.rotate_halves(x, torch.tensor([5]), 4, 50.0, tk.YARN)
    assert float(turned[0, 0, 4]) == 9.0 and float(torch.hypot(turned[0, 0, 0], turned[0, 0, 2])) == pytest.approx(5.0 * mag)
    assert plain.rotate_halves(x, torch.tensor([0]), 4, 50.0, tk.YARN)[0, 0, :4].tolist() == pytest.approx([3 * mag, mag, 4 * mag, 2 * mag])
    # all turns above `fast` keep their frequency, all below `slow` are divided
    f, _ = plain.turn_frequencies(32, 100.0, {"factor": 4.0, "original": 4000, "fast": 300.0, "slow": 100.0})
    base = [100.0 ** (-2 * i / 32) for i in range(16)]
    assert f[0] == base[0] and f[15] == pytest.approx(base[15] / 4.0) and any(b / 4.0 < v < b for v, b in zip(f.tolist(), base))
    # the router: biased logits choose, their softmax weighs
    W = {"router": torch.eye(4), "router.b": torch.tensor([0.0, 0.0, 2.0, -9.0])}
    idx, w = plain.route(torch.tensor([[1.0, 0.0, 0.0, 8.0]]), W, {"top": 2, "experts": 4})
    assert idx.tolist() == [[2, 0]] and w[0].tolist() == pytest.approx([1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])
    # an expert's unit at its limits
    one = torch.ones(1, 1)
    g = 1.5 / (1 + math.exp(-1.702 * 1.5))
    assert float(plain.clamped_expert(one, 9 * one, -9 * one, one, 1.5)) == pytest.approx(g * -0.5)
    assert plain.layer_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == \
        [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)]
    assert plain.layer_order({"layers": [0] * 2, "loop": {"start": 1, "stop": 1, "times": 5}}) == [(0, None), (1, None)]


def test_what_the_comparisons_rest_on_shows_in_the_plain_model(tmp_path):
    """A planted mistake in the plain model moves its logits: a window one token off at either end, the kept tokens, the
    sink, the gate, the mix before the first pass, the side input's columns, the router's bias, the shared expert's gate."""
    cfg, w = plain.read_model_dir(tk.write_model("mix", tmp_path / "mix"))
    toks = torch.randint(0, 411, (90,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(cfg, w, toks)

    def moved(change_cfg=None, change_w=None):
        c, ww = json.loads(json.dumps(cfg)), dict(w)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(ww)
        return float((plain.forward(c, ww, toks) - want).abs().max() / want.abs().max())

    mask = lambda i: (lambda c: c["layers"][i]["mixer"]["mask"])
    for i in (0, 1, 2, 3):
        for d in (-1, 1):
            assert moved(lambda c: mask(i)(c).update(size=mask(i)(c)["size"] + d)) > 1e-4, f"window of layer {i}"
    for i in (1, 2):
        for d in (-1, 1):
            assert moved(lambda c: mask(i)(c).update(keep_first=mask(i)(c)["keep_first"] + d)) > 1e-4, f"kept tokens of layer {i}"
    zero = lambda name: (lambda ww: ww.update({name: torch.zeros_like(ww[name])}))
    for name in ("l1.mix.sink", "l1.mix.g", "l0.mix.g", "l1.mlp.router.b", "l3.mlp.shared.sg", "l2.mix.q.b", "l0.norm1b.b"):
        assert moved(change_w=zero(name)) > 1e-4, name
    assert moved(change_w=lambda ww: ww.update({"side.embed": torch.roll(ww["side.embed"], 12, 1)})) > 1e-3
    assert moved(lambda c: c["loop"].update(times=2)) > 1e-3
    half = w["loop.in"].shape[0]
    assert moved(change_w=lambda ww: ww.update({"loop.in": torch.cat([ww["loop.in"][:, half:], ww["loop.in"][:, :half]], 1)})) > 1e-3
