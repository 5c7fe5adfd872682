"""Bimepel without a GPU: the configuration reader and its refusals, the builder's tensor names, shapes and run
order, the cache plan and the pages that passed chunks give back, the scaled rotation's table, and the plain
implementation's own pieces against closed forms."""
import copy
import json
import math

import pytest
import torch

import bimepel_models as BM
import plain_bimepel as P


def test_config_is_read_and_written_back():
    import kvcm
    for c in BM.CONFIGS.values():
        cfg = kvcm.config.config_from_dict(c["cfg"])
        assert cfg.architecture == "Bimepel" and cfg.width == c["cfg"]["width"] and cfg.has_loop == ("loop" in c["cfg"])
        assert kvcm.config.config_from_dict(cfg.to_json_dict()) == cfg


@pytest.mark.parametrize("edit,word", [
    (lambda d: d["layers"][0].__setitem__("type", "conv"), "unknown type"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("kv_heads", 3), "multiple"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "even"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("dims", 22), "within"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), "factor"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("base", 1.0), "base above 1"),
    (lambda d: d["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["decay"].pop(), "decay"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("decay", 0.9), "decay"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 9), "choose"),
    (lambda d: d["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda d: d["layers"][2]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][2]["mlp"].__setitem__("limit", -1.0), "limit"),
    (lambda d: d["layers"][2].__setitem__("mlp", {"kind": "conv"}), "dense"),
    (lambda d: d["loop"].__setitem__("stop", 5), "loop"),
    (lambda d: d["loop"].__setitem__("times", 0), "loop"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_config_refusals_name_the_key(edit, word):
    import kvcm
    d = json.loads(json.dumps(BM.CONFIGS["bim-a"]["cfg"]))
    edit(d)
    with pytest.raises(kvcm.config.ConfigError) as e:
        kvcm.config.config_from_dict(d)
    assert word in str(e.value)


def test_builder_names_every_tensor_once_and_orders_the_loop():
    import kvcm
    from kvcm.cache.pools import plan_cache
    from kvcm.engine.model_io import build_spec
    spec = build_spec(kvcm.config.config_from_dict(copy.deepcopy(BM.CONFIGS["bim-a"]["cfg"])))
    names = [n for b in spec.bindings for n, _ in b.sources]
    assert len(names) == len(set(names))
    for want in ("embed", "l0.norm1", "l0.shift", "l0.mix.norm", "l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.g", "l1.mlp.router",
                 "l1.mlp.e7.down", "l1.norm2", "l2.mlp.gate", "l2.mlp.up", "l3.mix.o", "final.norm"):
        assert want in names, want
    assert "l0.norm2" not in names
    shapes = dict(s for b in spec.bindings for s in b.sources)
    assert shapes["l1.mix.q"] == (80, 72) and shapes["l1.mix.k"] == (40, 72) and shapes["l1.mix.v"] == (24, 72)
    assert shapes["l1.mix.g"] == (48, 72) and shapes["l1.mix.o"] == (72, 48) and shapes["l2.mix.norm"] == (80,)
    assert [c.layer for c in spec.order] == [0, 1, 2, 1, 2, 1, 2, 3] == P.run_order(BM.CONFIGS["bim-a"]["cfg"])
    plan = plan_cache(spec)
    assert sorted(plan.chunks) == [0, 37] and plan.has_state
    assert all(s is not None and s.shape == (72,) and s.dtype == torch.float32 for s in plan.site_block_state)     # a shift per run
    assert [s is not None for s in plan.site_state] == [True, False, True, False, True, False, True, False]
    assert plan.site_state[2].shape == (2 * 24 * 40,)
    assert len({(g, l) for g, l in zip(plan.site_group, plan.site_layer) if g >= 0}) == 4                             # pages per pass
    b = build_spec(kvcm.config.config_from_dict(copy.deepcopy(BM.CONFIGS["bim-b"]["cfg"])))
    assert [c.layer for c in b.order] == [0, 1, 2] and sorted(plan_cache(b).chunks) == [50, 70]


def test_the_output_head_is_the_token_table():
    import kvcm
    from kvcm.engine.model_io import build_spec
    from kvcm.weights.loader import load_from_tensors
    from kvcm.weights.random_init import random_tensors
    cfg = kvcm.config.config_from_dict(copy.deepcopy(BM.CONFIGS["bim-c"]["cfg"]))
    w = dict(random_tensors(cfg, 1, torch.float32))
    assert "head" not in w
    spec = build_spec(cfg)
    w["l0.norm2"] = torch.ones(41)                      # a layer without a feed-forward may still carry its norm
    mixers = [b.mixer for b in spec.blocks]
    for m in mixers:                                     # (what prepare() asks of the kernel library needs no GPU here)
        m.prepare = lambda *a: None
    load_from_tensors(spec, w, "cpu", torch.float32)
    assert spec.lm_head.param("weight").data_ptr() == spec.embedding.param("weight").data_ptr()


@pytest.mark.parametrize("chunk,B", [(37, 16), (16, 16), (9, 8), (100, 16), (3, 8)])
def test_passed_chunks_give_their_pages_back(chunk, B):
    """Pages that no later position can see are given back, and no page is given back while its keys are visible."""
    from kvcm.cache import core
    kv = core.PagedManager(64, B, 256, False, 0, [core.LayerGroupSpec(0, chunk), core.LayerGroupSpec()])
    s = core.Sequence()
    s.id = 1
    s.extend_tokens([5] * 7)
    kv.admit(s)
    n = 7
    for step in (0, 1, 1, 30, 2, 1, 60, 1, 5, 90, 1):
        s.extend_tokens([5] * step)
        n += step
        assert kv.ensure(s, n)
        s.num_computed = n
        kv.commit(s)
        first = n // chunk * chunk                       # first key that position n (or a later one) sees
        assert core.LayerGroupSpec(0, chunk).first_live(n) == first
        table = s.table(0)
        for page, pid in enumerate(table):
            dead = (page + 1) * B <= first
            assert (pid < 0) == dead, (n, page)
        assert all(pid >= 0 for pid in s.table(1))
    kv.release(s)
    assert kv.blocks_in_use(0) == 0 and kv.blocks_in_use(1) == 0
    with pytest.raises(ValueError):
        core.PagedManager(8, 8, 64, True, 0, [core.LayerGroupSpec(0, 8)])           # prefix caching keeps every key
    with pytest.raises(ValueError):
        core.PagedManager(8, 8, 64, False, 0, [core.LayerGroupSpec(0, -1)])


@pytest.mark.parametrize("dims,base,sc", [
    (12, 1000.0, BM.yarn(3.0, 64, 8.0, 0.5)), (64, 500000.0, BM.yarn(16.0, 8192, 32.0, 1.0)), (32, 10000.0, BM.yarn(4.0, 40, 32.0, 1.0)),
    (8, 20.0, BM.yarn(2.0, 100000, 1.0, 1.0)), (2, 50.0, BM.yarn(1.0, 64, 32.0, 1.0)), (16, 10000.0, None),
])
def test_scaled_rotation_table(dims, base, sc):
    from kvcm.parts import RotaryEmbedding
    r = RotaryEmbedding(dims + 6, base, dims, "half", scaling=sc)
    f, amp = P.rotary_frequencies({"dims": dims, "base": base, "scaling": sc})
    assert torch.allclose(r.frequency_table().double(), f, rtol=1e-6) and r.amplitude == pytest.approx(amp)


def test_mixers_without_a_kernel_for_the_amplitude_refuse_it():
    from kvcm.parts import MIXERS, RotaryEmbedding
    pos = RotaryEmbedding(16, 1000.0, scaling=BM.yarn(2.0, 64, 8.0, 1.0))
    with pytest.raises(ValueError, match="scaled"):
        MIXERS.build("attention", hidden=32, num_heads=2, num_kv_heads=1, head_dim=16, position=pos)
    with pytest.raises(ValueError, match="chunks"):
        MIXERS.build("attention_general", hidden=32, num_heads=2, num_kv_heads=1, dk=16, dv=16, position=pos, window=8, keep_first=2, chunk=4)


def test_plain_yarn_in_closed_form():
    """Frequencies below the fast edge pass, above the slow edge are divided, between them a line."""
    rot = {"dims": 8, "base": math.e ** 4, "scaling": BM.yarn(4.0, 2 * math.pi * math.e ** 2, math.e ** 1.5, 1.0)}
    # dim(t) = 8 ln(e^2 / t) / 8 = 2 - ln t:  fast -> 0.5 (floor 0), slow -> 2
    f, amp = P.rotary_frequencies(rot)
    plain = [math.e ** (-4 * 2 * i / 8) for i in range(4)]
    assert f.tolist() == pytest.approx([plain[0], plain[1] * (0.5 / 4 + 0.5), plain[2] / 4, plain[3] / 4])
    assert amp == pytest.approx(0.1 * math.log(4) + 1)


def test_plain_rotation_shift_and_chunks():
    x = torch.arange(24, dtype=P.F).view(2, 1, 12) + 1.0
    y = P.rotate_halves(x, torch.tensor([0, 5]), {"dims": 4, "base": 100.0})
    assert torch.equal(y[0], x[0]) and torch.equal(y[1, :, 4:], x[1, :, 4:])
    a = 5 * 100.0 ** (-2.0 / 4)
    u, v = x[1, 0, 1].item(), x[1, 0, 3].item()
    assert y[1, 0, 1].item() == pytest.approx(u * math.cos(a) - v * math.sin(a))
    assert y[1, 0, 3].item() == pytest.approx(v * math.cos(a) + u * math.sin(a))
    h = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=P.F)
    assert P.token_shift(h, torch.tensor([0.5, 2.0], dtype=P.F)).tolist() == [[0.5, -2.0], [2.0, 0.0]]
    ok = P.visible(7, 3)
    assert ok[5].tolist() == [False, False, False, True, True, True, False] and ok[6].tolist() == [False] * 6 + [True]
    assert P.visible(4).tolist() == torch.tril(torch.ones(4, 4)).bool().tolist()


def test_plain_feed_forwards_and_router():
    w = {"gate": torch.tensor([[2.0]], dtype=P.F), "up": torch.tensor([[-3.0]], dtype=P.F), "down": torch.tensor([[1.0]], dtype=P.F)}
    y = P.clamped_ff(torch.tensor([[1.0]], dtype=P.F), {"limit": 1.5}, w)            # g = 1.5, u = -1.5
    assert y.item() == pytest.approx(1.5 / (1 + math.exp(-1.702 * 1.5)) * -0.5)
    y = P.clamped_ff(torch.tensor([[-2.0]], dtype=P.F), {"limit": 1.5}, w)           # g = -4 (no lower bound), u = 1.5
    assert y.item() == pytest.approx(-4.0 / (1 + math.exp(1.702 * 4.0)) * 2.5)
    idx, wt = P.route(torch.tensor([[3.0, -3.0, 1.0]], dtype=P.F), torch.eye(3, dtype=P.F), {"top": 2, "scale": 2.0})
    s = [1 / (1 + math.exp(-3.0)), 1 / (1 + math.exp(-1.0))]
    assert idx.tolist() == [[0, 2]] and wt[0].tolist() == pytest.approx([2 * s[0] / sum(s), 2 * s[1] / sum(s)])


def test_plain_lightning_in_closed_form_and_whole_model_runs():
    """One head, one key element: the state is a decayed sum."""
    silu = lambda z: z / (1 + math.exp(-z))
    w = {n: torch.tensor([[1.0]], dtype=P.F) for n in ("q", "k", "v", "o")}
    w["g"], w["norm"] = torch.tensor([[0.0]], dtype=P.F), torch.tensor([3.0], dtype=P.F)
    h = torch.tensor([[1.0], [2.0]], dtype=P.F)
    y = P.mixer_lightning(h, {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, w, 1e-2)
    S0 = silu(1.0) ** 2
    o = [S0 * silu(1.0), (0.5 * S0 + silu(2.0) ** 2) * silu(2.0)]
    assert y[:, 0].tolist() == pytest.approx([v / math.sqrt(v * v + 1e-2) * 3.0 * 0.5 for v in o])
    import kvcm
    c = BM.CONFIGS["bim-c"]
    cfg = kvcm.config.config_from_dict(c["cfg"])
    tensors = {n: t.double() for n, t in kvcm.weights.random_init.random_tensors(cfg, 3, torch.float32)}
    logits, after = P.trace(c["cfg"], tensors, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 97) and len(after) == 4 and torch.isfinite(logits).all()
    assert torch.allclose(P.forward(c["cfg"], tensors, [1, 2, 3]), logits[:3], atol=1e-12)      # causal: a prefix gives the same rows
