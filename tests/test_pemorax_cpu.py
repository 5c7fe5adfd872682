"""Pemorax without a GPU: the configuration reader and its refusals, the builder's tensor names, shapes and page and state
plan, the two mixers' shares of a call site's state, and the plain implementation's own pieces against closed forms."""
import copy
import json
import math

import pytest
import torch

import pemorax_models as BM
import plain_pemorax as P


def test_config_is_read_and_written_back():
    import kvcm
    for c in BM.CONFIGS.values():
        cfg = kvcm.config.config_from_dict(c["cfg"])
        assert cfg.architecture == "Pemorax" and cfg.width == c["cfg"]["width"] and cfg.norm_eps == c["cfg"]["norm"]["eps"]
        assert kvcm.config.config_from_dict(cfg.to_json_dict()) == cfg


LEFT = lambda d, i=0: d["layers"][i]["mixer"]["left"]
RIGHT = lambda d, i=0: d["layers"][i]["mixer"]["right"]


@pytest.mark.parametrize("edit,word", [
    (lambda d: d["layers"][0].__setitem__("type", "attention"), "unknown type"),
    (lambda d: d["layers"][0]["mixer"].pop("right"), "right"),
    (lambda d: LEFT(d).__setitem__("kv_heads", 3), "multiple"),
    (lambda d: LEFT(d)["rot"].__setitem__("dims", 7), "even"),
    (lambda d: LEFT(d)["rot"].__setitem__("dims", 22), "within"),
    (lambda d: LEFT(d)["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: LEFT(d)["rot"].__setitem__("base", 1.0), "base above 1"),
    (lambda d: LEFT(d)["mask"].__setitem__("size", 0), "size"),
    (lambda d: LEFT(d)["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda d: LEFT(d).__setitem__("softcap", 0.0), "softcap"),
    (lambda d: LEFT(d).__setitem__("conv", 0), "conv"),
    (lambda d: LEFT(d).pop("scale"), "scale"),
    (lambda d: RIGHT(d)["decay"].pop(), "decay"),
    (lambda d: RIGHT(d).__setitem__("dim", 0), "dim"),
    (lambda d: RIGHT(d)["rot"].__setitem__("dims", 12), "within"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 9), "choose"),
    (lambda d: d["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda d: d["layers"][2]["mlp"].pop("ff"), "ff"),
    (lambda d: d["layers"][2].__setitem__("mlp", {"kind": "conv"}), "dense"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_config_refusals_name_the_key(edit, word):
    import kvcm
    d = json.loads(json.dumps(BM.CONFIGS["pem-a"]["cfg"]))
    edit(d)
    with pytest.raises(kvcm.config.ConfigError) as e:
        kvcm.config.config_from_dict(d)
    assert word in str(e.value)


def test_builder_names_every_tensor_once_and_plans_pages_and_state():
    import kvcm
    from kvcm.cache.pools import plan_cache
    from kvcm.engine.model_io import build_spec
    spec = build_spec(kvcm.config.config_from_dict(copy.deepcopy(BM.CONFIGS["pem-a"]["cfg"])))
    shapes = [s for b in spec.bindings for s in b.sources]
    names = [n for n, _ in shapes]
    assert len(names) == len(set(names))
    shapes = dict(shapes)
    for n, want in (("embed", (203, 72)), ("head", (203, 72)), ("l0.norm1", (72,)), ("l0.norm1b", (72,)), ("l0.mix.left.out", (72,)),
                    ("l0.mix.left.q", (80, 72)), ("l0.mix.left.k", (40, 72)), ("l0.mix.left.v", (24, 72)), ("l0.mix.left.g", (48, 72)),
                    ("l0.mix.left.o", (72, 48)), ("l0.mix.left.q.conv", (80, 4)), ("l0.mix.left.v.conv", (24, 4)),
                    ("l0.mix.right.q", (30, 72)), ("l0.mix.right.v", (42, 72)), ("l0.mix.right.g", (42, 72)), ("l0.mix.right.o", (72, 42)),
                    ("l0.mix.right.out", (72,)), ("l1.norm2b", (72,)), ("l1.mlp.router", (8, 72)), ("l1.mlp.router.b", (8,)),
                    ("l1.mlp.e7.down", (72, 24)), ("l2.mlp.up", (100, 72)), ("final.norm", (72,))):
        assert shapes[n] == want, n
    assert "l0.norm2" not in shapes and "l2.mlp.gate" not in shapes
    plan = plan_cache(spec)
    # kept first tokens lie at the front of a request, where windows give pages back: such a layer keeps every page
    assert [g.spec.window for g in plan.groups] == [0, 21, 0] and plan.has_state
    left, right = 3 * (80 + 40 + 24), 3 * 10 * 14
    assert plan.site_state[0].shape == (left + right,) and plan.site_state[0].dtype == torch.float32
    c = build_spec(kvcm.config.config_from_dict(copy.deepcopy(BM.CONFIGS["pem-c"]["cfg"])))
    assert plan_cache(c).site_state[0].shape == (2 * (21 + 7 + 9) + 2 + 36,)      # each share starts at a multiple of four
    assert plan_cache(c).site_state[1].shape == (2 * 6 * 5,)                      # no convolution: the right mixer's alone


def test_the_mixers_see_their_own_part_of_the_state():
    from kvcm.parts import MIXERS, NoPositionEncoding, SiteCache
    left = MIXERS.build("attention_general", hidden=8, num_heads=1, num_kv_heads=1, dk=3, dv=2, position=NoPositionEncoding(), gate=True, taps=3)
    right = MIXERS.build("retention", hidden=8, heads=1, dk=2, dv=3, decay=[0.5], position=NoPositionEncoding(), norm_eps=1e-5)
    m = MIXERS.build("side_by_side", left=left, right=right, out_norm=True, hidden=8)
    n = m.state_spec().shape[0]
    assert left.state_spec().shape == (16,) and right.state_spec().shape == (6,) and n == 24
    slab = torch.arange(5 * n, dtype=torch.float32).view(5, n)
    a, b = m._sites(SiteCache(state=slab))
    assert a.state.shape == (5, 16) and b.state.shape == (5, 6) and a.state.stride(0) == b.state.stride(0) == n
    assert b.state[3, 0].item() == 3 * n + 16
    with pytest.raises(ValueError, match="cache"):
        MIXERS.build("side_by_side", left=left, right=left)


@pytest.mark.parametrize("kw,word", [
    (dict(taps=3, gate=True, qk_norm=True), "convolution"), (dict(taps=3), "convolution"), (dict(taps=2, gate=True, bias=True), "convolution"),
    (dict(sink=True, sink_score=0.0), "sink"),
])
def test_attention_refuses_what_it_has_no_kernel_for(kw, word):
    from kvcm.parts import MIXERS, NoPositionEncoding
    with pytest.raises(ValueError, match=word):
        MIXERS.build("attention_general", hidden=8, num_heads=2, num_kv_heads=1, dk=4, dv=4, position=NoPositionEncoding(), **kw)


def test_loaded_weights_become_one_input_product():
    """The two mixers' own matrices are views of the joint one after ``prepare``."""
    from kvcm.parts import MIXERS, NoPositionEncoding
    left = MIXERS.build("attention_general", hidden=8, num_heads=2, num_kv_heads=1, dk=4, dv=2, position=NoPositionEncoding(), gate=True, taps=2)
    right = MIXERS.build("retention", hidden=8, heads=1, dk=2, dv=3, decay=[0.5], position=NoPositionEncoding(), norm_eps=1e-5)
    right.prepare = lambda *a: None                      # (what it asks of the kernel library needs no GPU here)
    m = MIXERS.build("side_by_side", left=left, right=right, left_scale=0.5, right_scale=0.25, out_norm=True, hidden=8)
    g = torch.Generator().manual_seed(1)
    kept = {}
    for path, part in m.named_parts():
        for n, s in part.param_specs().items():
            kept[path, n] = torch.randn(s.shape, generator=g)
            part.set_param(n, kept[path, n])
    m.prepare(torch.device("cpu"), torch.float32)
    a, b = left.projection.param("weight"), right.projection.param("weight")
    assert torch.equal(m._joint, torch.cat([kept["left.qkv", "weight"], kept["right.qkvg", "weight"]]))
    assert a.data_ptr() == m._joint.data_ptr() and b.data_ptr() == m._joint[a.shape[0]:].data_ptr()
    assert torch.equal(m._multipliers[0], 0.5 * kept["", "left_out"]) and torch.equal(m._multipliers[1], 0.25 * kept["", "right_out"])


# ------------------------------------------------------------------------ the plain implementation's pieces

def test_plain_convolution_rotation_and_window():
    u, w = torch.tensor([[1.0], [2.0], [4.0]], dtype=P.F), torch.tensor([[10.0, 100.0]], dtype=P.F)
    assert P.short_conv(u, w).flatten().tolist() == [100.0, 210.0, 420.0]        # the last tap is the row itself
    x = torch.arange(24, dtype=P.F).view(2, 1, 12) + 1.0
    rot = {"dims": 4, "base": 100.0}
    for inter, (a, b) in ((True, (2, 3)), (False, (1, 3))):
        y = P.rotate(x, rot, inter)
        assert torch.equal(y[0], x[0]) and torch.equal(y[1, :, 4:], x[1, :, 4:])
        t = 100.0 ** (-2.0 / 4)
        u, v = x[1, 0, a].item(), x[1, 0, b].item()
        assert y[1, 0, a].item() == pytest.approx(u * math.cos(t) - v * math.sin(t))
        assert y[1, 0, b].item() == pytest.approx(v * math.cos(t) + u * math.sin(t))
    ok = P.visible(7, {"size": 2, "keep_first": 1})
    assert ok[5].tolist() == [True, False, False, False, True, True, False]
    assert P.visible(7, {"size": 2})[5].tolist() == [False] * 4 + [True, True, False]
    assert torch.equal(P.visible(4, None), torch.tril(torch.ones(4, 4)).bool())


def test_plain_yarn_in_closed_form():
    """Frequencies below the fast edge pass, above the slow edge are divided, between them a line."""
    rot = {"dims": 8, "base": math.e ** 4, "scaling": BM.yarn(4.0, 2 * math.pi * math.e ** 2, math.e ** 1.5, 1.0)}
    f, amp = P.rotary_frequencies(rot)                   # dim(t) = 2 - ln t: fast -> 0.5 (floor 0), slow -> 2
    plain = [math.e ** (-4 * 2 * i / 8) for i in range(4)]
    assert f.tolist() == pytest.approx([plain[0], plain[1] * (0.5 / 4 + 0.5), plain[2] / 4, plain[3] / 4])
    assert amp == pytest.approx(0.1 * math.log(4) + 1)
    y = P.rotate(torch.ones(2, 1, 8, dtype=P.F), rot, True)
    assert y[0].flatten().tolist() == pytest.approx([amp] * 8)                   # position 0 is scaled too


def test_plain_softmax_router_and_gelu():
    s = torch.tensor([[0.0, math.log(2.0), float("-inf")], [-50.0, -50.0, -50.0], [800.0, 0.0, 0.0]], dtype=P.F)
    p = P.softmax_with_one(s)
    assert p[0].tolist() == pytest.approx([1 / 4, 2 / 4, 0.0]) and p[1].sum().item() < 1e-20 and p[2].tolist() == pytest.approx([1.0, 0.0, 0.0])
    idx, wt = P.route(torch.tensor([[1.0, 2.0, 0.0]], dtype=P.F), torch.eye(3, dtype=P.F), torch.tensor([0.0, -5.0, 3.0], dtype=P.F), 2)
    assert idx.tolist() == [[2, 0]]                      # the bias takes part in the choice and in the weights
    assert wt[0].tolist() == pytest.approx([math.exp(3) / (math.exp(3) + math.exp(1)), math.exp(1) / (math.exp(3) + math.exp(1))])
    z = torch.tensor([-3.0, -0.5, 0.0, 0.7, 4.0], dtype=P.F)
    assert torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_plain_retention_in_closed_form_and_whole_model_runs():
    """One head of one key element: the state is a decayed sum, the head's norm leaves a sign."""
    w = {n: torch.tensor([[1.0]], dtype=P.F) for n in ("q", "k", "v", "o", "g")}
    h = torch.tensor([[1.0], [2.0]], dtype=P.F)
    y = P.retention(h, {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, w, 1e-2)
    o = [1.0, (0.5 + 4.0) * 2.0]
    assert y[:, 0].tolist() == pytest.approx([v / math.sqrt(v * v + 1e-2) * t / (1 + math.exp(-t)) for v, t in zip(o, (1.0, 2.0))])
    import kvcm
    for c in BM.CONFIGS.values():
        cfg = kvcm.config.config_from_dict(c["cfg"])
        tensors = {n: t.double() for n, t in kvcm.weights.random_init.random_tensors(cfg, 3, torch.float32)}
        logits, after = P.trace(c["cfg"], tensors, [1, 2, 3, 4, 5])
        assert logits.shape == (5, c["cfg"]["vocab"]) and len(after) == len(c["cfg"]["layers"]) and torch.isfinite(logits).all()
        assert torch.allclose(P.forward(c["cfg"], tensors, [1, 2, 3]), logits[:3], atol=1e-12)      # causal: a prefix gives the same rows
