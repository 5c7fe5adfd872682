"""Pemorax in the engine against the plain implementation (``plain_pemorax.py``, float64, whole sequences): every way of
cutting the work, every mechanism alone, pages and state slots that are used again, keys far away, at page borders and at
a window's edges, the first tokens, the rows before a portion, long decoding, the new kernels alone, and greedy generation
through the engine's own entry point and scheduler.

float32 engine: every logit within 5e-4 of the plain logits' spread.  bfloat16 engine: per position, the root mean square
of the difference (mean taken off) is held against the spread of the plain logits: at most 5 % of the positions
beyond 10 %, none beyond 40 % (a wrong kernel path, a stale page or a lost state moves most positions by the order of the
spread itself; what one lost key among hundreds does is the float32 engine's business).
"""
import itertools

import pytest
import torch

import helpers
import pemorax_models as BM
import plain_pemorax as P

pytestmark = pytest.mark.gpu

NAMES = ("pem-a", "pem-b", "pem-c")
LENGTHS = {"pem-a": [1, 9, 47, 130, 300], "pem-b": [3, 64, 150, 257], "pem-c": [2, 33, 190]}
CASES = [(n, d) for n in NAMES for d in ("float32", "bfloat16")]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[(name, dtype)] = BM.write_model(name, dtype, str(tmp_path_factory.mktemp(f"{name}_{dtype}")))
        return made[(name, dtype)]
    return get


@pytest.fixture(scope="module")
def oracle(folders):
    cache = {}

    def get(name, dtype, i):
        if (name, dtype, i) not in cache:
            cache[(name, dtype, i)] = BM.plain_logits(folders(name, dtype), tokens_of(name, i))
        return cache[(name, dtype, i)]
    return get


def tokens_of(name, i):
    return helpers.random_tokens(LENGTHS[name][i], BM.CONFIGS[name]["cfg"]["vocab"], 760 + i)


def replayer(folders, name, dtype, max_tokens, **kw):
    return helpers.Replayer(folders(name, dtype), dtype, max_tokens, BM.CONFIGS[name]["block_size"], **kw)


def close(got, ref, dtype, what):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    if dtype == "float32":
        worst, bound = (got - ref).abs().max().item(), 5e-4 * max(1.0, ref.std().item())
        assert worst <= bound, f"{what}: float32 logits differ by {worst:.3e} (bound {bound:.3e}) at {int((got - ref).abs().max(dim=-1).values.argmax())}"
        return
    d = got - ref
    d = d - d.mean(dim=-1, keepdim=True)
    err = d.pow(2).mean(dim=-1).sqrt() / ref.std().item()
    over = int((err > 0.10).sum())
    assert over <= max(1, int(0.05 * err.numel())) and err.max().item() < 0.4, \
        f"{what}: {over} of {err.numel()} positions beyond 10 % of the spread (worst {err.max().item():.3f} at {int(err.argmax())})"


# ------------------------------------------------------------------------ ways of cutting the work

@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_requests(name, dtype, folders, oracle):
    r = replayer(folders, name, dtype, 320)
    for i, n in enumerate(LENGTHS[name]):
        toks = tokens_of(name, i)
        got = r.step([dict(id=f"r{i}", tokens=toks, want=list(range(n)))], end=[f"r{i}"])
        close(got, oracle(name, dtype, i), dtype, f"{name} whole request {i}")
    assert r.kv.blocks_in_use() == 0
    for g in range(r.kv.num_groups()):
        if r.kv.group_window(g) == 0:
            assert r.stray_writes(g) == []


@pytest.mark.parametrize("name,dtype", CASES)
def test_prefill_against_token_by_token(name, dtype, folders, oracle):
    """The second request token by token from its first token on; the longest mostly as one portion, then 60 single
    tokens (windows pass over them)."""
    r = replayer(folders, name, dtype, 320)
    toks, ref = tokens_of(name, 1), oracle(name, dtype, 1)
    outs = [r.step([dict(id="x", tokens=[t], want=[0])]) for t in toks]
    close(torch.cat(outs), ref, dtype, f"{name} token by token")
    r.session.release("x")
    i = len(LENGTHS[name]) - 1
    toks, ref = tokens_of(name, i), oracle(name, dtype, i)
    head = len(toks) - 60
    outs = [r.step([dict(id="y", tokens=toks[:head], want=list(range(head)))])]
    outs += [r.step([dict(id="y", tokens=[t], want=[0])]) for t in toks[head:]]
    close(torch.cat(outs), ref, dtype, f"{name} prefill then 60 single tokens")


@pytest.mark.parametrize("name,dtype", CASES)
def test_portions_down_to_two_tokens(name, dtype, folders, oracle):
    r = replayer(folders, name, dtype, 320)
    sizes = itertools.cycle([7, 2, 13, 2, 1, 5, 31, 3, 2, 17, 64, 1, 1, 2])
    for i, n in enumerate(LENGTHS[name]):
        toks = tokens_of(name, i)
        outs, at = [], 0
        while at < n:
            k = min(next(sizes), n - at)
            outs.append(r.step([dict(id="p", tokens=toks[at:at + k], want=list(range(k)))]))
            at += k
        r.session.release("p")
        close(torch.cat(outs), oracle(name, dtype, i), dtype, f"{name} request {i} in portions")


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_requests_together_with_pages_used_again(name, dtype, folders, oracle):
    """Up to three live requests in a pool that cannot hold all requests at once: some bring a portion while others
    bring one token; a request that ends gives its pages and its state slot to the next one."""
    B = BM.CONFIGS[name]["block_size"]
    lens = LENGTHS[name]
    todo = list(range(len(lens))) + [1, 0]                       # two of them a second time
    pool = helpers.roundup(max(lens), B) + 2 * helpers.roundup(sorted(lens)[-2], B)
    r = replayer(folders, name, dtype, pool, max_live=3)
    cuts = itertools.cycle([11, 1, 2, 29, 1, 1, 5, 64, 3, 1])
    live, got, step_no = {}, {}, 0
    while todo or live:
        held = sum(helpers.roundup(len(tokens_of(name, i)), B) for i, _ in live.values())
        while todo and len(live) < 3 and held + helpers.roundup(lens[todo[0]], B) <= pool:
            i = todo.pop(0)
            held += helpers.roundup(lens[i], B)
            live[f"q{step_no}_{i}"] = (i, 0)
            got[f"q{step_no}_{i}"] = []
        entries, ends = [], []
        for rid, (i, at) in list(live.items()):
            toks = tokens_of(name, i)
            k = min(next(cuts), len(toks) - at)
            entries.append(dict(id=rid, tokens=toks[at:at + k], want=list(range(k))))
            live[rid] = (i, at + k)
            if at + k == len(toks):
                ends.append(rid)
        out = r.step(entries, end=())
        row = 0
        for e in entries:
            got[e["id"]].append(out[row:row + len(e["tokens"])])
            row += len(e["tokens"])
        for rid in ends:
            r.session.release(rid)
            del live[rid]
        step_no += 1
    for rid, parts in got.items():
        i = int(rid.split("_")[1])
        close(torch.cat(parts), oracle(name, dtype, i), dtype, f"{name} request {rid} among others")
    assert r.kv.blocks_in_use() == 0
    assert len(set(r.pages_seen)) < len(r.pages_seen)            # pages were handed out more than once


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, folders, oracle):
    """A short prompt, then 260 tokens one by one: the pages grow across many borders, windows pass over decoded tokens
    (one layer's pages are given back on the way), and both mixers' states are carried all along."""
    name = "pem-a"
    toks, ref = tokens_of(name, 4), oracle(name, dtype, 4)
    r = replayer(folders, name, dtype, 320)
    outs = [r.step([dict(id="d", tokens=toks[:40], want=list(range(40)))])]
    outs += [r.step([dict(id="d", tokens=[t], want=[0])]) for t in toks[40:]]
    close(torch.cat(outs), ref, dtype, "long decoding")


# ------------------------------------------------------------------------------ each mechanism alone

def one_layer_model(tmp_path, layers, dtype="float32", width=48, vocab=120, eps=3e-6, seed=5, decisive=False):
    cfg = BM.model(vocab, width, eps, layers if isinstance(layers, list) else [layers])
    return BM.write_model_from(cfg, seed, dtype, str(tmp_path / "m"), decisive=decisive)


_YARN = BM.yarn(4.0, 32, 4.0, 0.25)
_R = BM.right(6, 10, [0.9, 0.4], (30.0, 4))
_L = BM.left(2, 1, 8, 12, 0.5, 2, (100.0, 4), 30, 2, 5.0)
ALONE = [
    ("plain_attention", BM.layer(BM.left(2, 2, 8, 8, 0.6, 0), _R)),
    ("one_tap", BM.layer(BM.left(4, 2, 12, 20, 0.6, 1, (100.0, 6)), _R)),
    ("two_taps_small_window", BM.layer(BM.left(4, 2, 12, 20, 0.6, 2, (100.0, 6), 2), _R)),
    ("three_taps_odd_heads", BM.layer(BM.left(3, 1, 7, 9, 0.5, 3, (50.0, 6), 21, 1), _R)),
    ("four_taps_yarn_whole_head", BM.layer(BM.left(3, 1, 16, 8, 0.5, 4, (5000.0, 16, _YARN), 33, 17, 9.0), _R)),
    ("six_taps", BM.layer(BM.left(2, 1, 8, 4, 0.9, 6, (9.0, 2), 16, 5, 1.5), _R)),
    ("kept_tokens_beyond_the_window", BM.layer(BM.left(2, 1, 8, 16, 0.9, 3, (9.0, 8), 5, 50), _R)),
    ("long_heads", BM.layer(BM.left(2, 1, 300, 20, 0.05, 3, (50.0, 64), 40, 4, 2.0), BM.right(200, 9, [0.95, 1.0], (50.0, 200)))),
    ("retention_unrotated_no_memory", BM.layer(_L, BM.right(8, 33, [0.0]))),
    ("retention_odd", BM.layer(_L, BM.right(11, 7, [0.5, 0.99, 1.0], (77.0, 10)))),
    ("retention_wide_values", BM.layer(_L, BM.right(16, 300, [0.97], (77.0, 8)))),
    ("gelu_dense", BM.layer(_L, _R, BM.dense(100))),
    ("gelu_dense_odd", BM.layer(_L, _R, BM.dense(33))),
    ("experts", BM.layer(_L, _R, BM.moe(12, 3, 14))),
    ("experts_all_chosen", BM.layer(_L, _R, BM.moe(3, 3, 9))),
    ("expert_one_of_many", BM.layer(_L, _R, BM.moe(40, 1, 8))),
    ("three_layers", [BM.layer(_L, _R, BM.moe(6, 2, 8)), BM.layer(BM.left(3, 3, 5, 6, 0.4, 3), _R), BM.layer(_L, BM.right(5, 4, [0.8]), BM.dense(20))]),
]


@pytest.mark.parametrize("layers", [l for _, l in ALONE], ids=[n for n, _ in ALONE])
def test_one_layer_alone(tmp_path, layers):
    """Every branch of every mechanism in float32: whole, and in portions with single tokens at the end (portions shorter
    than the convolution's taps among them)."""
    folder = one_layer_model(tmp_path, layers)
    cfg, w = BM.read_model(folder)
    toks = helpers.random_tokens(90, 120, 77)
    ref = P.forward(cfg, w, toks)
    for opts in ({}, {"fuse": False}):
        r = helpers.Replayer(folder, "float32", 256, 16, options=opts)
        close(r.step([dict(id="a", tokens=toks, want=list(range(90)))], end=["a"]), ref, "float32", f"whole {opts}")
        outs, at = [], 0
        for k in (2, 2, 1, 3, 33, 1, 2, 37):
            outs.append(r.step([dict(id="b", tokens=toks[at:at + k], want=list(range(k)))]))
            at += k
        outs += [r.step([dict(id="b", tokens=[t], want=[0])]) for t in toks[at:]]
        close(torch.cat(outs), ref, "float32", f"portions {opts}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [
    BM.layer(BM.left(8, 2, 64, 64, 0.1, 3, (10000.0, 32, BM.yarn(4.0, 64, 32.0, 1.0)), 100, 4, 30.0), BM.right(64, 64, [0.5, 0.9, 0.99], (10000.0, 64)), BM.dense(512)),
    BM.layer(BM.left(6, 1, 128, 96, 0.07, 4, (250000.0, 128), 150, 70, 20.0), BM.right(128, 96, [0.7, 0.995], (500.0, 64))),
    BM.layer(BM.left(4, 4, 32, 48, 0.2, 2, (10000.0, 32), 64, 1), BM.right(32, 160, [0.9, 0.999], (10000.0, 32)), BM.moe(8, 2, 128)),
    BM.layer(BM.left(4, 2, 64, 160, 0.1, 3, (10000.0, 16), 37, 3, 4.0), BM.right(96, 64, [0.98], (10000.0, 96)), BM.moe(6, 3, 64)),
    BM.layer(BM.left(4, 2, 128, 128, 0.09, 3, (10000.0, 64), None, None, 50.0), BM.right(64, 128, [0.6, 0.9], (10000.0, 32)), BM.dense(264)),
], ids=["heads64_window100", "heads128_window150_keep70", "heads48_window64", "heads160_window37", "heads128_causal"])
def test_mixers_at_the_sizes_of_the_fast_kernels(tmp_path, layer, dtype):
    """Head sizes that take the tensor-core attention kernels (both prefill kernels), the chunked recurrence and experts
    that take the tensor-core products, in a prompt of three portions and 70 decoded tokens, beside a second request."""
    folder = one_layer_model(tmp_path, layer, dtype, width=256, vocab=200, decisive=True)
    cfg, w = BM.read_model(folder)
    toks, other = helpers.random_tokens(420, 200, 3), helpers.random_tokens(150, 200, 4)
    ref, ref2 = P.forward(cfg, w, toks), P.forward(cfg, w, other)
    r = helpers.Replayer(folder, dtype, 640, 16)
    outs = [r.step([dict(id="a", tokens=toks[:200], want=list(range(200)))]),
            r.step([dict(id="a", tokens=toks[200:203], want=[0, 1, 2]), dict(id="b", tokens=other[:100], want=list(range(100)))])]
    o2 = [outs[1][3:]]
    outs[1] = outs[1][:3]
    outs.append(r.step([dict(id="a", tokens=toks[203:350], want=list(range(147)))]))
    for k, t in enumerate(toks[350:]):
        e = [dict(id="a", tokens=[t], want=[0])]
        if k < 50:
            e.append(dict(id="b", tokens=[other[100 + k]], want=[0]))
        out = r.step(e)
        outs.append(out[:1])
        if k < 50:
            o2.append(out[1:])
    close(torch.cat(outs), ref, dtype, "first request")
    close(torch.cat(o2), ref2[:len(torch.cat(o2))], dtype, "second request")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_in_one_portion(tmp_path, dtype):
    """More rows than the head kernel's threshold for several rows a thread, in one step beside short portions and single
    tokens: the rows before a group's first, states read and written by the right rows."""
    layers = [BM.layer(BM.left(2, 1, 16, 12, 0.4, 4, (1000.0, 8), 50, 2, 6.0), BM.right(16, 8, [0.9, 0.99], (1000.0, 16)), BM.moe(6, 2, 16)),
              BM.layer(BM.left(3, 1, 8, 16, 0.4, 3, (1000.0, 8)), BM.right(8, 16, [0.8]), BM.dense(40))]
    folder = one_layer_model(tmp_path, layers, dtype, width=64, decisive=True)
    cfg, w = BM.read_model(folder)
    toks, other, third = (helpers.random_tokens(n, 120, 30 + n) for n in (1213, 18, 9))
    refs = [P.forward(cfg, w, t) for t in (toks, other, third)]
    r = helpers.Replayer(folder, dtype, 1536, 16)
    o2 = [r.step([dict(id="b", tokens=other[:5], want=list(range(5)))])]
    out = r.step([dict(id="c", tokens=third[:2], want=[0, 1]), dict(id="a", tokens=toks[:1101], want=list(range(1101))),
                  dict(id="b", tokens=[other[5]], want=[0])])
    o3, o1 = [out[:2]], [out[2:1103]]
    o2.append(out[1103:])
    out = r.step([dict(id="a", tokens=toks[1101:1203], want=list(range(102))), dict(id="b", tokens=other[6:18], want=list(range(12))),
                  dict(id="c", tokens=third[2:9], want=list(range(7)))])
    o1.append(out[:102])
    o2.append(out[102:114])
    o3.append(out[114:])
    o1 += [r.step([dict(id="a", tokens=[t], want=[0])]) for t in toks[1203:]]
    for got, ref, what in zip((o1, o2, o3), refs, ("long", "second", "third")):
        close(torch.cat(got), ref, dtype, what)


# ------------------------------------------------------------ one key that carries all the weight

D_PLANT, PLANTED = 48, 119


def plant(tmp_path, dtype, kind, window, keep):
    """A one-layer model in which every query points at the key of ONE token (id 119, used once per prompt) and all
    other scores are zero.  The token's row of the table lies along coordinate 0, every other token has a common
    component along coordinate 1 and nothing along 0; keys read coordinate 0 and queries coordinate 1, in head
    dimensions that the rotation leaves alone.  The convolutions pass their input on, the other mixer's result is zero.
    Losing the key, or seeing it one position too long, changes the logits completely.  For the recurrence only the
    planted token has a key at all."""
    D = D_PLANT
    H, G, dk, dv = 2, 1, 16, 12
    Hr, dr, dvr = 2, 6, 10
    layer = BM.layer(BM.left(H, G, dk, dv, 2.0, 3, (100.0, 8, BM.yarn(2.0, 64, 8.0, 1.0)), window or None, keep, 25.0),
                     BM.right(dr, dvr, [0.97, 0.999], (100.0, 4)))
    folder = one_layer_model(tmp_path, layer, dtype, width=D)
    cfg, w = BM.read_model(folder)
    g = torch.Generator().manual_seed(9)
    w["embed"] = torch.randn(120, D, generator=g, dtype=torch.float64) * 0.3
    w["embed"][:, :2] = 0
    w["embed"][:, 1] = 2.0
    w["embed"][PLANTED] = 0
    w["embed"][PLANTED, 0] = 6.0
    w["l0.norm1"] = torch.ones(D, dtype=torch.float64)
    p = "l0.mix.left."
    for n in ("q", "k", "v"):
        w[p + n + ".conv"] = torch.zeros_like(w[p + n + ".conv"])
        w[p + n + ".conv"][:, -1] = 1.0
    if kind == "attention":
        w["l0.mix.right.o"] = torch.zeros_like(w["l0.mix.right.o"])
        wk = torch.randn(G * dk, D, generator=g, dtype=torch.float64) * 0.1
        wk[:, :2] = 0
        wk[12:16] = 0                                # dimensions 12..15 are not rotated: no other token's key reaches into them ...
        wk[12:16, 0] = 1.0                           # ... they hold the planted token's key
        wq = torch.zeros(H * dk, D, dtype=torch.float64)
        for h in range(H):
            wq[h * dk + 12:h * dk + 16, 1] = 1.0
        w[p + "q"], w[p + "k"] = wq, wk
    else:
        w[p + "o"] = torch.zeros_like(w[p + "o"])
        p = "l0.mix.right."
        wk, wq = torch.zeros(Hr * dr, D, dtype=torch.float64), torch.zeros(Hr * dr, D, dtype=torch.float64)
        for h in range(Hr):
            wk[h * dr + 4:h * dr + 6, 0] = 0.6       # (the dimensions behind the rotated ones)
            wq[h * dr + 4:h * dr + 6, 1] = 0.5
        w[p + "q"], w[p + "k"] = wq, wk
        w[p + "v"][:, 0] = torch.randn(Hr * dvr, generator=g, dtype=torch.float64) * 2.0
    BM.save_weights(folder, w, dtype)
    return folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,window,keep", [("attention", 0, 0), ("attention", 40, 3), ("attention", 33, 0), ("attention", 64, 17), ("attention", 5, 70),
                                              ("retention", 0, 0)])
def test_one_key_that_stands_out(tmp_path, dtype, kind, window, keep):
    """The planted key is tried as first key, as the last kept and the first that is not, just before, at and behind page
    borders, and far back; the asking positions are in a prompt's portion and decoded alone.  With a window the key is
    seen up to exactly ``window`` - 1 positions later, a kept one from everywhere; the check that the plant works
    compares exactly these positions in the plain implementation."""
    folder = plant(tmp_path, dtype, kind, window, keep)
    cfg, w = BM.read_model(folder)
    n, head = 200, 120
    places = [0, 1, 15, 16, 17, 31, 32, 33, 79, 81, 100, 150]
    if window:
        places += [p for p in (keep - 1, keep, head - window, head - window + 1, 130 - window) if p >= 0]
    for far in sorted(set(places)):
        toks = helpers.random_tokens(n, PLANTED, 40 + far)
        toks[far] = PLANTED
        ref = P.forward(cfg, w, toks)
        r = helpers.Replayer(folder, dtype, 256, 16)
        outs = [r.step([dict(id="f", tokens=toks[:far + 1], want=list(range(far + 1)))])]
        if far + 1 < head:
            outs.append(r.step([dict(id="f", tokens=toks[far + 1:head], want=list(range(head - far - 1)))]))
        outs += [r.step([dict(id="f", tokens=[t], want=[0])]) for t in toks[max(head, far + 1):]]
        close(torch.cat(outs), ref, dtype, f"planted key at {far}")
        spread = ref.std().item()
        toks2 = list(toks)
        toks2[far] = 5
        without = P.forward(cfg, w, toks2)
        first_out = n if not window or far < keep else min(n, far + window)
        if first_out - 1 > far:                   # the key is seen up to here and carries the weight
            assert (without[first_out - 1] - ref[first_out - 1]).abs().max().item() > 0.5 * spread
        if first_out < n:                         # and not one position later
            assert (without[first_out] - ref[first_out]).abs().max().item() < 1e-6 * max(1.0, spread)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [2, 3, 4, 5])
def test_the_rows_before_a_portion(tmp_path, dtype, taps):
    """All the convolutions' weight on the oldest tap: what is projected IS the row taps - 1 earlier.  Wherever a portion or a
    single token begins, its first rows depend on the request's own kept rows; portions shorter than the taps move kept
    rows on; two requests swap slots after the first ends."""
    layer = BM.layer(BM.left(2, 1, 16, 12, 0.3, taps, (100.0, 8), 24, 2), BM.right(8, 4, [0.9], (100.0, 8)), BM.dense(24))
    folder = one_layer_model(tmp_path, [layer, layer], dtype)
    cfg, w = BM.read_model(folder)
    for n in w:
        if n.endswith(".conv"):
            w[n] = w[n] * 0.05
            w[n][:, 0] = 1.0
    BM.save_weights(folder, w, dtype)
    toks, other = helpers.random_tokens(70, 120, 3), helpers.random_tokens(70, 120, 4)
    ref, ref2 = P.forward(cfg, w, toks), P.forward(cfg, w, other)
    r = helpers.Replayer(folder, dtype, 192, 16, max_live=2)
    for a, b, ra, rb in ((toks, other, ref, ref2), (other, toks, ref2, ref)):
        at, got_a, got_b = 0, [], []
        for k in (1, 2, 3, 1, 1, 20, 2, 2, 17, 1, 20):
            out = r.step([dict(id="a", tokens=a[at:at + k], want=list(range(k))), dict(id="b", tokens=b[at:at + k], want=list(range(k)))])
            got_a.append(out[:k])
            got_b.append(out[k:])
            at += k
        assert at == 70
        r.session.release("b")
        r.session.release("a")
        close(torch.cat(got_a), ra, dtype, "first")
        close(torch.cat(got_b), rb, dtype, "second")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_one_in_the_denominator(tmp_path, dtype):
    """Every score is far below zero (a common coordinate makes q . k strongly negative): the added one takes nearly all of
    the weight, the attention's result is close to nothing, and its norm lifts what is left of it.  The plain result with
    an ordinary softmax is far away."""
    D = 48
    layer = BM.layer(BM.left(2, 1, 16, 12, 1.0, 2, (100.0, 8), 30, 2, 6.0), BM.right(8, 4, [0.9], (100.0, 8)))
    folder = one_layer_model(tmp_path, layer, dtype, width=D, eps=1e-3)
    cfg, w = BM.read_model(folder)
    p = "l0.mix.left."
    w["embed"][:, 0] = 3.0
    w["l0.norm1"] = torch.ones(D, dtype=torch.float64)
    w["l0.mix.right.o"] = torch.zeros_like(w["l0.mix.right.o"])
    for n, s in (("q", 1.0), ("k", -1.0)):
        w[p + n][8:16, 0] = s
        w[p + n + ".conv"] = torch.tensor([0.1, 1.0], dtype=torch.float64).expand_as(w[p + n + ".conv"]).contiguous()
    w[p + "q"][24:32, 0] = 1.0
    BM.save_weights(folder, w, dtype)
    toks = helpers.random_tokens(80, 120, 8)
    ref = P.forward(cfg, w, toks)
    kept, P.softmax_with_one = P.softmax_with_one, lambda s: torch.softmax(s, dim=-1)
    try:
        assert (P.forward(cfg, w, toks) - ref).abs().max().item() > 0.3 * ref.std().item()
    finally:
        P.softmax_with_one = kept
    r = helpers.Replayer(folder, dtype, 128, 16)
    outs = [r.step([dict(id="a", tokens=toks[:60], want=list(range(60)))])]
    outs += [r.step([dict(id="a", tokens=[t], want=[0])]) for t in toks[60:]]
    close(torch.cat(outs), ref, dtype, "the one in the denominator")


# --------------------------------------------------------------------------------- kernels alone

class _Ctx:
    """The index tensors that a step's kernels read, for requests of the given numbers of rows, slots and first positions."""

    def __init__(self, lens, slots, first=None):
        start = [sum(lens[:i]) for i in range(len(lens))]
        ints = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        self.row_seq = ints([i for i, n in enumerate(lens) for _ in range(n)])
        self.positions = ints([p + (first[i] if first else 0) for i, n in enumerate(lens) for p in range(n)])
        self.seq_q_start, self.seq_q_len, self.seq_state_slot = ints(start), ints(lens), ints(slots)
        self.seqs = len(lens)
        tiles = [(i, q) for i, m in enumerate(lens) if m > 1 for q in range(0, m, 64)]
        self.tile_seq, self.tile_q0 = ints([i for i, _ in tiles]), ints([q for _, q in tiles])
        self.prefill_tiles, self.tile_rows = len(tiles), 64


def turned(x, pos, freq, amp, inter):
    """x [T, heads, n] float64, the first 2 * len(freq) elements turned (by the float32 product of position and frequency)."""
    out = x.clone()
    m = len(freq)
    a = (pos.float()[:, None] * freq[None, :]).double()
    c, s = (amp * torch.cos(a))[:, None], (amp * torch.sin(a))[:, None]
    ia, ib = (slice(0, 2 * m, 2), slice(1, 2 * m, 2)) if inter else (slice(0, m), slice(m, 2 * m))
    u, v = x[..., ia], x[..., ib]
    out[..., ia], out[..., ib] = u * c - v * s, v * c + u * s
    return out


@pytest.mark.parametrize("lens", [[1], [1, 1, 1], [5], [1, 2, 3, 4, 5, 6, 7], [300], [1, 1, 615, 2, 3, 1, 600]])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 8, 12, 2, 24, 3), (2, 1, 64, 48, 32, 4, 32, 4), (6, 3, 20, 28, 6, 3, 12, 2), (3, 1, 7, 9, 6, 2, 5, 3),
                                   (2, 2, 8, 16, 8, 1, 16, 6), (2, 1, 12, 4, 4, 2, 8, 1)])
def test_head_kernel(lens, sizes):
    """One launch for an attention's q, k, v (convolved, interleaved rotation, padded rows and page slots) and a recurrence's q
    and k (rotate-half, scaled, in place), against float64: sizes in fours and others, one to six taps, states read and
    written per slot, portions shorter than the taps, padding entries (no slot), what must not be touched."""
    from kvcm.kernels import library as K
    nh, nkv, dk, dv, rot, H2, d2, taps = sizes
    g = torch.Generator(device="cuda").manual_seed(sum(lens) + dk)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    T, B, HD = sum(lens), 8, (max(dk, dv) + 15) // 16 * 16
    nq, nk, nv = nh * dk, nkv * dk, nkv * dv
    C, extra = nq + nk + nv, 5 if dk % 4 else 8
    width = C + extra + 2 * H2 * d2 + 4
    slots = [(5 * i + 2) % 23 for i in range(len(lens))]
    if len(lens) > 2:
        slots[-1] = -1
    ctx = _Ctx(lens, slots, [11 * i for i in range(len(lens))])
    proj, conv_w, wide = rnd(T, width), rnd(C, taps), rnd(23, (taps - 1) * C + 12)
    state = wide[:, 4:4 + max((taps - 1) * C, 1)]
    old, before = state.double().clone(), wide.clone()
    f1, f2 = (torch.rand(n, device="cuda", generator=g) for n in (rot // 2, d2 // 4 if d2 % 16 == 0 else d2 // 2))
    cache_slots = torch.randperm(T + 40, device="cuda", generator=g)[:T].to(torch.int32)
    if slots[-1] < 0:
        cache_slots[-1] = -1
    pages = (T + 40 + B - 1) // B
    # the convolution in float64
    u, y, want_state, at = proj[:, :C].double(), torch.zeros(T, C, dtype=torch.float64, device="cuda"), old.clone(), 0
    for n, s in zip(lens, slots):
        hist = old[s, :(taps - 1) * C].view(taps - 1, C) if s >= 0 else torch.zeros(taps - 1, C, dtype=torch.float64, device="cuda")
        full = torch.cat([hist, u[at:at + n]])
        for j in range(taps):
            y[at:at + n] += conv_w[:, j].double() * full[j:j + n]
        if s >= 0 and taps > 1:
            want_state[s, :(taps - 1) * C] = full[n:].reshape(-1)
        at += n
    pos = ctx.positions
    q = turned(y[:, :nq].view(T, nh, dk), pos, f1, 1.3, True) * 0.7
    k = turned(y[:, nq:nq + nk].view(T, nkv, dk), pos, f1, 1.3, True)
    v = y[:, nq + nk:].view(T, nkv, dv)
    b2 = C + extra
    q2 = turned(proj[:, b2:b2 + H2 * d2].double().view(T, H2, d2), pos, f2, 1.0, False)
    k2 = turned(proj[:, b2 + H2 * d2:b2 + 2 * H2 * d2].double().view(T, H2, d2), pos, f2, 1.0, False) * 0.25
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        wide.copy_(before)
        p = proj.clone()
        qo = torch.full((T, nh * HD), 9.0, dtype=dt, device="cuda")
        kc, vc = (torch.full((pages, nkv, B, HD), 9.0, dtype=dt, device="cuda") for _ in range(2))
        turn = dict(inv_freq=f1, amplitude=1.3, interleaved=True)
        segs = [K.HeadSegment(nh, dk, 0, "rows", qo, conv=0, scale=0.7, **turn), K.HeadSegment(nkv, dk, nq, "pages", kc, conv=nq, **turn),
                K.HeadSegment(nkv, dv, nq + nk, "pages", vc, conv=nq + nk),
                K.HeadSegment(H2, d2, b2, "float", p, inv_freq=f2, out_col=b2),
                K.HeadSegment(H2, d2, b2 + H2 * d2, "float", p, inv_freq=f2, scale=0.25, out_col=b2 + H2 * d2)]
        K.prepare_heads(p, segs, ctx, dt, K.HeadConv(conv_w, state if taps > 1 else None, 0), cache_slots, B)
        amp = max(q.abs().max().item(), 1.0)
        got = qo.view(T, nh, HD).double()
        assert torch.allclose(got[..., :dk], q, atol=tol * amp) and bool((got[..., dk:] == 0).all())
        flat = lambda c: c.permute(0, 2, 1, 3).reshape(pages * B, nkv, HD).double()
        live = cache_slots >= 0
        rows = cache_slots[live].long()
        for c, want, d in ((kc, k, dk), (vc, v, dv)):
            got = flat(c)
            assert torch.allclose(got[rows][..., :d], want[live], atol=tol * max(1.0, want.abs().max().item())) and bool((got[rows][..., d:] == 0).all())
            rest = torch.ones(pages * B, dtype=torch.bool, device="cuda")
            rest[rows] = False
            assert bool((got[rest] == 9.0).all())
        assert torch.allclose(p[:, b2:b2 + H2 * d2].double().view(T, H2, d2), q2, atol=2e-5 * q2.abs().max().item())
        assert torch.allclose(p[:, b2 + H2 * d2:b2 + 2 * H2 * d2].double().view(T, H2, d2), k2, atol=2e-5 * q2.abs().max().item())
        same = torch.ones(width, dtype=torch.bool, device="cuda")
        same[b2:b2 + 2 * H2 * d2] = False
        assert torch.equal(p[:, same], proj[:, same])
        if taps > 1:
            assert torch.allclose(state.double(), want_state, atol=1e-6)
        assert torch.equal(wide[:, :4], before[:, :4]) and torch.equal(wide[:, 4 + (taps - 1) * C:], before[:, 4 + (taps - 1) * C:])
    assert K.head_layouts_match()


@pytest.mark.parametrize("T,H1,dv1,HD,H2,dv2", [(1, 2, 12, 16, 3, 8), (9, 6, 48, 48, 2, 64), (5, 3, 7, 16, 2, 9), (700, 4, 128, 128, 3, 96), (3, 2, 20, 32, 2, 600)])
def test_gate_kernel(T, H1, dv1, HD, H2, dv2):
    """Padded heads with a sigmoid gate and normalised float heads with a SiLU gate in one launch."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(T)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    n1, n2 = H1 * dv1, H2 * dv2
    proj, o = rnd(T, 4 + n1 + n2), rnd(T, n2) * 3
    z1, z2 = proj[:, 4:4 + n1].double(), proj[:, 4 + n1:].double()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        x = rnd(T, H1 * HD).to(dt)
        a, b = torch.empty(T, n1, dtype=dt, device="cuda"), torch.empty(T, n2, dtype=dt, device="cuda")
        K.gate_heads(proj, [K.GateSegment(x, a, H1, dv1, 4, None, "sigmoid"), K.GateSegment(o, b, H2, dv2, 4 + n1, 1e-2, "silu")])
        wa = x.double().view(T, H1, HD)[..., :dv1].reshape(T, n1) * torch.sigmoid(z1)
        wb = P.rms_div(o.double().view(T, H2, dv2), 1e-2).view(T, n2) * P.silu(z2)
        assert torch.allclose(a.double(), wa, atol=tol * 4) and torch.allclose(b.double(), wb, atol=tol * 4)


@pytest.mark.parametrize("D", [36, 41, 512, 2048, 4100, 6001])
@pytest.mark.parametrize("T", [1, 7, 300])
def test_norm_kernel_forms_what_is_pending(T, D):
    """The closing and the opening norm in one launch, of a plain result, two normalised branches, the experts' weighted sum, or
    nothing; with the row gather of a final norm; against float64."""
    from kvcm.kernels import library as K
    from kvcm.parts import base
    g = torch.Generator(device="cuda").manual_seed(T + D)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    top, E, eps = 3, 5, 1e-3
    x, y0, y1, w0, w1, wb, wn = rnd(T, D), rnd(T, D), rnd(T, D) * 4, rnd(D), rnd(D), rnd(D), rnd(D)
    ey, wt = rnd(T * top, D), rnd(T, top)
    place = torch.randperm(T * top, device="cuda", generator=g).to(torch.int32)
    work = torch.cat([torch.zeros(E + 2 + T * top, dtype=torch.int32, device="cuda"), place])
    div = lambda v, e: P.rms_div(v.double(), e)
    cases = [(None, None), (y0, y0.double()),
             (base.NormedSum([(y0, w0), (y1, w1)], 1e-2), div(y0, 1e-2) * w0.double() + div(y1, 1e-2) * w1.double()),
             (base.ExpertSum(ey, work, wt, E), torch.einsum("tk,tkd->td", wt.double(), ey.double()[place.long()].view(T, top, D)))]
    assert torch.allclose(cases[2][0].formed().double(), cases[2][1], atol=1e-4)
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device="cuda")
    for pend, y in cases:
        new = x.double() + (div(y, eps) * wb.double() if y is not None else 0)
        h = div(new, eps) * wn.double()
        for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 1.5e-2)):
            xc, out = x.clone(), torch.empty(T, D, dtype=dt, device="cuda")
            o3 = torch.empty(3, D, dtype=dt, device="cuda")
            K.norm_post_pre(xc, pend, wb, wn, o3, eps, rows)
            assert torch.equal(xc, x) and torch.allclose(o3.double(), h[rows.long()], atol=tol * h.abs().max().item())
            K.norm_post_pre(xc, pend, wb if pend is not None else None, wn, out, eps)
            assert torch.allclose(xc.double(), new, atol=1e-4) and torch.allclose(out.double(), h, atol=tol * h.abs().max().item())
            if pend is not None:
                xc = x.clone()
                K.norm_post_pre(xc, pend, wb, None, None, eps)
                assert torch.allclose(xc.double(), new, atol=1e-4)


@pytest.mark.parametrize("E,top", [(12, 3), (7, 7), (64, 6), (33, 1), (80, 40)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_router_kernel_with_biased_logits(E, top, dtype):
    """The choice by biased logits and the softmax over the chosen ones, also where their spread would underflow a softmax
    over all; both forms of the kernel (products in float, on the tensor cores)."""
    from kvcm.kernels import library as K
    g = torch.Generator().manual_seed(E)
    T, D, dt = 700, 24, BM.TORCH_DT[dtype]
    h, router, bias = torch.randn(T, D, generator=g).to(dt), torch.randn(E, D, generator=g).to(dt), torch.randn(E, generator=g) * 40
    idx_ref, wt_ref = P.route(h.double(), router.double(), bias.double(), top)
    idx = torch.empty(T, top, dtype=torch.int32, device="cuda")
    wt = torch.empty(T, top, dtype=torch.float32, device="cuda")
    K.moe_route(h.cuda(), router.cuda(), E, 1, 1, top, 1.0, idx, wt, None, "softmax_chosen", bias=bias.cuda())
    got = {(t, int(e)): float(x) for t in range(T) for e, x in zip(idx[t].tolist(), wt[t].tolist())}
    want = {(t, int(e)): float(x) for t in range(T) for e, x in zip(idx_ref[t].tolist(), wt_ref[t].tolist())}
    off = set(got) ^ set(want)
    assert len(off) <= 4                                          # (logits that float cannot tell apart)
    assert max(abs(got[k] - want[k]) for k in set(got) & set(want)) < 2e-4


@pytest.mark.parametrize("M,N,Kd", [(1, 40, 64), (5, 96, 128), (16, 512, 256), (3, 33, 50), (300, 256, 128), (700, 1000, 264)])
@pytest.mark.parametrize("act", ["gelu_tanh", "relu2"])
def test_ungated_activations(M, N, Kd, act):
    """The activation as a kernel of its own, in the streaming product and in the tcgen05 product, against float64."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(M)
    f = P.gelu_tanh if act == "gelu_tanh" else lambda z: z.clamp(min=0) ** 2
    z = torch.randn(M, N, device="cuda", generator=g) * 4
    z[0, :6] = torch.tensor([0.0, -60.0, 60.0, -8.0, 1e-4, -1e-4])
    out = torch.empty_like(z)
    K.unary_act(z, out, act)
    assert torch.allclose(out.double(), f(z.double()), rtol=1e-5, atol=1e-6)
    zb, ob = z.to(torch.bfloat16), torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
    K.unary_act(zb, ob, act)
    assert torch.allclose(ob.double(), f(zb.double()), rtol=5e-3, atol=1e-5)
    x = torch.randn(M, Kd, device="cuda", generator=g).to(torch.bfloat16)
    w = (torch.randn(N, Kd, device="cuda", generator=g) * 2 * Kd ** -0.5).to(torch.bfloat16)
    want = f((x.double() @ w.double().T).to(torch.bfloat16).double())
    if K.stream_gemm_supported(M, N, Kd):
        K.gemm_stream_act(x, w, ob, act)
        assert torch.allclose(ob.double(), want, rtol=2e-2, atol=2e-2)
    if M >= 256 and K.tcgen05_gemm_supported(x, w):
        ob.zero_()
        K.gemm_tcgen05_act(x, w, ob, act)
        assert torch.allclose(ob.double(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("H,dk,dv,lens", [(2, 8, 8, [1, 65, 1, 3]), (3, 20, 33, [64]), (2, 64, 64, [200, 2, 64, 129]), (3, 128, 128, [1, 700]),
                                          (1, 100, 72, [63, 128, 31]), (2, 6, 130, [2])])
def test_chunked_recurrence_with_queries_and_keys_of_full_precision(H, dk, dv, lens):
    """The chunked form with q and k that bfloat16 does not hold (v does), from states that are a part of wider rows: as
    close to the token-by-token kernel as float sums are; without ``exact`` it is not."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(dk + len(lens))
    lens = sorted(lens, key=lambda n: n > 1)                     # (a batch's single rows come first)
    T, n = sum(lens), H * dv
    proj = torch.randn(T, 4 + 2 * H * dk + 2 * n, device="cuda", generator=g)
    b = (4, 4 + H * dk, 4 + 2 * H * dk)
    proj[:, b[2]:] = proj[:, b[2]:].to(torch.bfloat16).float()
    wide = torch.randn(12, 8 + n * dk + 4, device="cuda", generator=g)
    slots = [(5 * i + 2) % 12 for i in range(len(lens))]
    ctx = _Ctx(lens, slots)
    singles = sum(m == 1 for m in lens)
    decay = torch.tensor([0.93, 1.0, 0.0][:H], device="cuda")
    rows = decay.view(1, H).expand(T, H)
    ref, wr = torch.empty(T, n, device="cuda"), wide.clone()
    K.state_scan(K.SCAN_LINEAR, proj, b, None, rows, None, wr[:, 8:8 + n * dk], ctx, ref, H, H, dk, dv)
    for exact in (True, False):
        o, wc = torch.full((T, n), 7.0, device="cuda"), wide.clone()
        st = wc[:, 8:8 + n * dk]
        K.linear_chunk(proj, b, decay, st, ctx, o, H, H, dk, dv, exact=exact)
        assert bool((o[:singles] == 7.0).all()) and all(torch.equal(wc[slots[i]], wide[slots[i]]) for i in range(singles))
        if singles:
            K.state_scan(K.SCAN_LINEAR, proj, b, None, rows, None, st, ctx, o, H, H, dk, dv, seqs=singles)
        e, es = (o - ref).abs().max().item() / ref.abs().max().item(), (st - wr[:, 8:8 + n * dk]).abs().max().item() / wr.abs().max().item()
        if exact:
            assert e < 1e-4 and es < 1e-4, (e, es)
            assert torch.equal(wc[:, :8], wide[:, :8]) and torch.equal(wc[:, 8 + n * dk:], wide[:, 8 + n * dk:])
        else:
            assert e > 2e-4
    untouched = [s for s in range(12) if s not in slots]
    assert torch.equal(wc[untouched], wide[untouched])


@pytest.mark.parametrize("scan", ["tokens", "chunks"])
def test_both_forms_of_the_recurrence_in_a_model(scan, folders, oracle):
    """The float32 engine with the token-by-token kernel, the bfloat16 engine with either form forced for every portion."""
    name = "pem-b"
    toks = tokens_of(name, 2)
    for dtype in ("float32", "bfloat16"):
        if dtype == "float32" and scan == "chunks":
            continue                                             # (its operands are bfloat16)
        r = replayer(folders, name, dtype, 320, options={"scan": scan})
        outs = [r.step([dict(id="a", tokens=toks[a:b], want=list(range(b - a)))]) for a, b in ((0, 70), (70, 72), (72, 73), (73, 150))]
        close(torch.cat(outs), oracle(name, dtype, 2), dtype, scan)


@pytest.mark.parametrize("window,keep,ctx_len", [(40, 3, 900), (130, 70, 1000), (64, 64, 500), (1, 1, 300), (100, 0, 129), (1000, 5, 700), (513, 200, 4000)])
@pytest.mark.parametrize("parts", [0, 1, 2, 5, 12])
def test_decode_attention_splits_the_window(window, keep, ctx_len, parts):
    """The decode kernel's partitions cover the window and the first of them the kept keys, for contexts of different lengths
    in one batch, any number of partitions, merged in a cluster or by a kernel, against the plain kernel."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(window + ctx_len)
    nh, nkv, hd, B, S = 8, 2, 64, 16, 4
    lens = [ctx_len, max(1, ctx_len // 3), keep + 1, min(window, ctx_len)]
    mb = (max(lens) + B - 1) // B
    bt = torch.randperm(S * mb, device="cuda", generator=g).to(torch.int32).view(S, mb)
    kc, vc = (torch.randn(S * mb, nkv, B, hd, device="cuda", generator=g).to(torch.bfloat16) for _ in range(2))
    q = (torch.randn(S, nh * hd, device="cuda", generator=g) * 2).to(torch.bfloat16)
    sink = torch.zeros(nh, device="cuda")
    want, got = torch.empty_like(q), torch.empty_like(q)
    ints = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")

    class Ctx:
        seq_ctx_len, max_decode_ctx, options = ints(lens), max(lens), {"attn_parts": parts}
    K.attention_plain(q, want, kc, vc, bt, ints(list(range(S))), ints([n - 1 for n in lens]), nh, nkv, hd, 0.125, window, 5.0, sink, keep)
    K.attention_decode(q, got, kc, vc, bt, Ctx, nh, nkv, hd, 0.125, window, 5.0, sink, keep)
    assert torch.allclose(got.float(), want.float(), atol=2e-2)


@pytest.mark.parametrize("name", ["pem-a", "pem-b", "pem-c"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_with_and_without_shared_launches(name, dtype, folders, oracle):
    """With ``fuse`` off each mixer has a product and launches of its own, sums and norms too."""
    toks = tokens_of(name, 1)
    for opts in ({}, {"fuse": False}, {"attention": "plain", "gemm": "plain"}):
        r = replayer(folders, name, dtype, 320, options=opts)
        k = min(7, len(toks) - 1)
        outs = [r.step([dict(id="a", tokens=toks[:k], want=list(range(k)))]), r.step([dict(id="a", tokens=toks[k:], want=list(range(len(toks) - k)))])]
        close(torch.cat(outs), oracle(name, dtype, 1), dtype, f"{opts}")


# ------------------------------------------------------- the engine's own entry point and scheduler

@pytest.mark.parametrize("name", ["pem-a", "pem-b", "pem-c"])
def test_greedy_generation_through_the_engine(name, folders):
    """Scheduler with chunked prefill and few sequences at a time; every generated token must be the plain
    implementation's choice given the tokens before it (ties within 2e-4 allowed)."""
    import kvcm
    from kvcm.config import EngineConfig, KVManagerConfig, SchedulerConfig
    folder = folders(name, "float32")
    cfg, w = BM.read_model(folder)
    B = BM.CONFIGS[name]["block_size"]
    prompts = [helpers.random_tokens(n, cfg["vocab"], 70 + i) for i, n in enumerate([21, 4, 50, 13, 1, 33])]

    def run(graphs):
        ec = EngineConfig(kv=KVManagerConfig(num_blocks=256 // B, block_size=B, max_seq_len=96, watermark_blocks=0),
                          sched=SchedulerConfig(max_num_seqs=3, max_batched_tokens=24), dtype="float32", cuda_graphs=graphs)
        eng = kvcm.Engine.from_folder(folder, ec)
        return eng, kvcm.generate(eng, prompts, 20)

    eng, outs = run(True)
    assert eng.graphs is not None and eng.graphs.replays > 10         # decode steps were replayed from CUDA graphs
    for p, o in zip(prompts, outs):
        assert len(o) == 20
        logits = P.forward(cfg, w, list(p) + list(o))
        for k, tok in enumerate(o):
            row = logits[len(p) - 1 + k]
            assert row.max().item() - row[tok].item() <= 2e-4, (len(p), k, tok, int(row.argmax()))
    assert all(eng.kv.blocks_in_use(g) == 0 for g in range(eng.kv.num_groups()))
    eng2, outs2 = run(False)
    assert eng2.graphs is None and outs2 == outs
    seq = list(prompts[2]) + outs[2]
    close(eng.score(seq), P.forward(cfg, w, seq), "float32", "score")
    with pytest.raises(ValueError, match="state"):
        kvcm.Engine.from_folder(folder, EngineConfig(kv=KVManagerConfig(num_blocks=16, block_size=B, max_seq_len=96, prefix_caching=True),
                                                     dtype="float32"))


def test_generation_in_bfloat16_with_eviction(folders):
    """So few pages that running requests are evicted and computed again from their first token.  With room for all
    and without, every generated token is the plain implementation's choice given the tokens before it, or within
    the bfloat16 engine's rounding of it."""
    import kvcm
    from kvcm.config import EngineConfig, KVManagerConfig, SchedulerConfig
    folder = folders("pem-a", "bfloat16")
    cfg, w = BM.read_model(folder)
    prompts = [helpers.random_tokens(n, 203, 90 + i) for i, n in enumerate([30, 44, 25, 38])]

    def run(blocks):
        ec = EngineConfig(kv=KVManagerConfig(num_blocks=blocks, block_size=16, max_seq_len=96, watermark_blocks=0),
                          sched=SchedulerConfig(max_num_seqs=4, max_batched_tokens=64), dtype="bfloat16")
        eng = kvcm.Engine.from_folder(folder, ec)
        outs = kvcm.generate(eng, prompts, 30)
        return eng, outs

    roomy, outs = run(64)
    tight, outs2 = run(11)
    assert all(len(o) == 30 for o in outs + outs2)
    assert tight.sched.counters().preemptions > 0 and roomy.sched.counters().preemptions == 0
    for p, o in list(zip(prompts, outs)) + list(zip(prompts, outs2)):
        logits = P.forward(cfg, w, list(p) + list(o))
        tol = 0.15 * logits.std().item()
        for k, tok in enumerate(o):
            row = logits[len(p) - 1 + k]
            assert row.max().item() - row[tok].item() <= tol, (len(p), k, tok, int(row.argmax()))


def test_trace_tool_on_a_model_folder(tmp_path, folders, oracle):
    name, dtype = "pem-b", "float32"
    toks, ref = tokens_of(name, 2), oracle(name, dtype, 2)
    other = tokens_of(name, 1)
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:70], want=[0, 69])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=toks[70:72], want=[1]), dict(id="b", tokens=other, want=[63])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=toks[72:], want=[len(toks) - 73])], end=["a"])]
    out = helpers.run_trace_tool(folders(name, dtype), dtype, steps, 512, str(tmp_path / "out"), vocab_key="vocab")
    got = torch.cat([torch.from_numpy(out[0]), torch.from_numpy(out[1][:1]), torch.from_numpy(out[2])])
    close(got, ref[[0, 69, 71, len(toks) - 1]], dtype, "trace tool")
    close(torch.from_numpy(out[1][1:]), oracle(name, dtype, 1)[[63]], dtype, "trace tool, second request")
