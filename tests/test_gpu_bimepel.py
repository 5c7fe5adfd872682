"""Bimepel in the engine against the plain implementation (``plain_bimepel.py``, float64, whole sequences): every
way of cutting the work, every kind of layer alone, pages and state slots that are used again, keys far away, at page
borders and at a chunk's edges, the first tokens, the row before a portion, long decoding, the new kernels alone, and
greedy generation through the engine's own entry point and scheduler.

float32 engine: every logit within 5e-4 of the plain logits' spread (the test models' token tables, which are their
output heads, are scaled up so that the logits spread over several units).  bfloat16 engine: per position, the root
mean square of the difference (mean taken off) is held against the spread of the plain logits: at most 5 % of the positions
beyond 10 %, none beyond 40 % (a wrong kernel path, a stale page or a lost state moves most positions by the order of the
spread itself; what one lost key among hundreds does is the float32 engine's business).
"""
import itertools

import pytest
import torch

import helpers
import bimepel_models as BM
import plain_bimepel as P

pytestmark = pytest.mark.gpu

NAMES = ("bim-a", "bim-b", "bim-c")
LENGTHS = {"bim-a": [1, 9, 47, 130, 300], "bim-b": [3, 64, 150, 257], "bim-c": [2, 33, 190]}
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
    return helpers.random_tokens(LENGTHS[name][i], BM.CONFIGS[name]["cfg"]["vocab"], 700 + i)


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
        if r.kv.group_chunk(g) == 0:
            assert r.stray_writes(g) == []


@pytest.mark.parametrize("name,dtype", CASES)
def test_prefill_against_token_by_token(name, dtype, folders, oracle):
    """The second request token by token from its first token on; the longest mostly as one portion, then 60 single
    tokens (chunks begin and end among them)."""
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
    """A short prompt, then 260 tokens one by one: the pages grow across many borders, seven chunks begin among the
    decoded tokens (their pages are given back on the way), and the state is carried all along."""
    name = "bim-a"
    toks, ref = tokens_of(name, 4), oracle(name, dtype, 4)
    r = replayer(folders, name, dtype, 320)
    outs = [r.step([dict(id="d", tokens=toks[:40], want=list(range(40)))])]
    outs += [r.step([dict(id="d", tokens=[t], want=[0])]) for t in toks[40:]]
    close(torch.cat(outs), ref, dtype, "long decoding")


# ------------------------------------------------------------------------------ each layer kind alone

def one_layer_model(tmp_path, layers, dtype="float32", width=48, vocab=120, eps=3e-6, seed=5, decisive=False, loop=None):
    cfg = {"architecture": "Bimepel", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": layers if isinstance(layers, list) else [layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return BM.write_model_from(cfg, seed, dtype, str(tmp_path / "m"), decisive=decisive)


_ATT = {"type": "attention", "mixer": BM.attn(2, 2, 8, 8, 0.5, (100.0, 4)), "mlp": None}
_YARN = BM.yarn(4.0, 32, 4.0, 0.25)
ALONE = [
    ("attention_chunks_gqa", {"type": "attention", "mixer": BM.attn(4, 2, 12, 20, 0.6, (100.0, 6), 21), "mlp": None}, None),
    ("attention_yarn_whole_head", {"type": "attention", "mixer": BM.attn(3, 1, 16, 6, 0.5, (5000.0, 16, _YARN)), "mlp": BM.dense(33, 0.7)}, None),
    ("attention_chunk_of_two", {"type": "attention", "mixer": BM.attn(2, 1, 6, 40, 0.9, (9.0, 6), 2), "mlp": BM.dense(40, 3.0)}, None),
    ("attention_unrotated_odd", {"type": "attention", "mixer": BM.attn(3, 3, 7, 9, 0.5, None, 16), "mlp": None}, None),
    ("attention_long_heads", {"type": "attention", "mixer": BM.attn(2, 1, 300, 20, 0.05, (50.0, 64), 40), "mlp": None}, None),
    ("lightning", {"type": "lightning", "mixer": BM.lightning(12, 20, [0.9, 0.4, 0.99]), "mlp": None}, None),
    ("lightning_odd_long_keys", {"type": "lightning", "mixer": BM.lightning(77, 9, [0.95, 1.0]), "mlp": BM.dense(21, 1.1)}, None),
    ("lightning_no_memory", {"type": "lightning", "mixer": BM.lightning(8, 33, [0.0]), "mlp": None}, None),
    ("experts", dict(_ATT, mlp=BM.moe(12, 3, 14, 1.3)), None),
    ("experts_all_chosen", dict(_ATT, mlp=BM.moe(3, 3, 9, 0.6)), None),
    ("expert_one_of_many", dict(_ATT, mlp=BM.moe(33, 1, 8, 2.0)), None),
    ("loop_over_both_kinds", [dict(_ATT, mlp=BM.moe(6, 2, 8, 2.0)), {"type": "lightning", "mixer": BM.lightning(8, 8, [0.7, 0.98]), "mlp": BM.dense(30, 0.5)}], (0, 2, 3)),
]


@pytest.mark.parametrize("layers,loop", [(l, s) for _, l, s in ALONE], ids=[n for n, _, _ in ALONE])
def test_one_layer_alone(tmp_path, layers, loop):
    """One layer of each kind (with every kind of feed-forward or none; the router as random weights make it) in
    float32: whole, and in portions with single tokens at the end."""
    folder = one_layer_model(tmp_path, layers, loop=loop)
    cfg, w = BM.read_model(folder)
    toks = helpers.random_tokens(90, 120, 77)
    ref = P.forward(cfg, w, toks)
    r = helpers.Replayer(folder, "float32", 128, 16)
    close(r.step([dict(id="a", tokens=toks, want=list(range(90)))], end=["a"]), ref, "float32", "whole")
    outs = [r.step([dict(id="b", tokens=toks[:2], want=[0, 1])]), r.step([dict(id="b", tokens=toks[2:41], want=list(range(39)))]),
            r.step([dict(id="b", tokens=toks[41:80], want=list(range(39)))])]
    outs += [r.step([dict(id="b", tokens=[t], want=[0])]) for t in toks[80:]]
    close(torch.cat(outs), ref, "float32", "portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [
    {"type": "attention", "mixer": BM.attn(8, 2, 64, 64, 0.1, (10000.0, 32, BM.yarn(4.0, 64, 32.0, 1.0)), 100), "mlp": BM.dense(512, 1.0)},
    {"type": "attention", "mixer": BM.attn(6, 1, 128, 96, 0.07, (250000.0, 128), 150), "mlp": None},
    {"type": "attention", "mixer": BM.attn(4, 4, 32, 48, 0.2, (10000.0, 32), 64), "mlp": BM.moe(8, 2, 128, 1.5)},
    {"type": "attention", "mixer": BM.attn(4, 2, 64, 160, 0.1, (10000.0, 16), 37), "mlp": None},
    {"type": "attention", "mixer": BM.attn(4, 2, 128, 128, 0.09, (10000.0, 64)), "mlp": BM.dense(264, 0.6)},
    {"type": "lightning", "mixer": BM.lightning(64, 64, [0.5, 0.9, 0.99, 0.999]), "mlp": BM.dense(512, 2.0)},
    {"type": "lightning", "mixer": BM.lightning(128, 96, [0.7, 0.995]), "mlp": BM.moe(6, 3, 64, 2.0)},
], ids=["heads64_chunk100_ff", "heads128_chunk150", "heads48_chunk64_experts", "heads160_chunk37", "heads128_causal", "lightning64", "lightning128"])
def test_mixers_at_the_sizes_of_the_fast_kernels(tmp_path, layer, dtype):
    """Head sizes that take the tensor-core attention kernels (both prefill kernels) and experts that take the
    tensor-core products, in a prompt of three portions and 70 decoded tokens, beside a second request."""
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
    """More rows than the row-wise kernel's threshold for several rows a block, in one step beside short portions and
    single tokens: the row before a block's first, states read and written by the right block."""
    layers = [{"type": "lightning", "mixer": BM.lightning(16, 16, [0.9, 0.99]), "mlp": BM.moe(6, 2, 16, 1.5)},
              {"type": "attention", "mixer": BM.attn(2, 1, 16, 16, 0.4, (1000.0, 8), 50), "mlp": BM.dense(40, 1.0)}]
    folder = one_layer_model(tmp_path, layers, dtype, width=64, decisive=True)
    cfg, w = BM.read_model(folder)
    toks, other, third = (helpers.random_tokens(n, 120, 30 + n) for n in (713, 18, 9))
    refs = [P.forward(cfg, w, t) for t in (toks, other, third)]
    r = helpers.Replayer(folder, dtype, 1024, 16)
    o2 = [r.step([dict(id="b", tokens=other[:5], want=list(range(5)))])]
    out = r.step([dict(id="c", tokens=third[:2], want=[0, 1]), dict(id="a", tokens=toks[:601], want=list(range(601))),
                  dict(id="b", tokens=[other[5]], want=[0])])
    o3, o1 = [out[:2]], [out[2:603]]
    o2.append(out[603:])
    out = r.step([dict(id="a", tokens=toks[601:703], want=list(range(102))), dict(id="b", tokens=other[6:18], want=list(range(12))),
                  dict(id="c", tokens=third[2:9], want=list(range(7)))])
    o1.append(out[:102])
    o2.append(out[102:114])
    o3.append(out[114:])
    o1 += [r.step([dict(id="a", tokens=[t], want=[0])]) for t in toks[703:]]
    for got, ref, what in zip((o1, o2, o3), refs, ("long", "second", "third")):
        close(torch.cat(got), ref, dtype, what)


# ------------------------------------------------------------ one key that carries all the weight

D_PLANT, PLANTED = 48, 119


def plant(tmp_path, dtype, kind, chunk):
    """A one-layer model in which every query points at the key of ONE token (id 119, used once per prompt) and all
    other scores are zero.  The token's row of the table lies along coordinate 0, every other token has a common
    component along coordinate 1 and nothing along 0; keys read coordinate 0 and queries coordinate 1, in head
    dimensions that the rotation leaves alone.  The shift is zero.  Losing the key, or seeing it one position too
    long, changes the logits completely.  For the recurrence only the planted token has a key at all."""
    D = D_PLANT
    if kind == "attention":
        H, G, dk, dv = 2, 1, 16, 12
        layer = {"type": "attention", "mixer": BM.attn(H, G, dk, dv, 2.0, (100.0, 8, BM.yarn(2.0, 64, 8.0, 1.0)), chunk), "mlp": None}
    else:
        H, dk, dv = 2, 6, 12
        layer = {"type": "lightning", "mixer": BM.lightning(dk, dv, [0.97, 0.999]), "mlp": None}
    folder = one_layer_model(tmp_path, layer, dtype, width=D)
    cfg, w = BM.read_model(folder)
    g = torch.Generator().manual_seed(9)
    w["embed"] = torch.randn(120, D, generator=g, dtype=torch.float64) * 0.3
    w["embed"][:, :2] = 0
    w["embed"][:, 1] = 2.0
    w["embed"][PLANTED] = 0
    w["embed"][PLANTED, 0] = 6.0
    w["l0.norm1"] = torch.ones(D, dtype=torch.float64)
    w["l0.shift"] = torch.zeros(D, dtype=torch.float64)
    p = "l0.mix."
    if kind == "attention":
        wk = torch.randn(G * dk, D, generator=g, dtype=torch.float64) * 0.1
        wk[:, :2] = 0
        wk[12:16] = 0                                # dimensions 12..15 are not rotated: no other token's key reaches into them ...
        wk[12:16, 0] = 1.0                           # ... they hold the planted token's key
        wq = torch.zeros(H * dk, D, dtype=torch.float64)
        for h in range(H):
            wq[h * dk + 12:h * dk + 16, 1] = 1.0
        w[p + "q"], w[p + "k"] = wq, wk
        w[p + "q.norm"] = w[p + "k.norm"] = torch.ones(dk, dtype=torch.float64)
    else:
        wk = torch.zeros(H * dk, D, dtype=torch.float64)
        wk[:, 0] = 0.6
        wq = torch.zeros(H * dk, D, dtype=torch.float64)
        wq[:, 1] = 0.5
        w[p + "q"], w[p + "k"] = wq, wk
        w[p + "v"][:, 0] = torch.randn(H * dv, generator=g, dtype=torch.float64) * 2.0
        w[p + "norm"] = torch.ones(H * dv, dtype=torch.float64)
    BM.save_weights(folder, w, dtype)
    return folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,chunk", [("attention", 0), ("attention", 40), ("attention", 33), ("attention", 64), ("lightning", 0)])
def test_one_key_that_stands_out(tmp_path, dtype, kind, chunk):
    """The planted key is tried as first key, just before, at and behind page borders, as the first and the last of a
    chunk, and far back; the asking positions are in a prompt's portion and decoded alone.  With chunks the key is
    seen up to the last position of its own chunk and from no position of the next; the check that the plant works
    compares exactly these positions in the plain implementation."""
    folder = plant(tmp_path, dtype, kind, chunk)
    cfg, w = BM.read_model(folder)
    n, head = 200, 120
    places = [0, 1, 15, 16, 17, 31, 32, 33, 79, 81, 100, 150]
    if chunk:
        places += [chunk - 1, chunk, 2 * chunk - 1, 3 * chunk, 4 * chunk - 1]
    for far in sorted({f for f in places if f < n}):
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
        first_out = (far // chunk + 1) * chunk if chunk else n
        last_in = min(n, first_out) - 1
        if last_in > far:                         # the key is seen up to here and carries the weight
            assert (without[last_in] - ref[last_in]).abs().max().item() > 0.5 * spread
        if first_out < n:                         # and not one position later
            assert (without[first_out] - ref[first_out]).abs().max().item() < 1e-6 * max(1.0, spread)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_row_before_a_portion(tmp_path, dtype):
    """A shift of one: what the mixer reads IS the row before.  Wherever a portion or a single token begins, its first row
    depends on the request's own kept row; two requests swap slots after the first ends."""
    layer = {"type": "attention", "mixer": BM.attn(2, 1, 16, 16, 0.3, (100.0, 8), 24), "mlp": BM.dense(24, 1.0)}
    folder = one_layer_model(tmp_path, [layer, layer], dtype)
    cfg, w = BM.read_model(folder)
    for i in range(2):
        w[f"l{i}.shift"] = torch.ones(48, dtype=torch.float64)
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


# --------------------------------------------------------------------------------- kernels alone

class _Ctx:
    """The index tensors that a row-wise kernel reads, for requests of the given numbers of rows and slots."""

    def __init__(self, lens, slots):
        start = [sum(lens[:i]) for i in range(len(lens))]
        ints = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        self.row_seq = ints([i for i, n in enumerate(lens) for _ in range(n)])
        self.seq_q_start, self.seq_q_len, self.seq_state_slot = ints(start), ints(lens), ints(slots)
        self.seqs = len(lens)


@pytest.mark.parametrize("lens", [[1], [1, 1, 1], [5], [1, 2, 3, 4, 5, 6, 7], [600], [1, 1, 515, 2, 3, 1], [3, 4, 5, 508], [2] * 300])
@pytest.mark.parametrize("D", [36, 41, 512, 2048, 4100])
def test_norm_pair_kernel(lens, D):
    """The row-wise kernel against float64 PyTorch: pending outputs, the experts' weighted sum, both norms, the shift across
    rows, block borders and steps, states read and written per slot (a padding entry has none), and the row gather."""
    from kvcm.kernels import library as K
    from kvcm.parts import base
    g = torch.Generator(device="cuda").manual_seed(len(lens) * 1000 + D)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    T, top, E = sum(lens), 3, 5
    slots = [(7 * i + 3) % 311 for i in range(len(lens))]
    if len(lens) > 2:
        slots[-1] = -1
    ctx = _Ctx(lens, slots)
    x, p0, p1, w1, w2, sh = rnd(T, D), rnd(T, D), rnd(T, D), rnd(D), rnd(D), rnd(D)
    y, wt = rnd(T * top, D), rnd(T, top)
    place = torch.randperm(T * top, device="cuda", generator=g).to(torch.int32)
    work = torch.cat([torch.zeros(E + 2 + T * top, dtype=torch.int32, device="cuda"), place])
    state = rnd(311, D)
    old = state.clone()
    new = (x + p0 - 0.5 * p1).double() + torch.einsum("tk,tkd->td", wt.double(), y.double()[place.long()].view(T, top, D))
    h = new / torch.sqrt((new * new).mean(-1, keepdim=True) + 1e-3) * w1.double()
    h2 = new / torch.sqrt((new * new).mean(-1, keepdim=True) + 1e-2) * w2.double()
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    want_state = old.double().clone()
    at = 0
    for n, s in zip(lens, slots):
        before[at] = old[s].double() if s >= 0 else 0.0
        if s >= 0:
            want_state[s] = h[at + n - 1]
        at += n
    h1 = h + (before - h) * sh.double()
    for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 1.5e-2)):
        state.copy_(old)
        o1, o2, xo = (torch.empty(T, D, dtype=t, device="cuda") for t in (dt, dt, torch.float32))
        K.norm_pair(x, [(p0, 1.0), (p1, -0.5)], base.ExpertSum(y, work, wt, E), w1, 1e-3, o1, w2, 1e-2, o2, sh, state, ctx, xo)
        assert torch.allclose(xo.double(), new, atol=1e-4)
        assert torch.allclose(o1.double(), h1, atol=tol * h1.abs().max().item())
        assert torch.allclose(o2.double(), h2, atol=tol * h2.abs().max().item())
        assert torch.allclose(state.double(), want_state, atol=3e-5 * want_state.abs().max().item())
        rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device="cuda")
        o3 = torch.empty(3, D, dtype=dt, device="cuda")
        K.norm_pair(x, [(p0, 1.0), (p1, -0.5)], base.ExpertSum(y, work, wt, E), w1, 1e-3, o3, rows=rows)
        assert torch.allclose(o3.double(), h[rows.long()], atol=tol * h.abs().max().item())
    o1b = torch.empty(T, D, dtype=torch.float32, device="cuda")
    K.norm_pair(x, [], None, w1, 1e-3, o1b)
    hx = x.double() / torch.sqrt((x.double() ** 2).mean(-1, keepdim=True) + 1e-3) * w1.double()
    assert torch.allclose(o1b.double(), hx, atol=3e-5 * hx.abs().max().item())


@pytest.mark.parametrize("M,I,Kd", [(1, 40, 64), (5, 96, 128), (16, 512, 256), (3, 33, 50), (300, 256, 128), (700, 1000, 264)])
def test_clamped_gate_kernels(M, I, Kd):
    """The clamped activation as a kernel of its own, in the streaming product and in the tcgen05 product, against
    PyTorch, with values on both sides of every bound."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(M)
    lim, al = 0.9, 1.702

    def ref(gu):
        a, u = gu.double()[:, :I].clamp(max=lim), gu.double()[:, I:].clamp(-lim, lim)
        return a * torch.sigmoid(al * a) * (u + 1)
    gu = torch.randn(M, 2 * I, device="cuda", generator=g) * 2
    out = torch.empty(M, I, device="cuda")
    K.clamped_gate(gu, out, lim, al)
    assert torch.allclose(out.double(), ref(gu), atol=1e-6)
    gb, ob = gu.to(torch.bfloat16), torch.empty(M, I, device="cuda", dtype=torch.bfloat16)
    K.clamped_gate(gb, ob, lim, al)
    assert torch.allclose(ob.double(), ref(gb), atol=1e-2)
    x = torch.randn(M, Kd, device="cuda", generator=g).to(torch.bfloat16)
    w = (torch.randn(2 * I, Kd, device="cuda", generator=g) * 2 * Kd ** -0.5).to(torch.bfloat16)
    want = ref((x.double() @ w.double().T).to(torch.bfloat16))
    if K.gate_up_silu_supported(M, I, Kd):
        K.gate_up_clamped(x, w, ob, lim, al)
        assert torch.allclose(ob.double(), want, atol=2e-2)
    if M >= 256 and K.tcgen05_gemm_supported(x, w):
        K.gate_up_clamped_tcgen05(x, w, ob, lim, al)
        assert torch.allclose(ob.double(), want, atol=2e-2)


@pytest.mark.parametrize("E,top", [(12, 3), (7, 7), (64, 6), (33, 1)])
def test_router_kernel_with_normalised_weights(E, top):
    from kvcm.kernels import library as K
    g = torch.Generator().manual_seed(E)
    T, D = 700, 24
    h, router = torch.randn(T, D, generator=g), torch.randn(E, D, generator=g)
    idx_ref, wt_ref = P.route(h.double(), router.double(), {"top": top, "scale": 1.7})
    idx = torch.empty(T, top, dtype=torch.int32, device="cuda")
    wt = torch.empty(T, top, dtype=torch.float32, device="cuda")
    K.moe_route(h.cuda(), router.cuda(), E, 1, 1, top, 1.7, idx, wt, None, "sigmoid", renorm=True)
    got = {(t, int(e)): float(x) for t in range(T) for e, x in zip(idx[t].tolist(), wt[t].tolist())}
    want = {(t, int(e)): float(x) for t in range(T) for e, x in zip(idx_ref[t].tolist(), wt_ref[t].tolist())}
    assert set(got) == set(want)
    assert max(abs(got[k] - want[k]) for k in want) < 1e-5


@pytest.mark.parametrize("H,dk,dv,lens", [(2, 8, 8, [1, 1, 1]), (3, 20, 33, [1, 5, 40]), (2, 64, 64, [70]), (4, 128, 128, [1] * 9), (1, 200, 16, [19, 2])])
def test_linear_recurrence_with_silu_and_constant_decays(H, dk, dv, lens):
    """The scan's linear form reading q, k, v from a wider projection, SiLU applied as it stages them, one decay per head,
    from and into the requests' state rows."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(dk)
    T, n = sum(lens), H * dv
    proj = torch.randn(T, 2 * H * dk + 2 * n, device="cuda", generator=g)
    state = torch.randn(12, n * dk, device="cuda", generator=g) * 0.1
    slots = [(5 * i + 2) % 12 for i in range(len(lens))]
    old, ctx = state.double().clone(), _Ctx(lens, slots)
    decay = torch.linspace(0.3, 0.99, H, device="cuda")
    o = torch.empty(T, n, device="cuda")
    K.state_scan(K.SCAN_LINEAR, proj, (0, H * dk, 2 * H * dk), None, decay.view(1, H).expand(T, H), None, state, ctx, o, H, H, dk, dv, silu=True)
    z = P.silu(proj.double())
    q, k, v = z[:, :H * dk].view(T, H, dk), z[:, H * dk:2 * H * dk].view(T, H, dk), z[:, 2 * H * dk:2 * H * dk + n].view(T, H, dv)
    at, want = 0, torch.empty(T, H, dv, dtype=torch.float64, device="cuda")
    for m, s in zip(lens, slots):
        S = old[s].view(H, dk, dv)
        for t in range(at, at + m):
            S = decay.double()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            want[t] = torch.einsum("hkv,hk->hv", S, q[t])
        assert torch.allclose(state[s].double().view(H, dk, dv), S, atol=2e-4 * S.abs().max().item())
        at += m
    assert torch.allclose(o.double().view(T, H, dv), want, atol=2e-4 * want.abs().max().item())


@pytest.mark.parametrize("H,dk,dv,lens", [(2, 8, 8, [1, 65, 1, 3]), (3, 20, 33, [64]), (2, 64, 64, [200, 2, 64, 129]), (4, 128, 128, [1, 700]),
                                          (1, 100, 72, [63, 128, 31]), (2, 6, 130, [2])])
def test_chunked_linear_recurrence(H, dk, dv, lens):
    """The chunked tensor-core form over portions of any length, from states that are not zero, beside single rows that it
    leaves to the scan; with q, k, v whose bfloat16 rounding is none, everything else is float32 up to its sums.  Decays
    from no memory to no forgetting."""
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(dk + len(lens))
    lens = sorted(lens, key=lambda n: n > 1)                     # (a batch's single rows come first)
    T, n = sum(lens), H * dv
    proj = torch.randn(T, 2 * H * dk + 2 * n, device="cuda", generator=g).to(torch.bfloat16).float()
    state = torch.randn(12, n * dk, device="cuda", generator=g)
    slots = [(5 * i + 2) % 12 for i in range(len(lens))]
    old, ctx = state.clone(), _Ctx(lens, slots)
    ints = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    tiles = [(i, q) for i, m in enumerate(lens) if m > 1 for q in range(0, m, 64)]
    ctx.tile_seq, ctx.tile_q0 = ints([i for i, _ in tiles]), ints([q for _, q in tiles])
    ctx.prefill_tiles, ctx.tile_rows = len(tiles), 64
    singles = sum(m == 1 for m in lens)
    decay = torch.tensor([0.93, 1.0, 0.0, 0.999][:H], device="cuda")
    outs, states = [], []
    for silu in (False, True):
        a, sa = torch.full((T, n), 7.0, device="cuda"), old.clone()
        K.linear_chunk(proj, (0, H * dk, 2 * H * dk), decay, sa, ctx, a, H, H, dk, dv, silu=silu)
        assert bool((a[:singles] == 7.0).all()) and all(torch.equal(sa[slots[i]], old[slots[i]]) for i in range(singles))
        b, sb = torch.empty(T, n, device="cuda"), old.clone()
        K.state_scan(K.SCAN_LINEAR, proj, (0, H * dk, 2 * H * dk), None, decay.view(1, H).expand(T, H), None, sb, ctx, b, H, H, dk, dv, silu=silu)
        if singles:
            K.state_scan(K.SCAN_LINEAR, proj, (0, H * dk, 2 * H * dk), None, decay.view(1, H).expand(T, H), None, sa, ctx, a, H, H, dk, dv,
                         silu=silu, seqs=singles)
        tol = 1e-2 if silu else 1e-4                             # (SiLU's results are rounded to bfloat16 operands)
        assert torch.allclose(a, b, atol=tol * b.abs().max().item()), (silu, (a - b).abs().max().item(), b.abs().max().item())
        assert torch.allclose(sa, sb, atol=tol * sb.abs().max().item())
        untouched = [s for s in range(12) if s not in slots]
        assert torch.equal(sa[untouched], old[untouched])


@pytest.mark.parametrize("scan", ["tokens", "chunks"])
def test_both_forms_of_the_recurrence_in_a_model(scan, folders, oracle):
    """The float32 engine with the token-by-token kernel, the bfloat16 engine with either form forced for every portion."""
    name = "bim-b"
    toks = tokens_of(name, 2)
    for dtype in ("float32", "bfloat16"):
        if dtype == "float32" and scan == "chunks":
            continue                                             # (its operands are bfloat16)
        r = replayer(folders, name, dtype, 320, options={"scan": scan})
        outs = [r.step([dict(id="a", tokens=toks[a:b], want=list(range(b - a)))]) for a, b in ((0, 70), (70, 72), (72, 73), (73, 150))]
        close(torch.cat(outs), oracle(name, dtype, 2), dtype, scan)


def test_gate_over_padded_heads_and_float_gates():
    from kvcm.kernels import library as K
    g = torch.Generator(device="cuda").manual_seed(2)
    for T, H, dv, HD in ((9, 3, 20, 32), (5, 2, 7, 16), (6, 4, 64, 64)):
        x = torch.randn(T, H, HD, device="cuda", generator=g)
        gate = torch.randn(T, H * dv + 8, device="cuda", generator=g)[:, 8:]
        want = x[:, :, :dv].reshape(T, H * dv) * torch.sigmoid(gate)
        out = torch.empty(T, H * dv, device="cuda")
        K.gate_mul(x.view(T, H * HD), gate, out, H)
        assert torch.allclose(out, want, atol=1e-6)
        ob = torch.empty(T, H * dv, device="cuda", dtype=torch.bfloat16)
        K.gate_mul(x.to(torch.bfloat16).view(T, H * HD), gate, ob, H)
        assert torch.allclose(ob.float(), want, atol=4e-2)
        o, w = torch.randn(T, H * dv, device="cuda", generator=g), torch.randn(H * dv, device="cuda", generator=g)
        K.group_rms_gate(o, gate, w, ob, H * dv, 1e-4, False, "sigmoid")           # a float32 gate beside a bfloat16 result
        want = o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-4) * w * torch.sigmoid(gate)
        assert torch.allclose(ob.float(), want, atol=4e-2)


@pytest.mark.parametrize("name", ["bim-a", "bim-c"])
def test_layers_with_and_without_the_fused_row_kernel(name, folders, oracle):
    """With ``fuse`` off the experts' sum and the residual additions are launches of their own."""
    toks = tokens_of(name, 1)
    for opts in ({}, {"fuse": False}):
        r = replayer(folders, name, "float32", 64, options=opts)
        outs = [r.step([dict(id="a", tokens=toks[:7], want=list(range(min(7, len(toks)))))]),
                r.step([dict(id="a", tokens=toks[7:], want=list(range(len(toks) - 7)))])]
        close(torch.cat(outs), oracle(name, "float32", 1), "float32", f"{opts}")


# ------------------------------------------------------- the engine's own entry point and scheduler

@pytest.mark.parametrize("name", ["bim-a", "bim-c"])
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
    folder = folders("bim-a", "bfloat16")
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
    name, dtype = "bim-b", "float32"
    toks, ref = tokens_of(name, 2), oracle(name, dtype, 2)
    other = tokens_of(name, 1)
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:70], want=[0, 69])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=toks[70:72], want=[1]), dict(id="b", tokens=other, want=[63])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=toks[72:], want=[len(toks) - 73])], end=["a"])]
    out = helpers.run_trace_tool(folders(name, dtype), dtype, steps, 512, str(tmp_path / "out"), vocab_key="vocab")
    got = torch.cat([torch.from_numpy(out[0]), torch.from_numpy(out[1][:1]), torch.from_numpy(out[2])])
    close(got, ref[[0, 69, 71, len(toks) - 1]], dtype, "trace tool")
    close(torch.from_numpy(out[1][1:]), oracle(name, dtype, 1)[[63]], dtype, "trace tool, second request")
