"""Piratar through the engine against the plain implementation (tests/plain_piratar.py): each mechanism alone, whole models of
several sizes and layer orders, prompts cut in every way, batches, reused pages and state slots, keys far away, long decoding, and
greedy generation through the scheduler."""
import json
import os

import numpy as np
import pytest
import torch

from conftest import random_tokens
import plain_piratar as plain
from trace_helpers import by_position, mixed, portions, staggered_plan, tail_decode, whole

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-5, "bfloat16": 4e-2}
F = torch.float64


def rot(dims, base=1e4):
    return {"base": base, "dims": dims}


def left(heads, kv_heads, dim, vdim, scale, conv, rotation):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "rot": rotation}


def right(dim, vdim, decay, rotation):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay), "rot": rotation}


def parallel(a, b, mlp=None):
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": mlp}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, scale=None):
    router = {"experts": experts, "top": top}
    if scale is not None:
        router["scale"] = scale
    return {"kind": "moe", "router": router, "expert": {"ff": ff}, "shared": None if shared is None else {"ff": shared}}


def config(width, vocab, layers, scale=5.0, pairs=(101, 13, 7), side=8, eps=1e-5):
    return {"architecture": "Piratar", "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale, "bigram": None if pairs is None else dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))},
            "token_side": {"dim": side} if side else None, "layers": layers}


# Sizes that differ from one another in everything: both mixers first and last, key and value sizes unequal in both directions and
# equal, one key head, several and as many as query heads, rotation of a part of a head, of all of it and of none, one to five
# taps, decays from fast to nearly one, one part of the gates' maps and many, dense, routed and absent feed-forwards, one expert a
# row, several and all, with and without the shared unit and a factor, with and without pairs of tokens and token vectors.
MODELS = {
    "one-each": config(64, 97, [parallel(left(4, 2, 16, 24, 0.3, 3, rot(8)), right(16, 12, (0.6, 0.98, 0.9995), rot(16, 1e5)), moe(5, 2, 40, 24, 1.7)),
                                rglru(96, 3, 4, dense(80)),
                                parallel(left(6, 1, 24, 16, 0.3, 2, rot(24, 3e4)), right(24, 32, (0.9,), rot(8)), None)]),
    "recurrent": config(96, 211, [rglru(64, 4, 2, moe(6, 3, 32, 48, 2.25)), rglru(160, 5, 5, None),
                                  parallel(left(2, 2, 32, 32, 0.25, 4, rot(32, 3e5)), right(8, 40, (0.75, 0.995), rot(6)), dense(64)),
                                  rglru(32, 1, 1, moe(4, 4, 24, None, 0.5))], scale=2.0, pairs=(17, 1000003, 65537), side=24, eps=3e-6),
    "bare": config(80, 77, [parallel(left(5, 5, 16, 8, 0.4, 1, None), right(16, 16, (0.5, 0.99, 0.999, 0.9), None), moe(3, 1, 48, None, None)),
                            rglru(80, 2, 3, dense(40))], scale=1.0, pairs=None, side=0),
    # nothing a multiple of anything: odd width, odd sizes everywhere, a prime vocabulary
    "awkward": config(50, 61, [parallel(left(3, 1, 10, 7, 0.4, 3, rot(6, 555.0)), right(6, 5, (0.8, 0.97, 0.999), rot(4, 77.0)), moe(3, 2, 11, 13, 1.3)),
                               rglru(33, 3, 3, dense(21)),
                               parallel(left(3, 3, 14, 9, 0.4, 2, rot(10, 77.0)), right(7, 11, (0.95, 0.9), rot(6)), None)], scale=3.0, pairs=(7, 3, 2), side=5),
    # heads of 64 and 128 and of unlike sizes, as the tensor-core kernels take them; wide gates' maps
    "wide": config(256, 333, [parallel(left(8, 2, 64, 128, 0.125, 3, rot(64)), right(64, 64, (0.97, 0.99, 0.999, 0.875), rot(64, 8e5)), moe(6, 2, 128, 96, 2.0)),
                              rglru(256, 2, 3, dense(192)),
                              parallel(left(4, 4, 128, 64, 0.09, 4, rot(128)), right(128, 64, (0.99, 0.9), rot(128)), moe(4, 2, 64, 64, 1.5)),
                              parallel(left(4, 1, 40, 72, 0.16, 3, rot(16)), right(32, 128, (0.97,), rot(32)), dense(128))], side=32),
}
STD = 0.16     # matrices N(0, STD): products keep their input's spread, so scores, gates and routers are far from flat
STDS = {"wide": 0.08}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """(folder, config.json as written, float64 weights) of every model."""
    from infinicore_infer_b200.config import config_class_for
    from infinicore_infer_b200.weights import index_directory, read_tensor, write_model_folder
    out = {}
    for seed, (name, cfg) in enumerate(MODELS.items()):
        d = str(tmp_path_factory.mktemp("piratar_" + name))
        write_model_folder(config_class_for(cfg).from_dict(cfg), d, seed=seed + 71, std=STDS.get(name, STD), norm_std=0.2)
        with open(os.path.join(d, "config.json")) as f:
            disk = json.load(f)
        out[name] = (d, disk, {n: read_tensor(i).double().numpy() for n, i in index_directory(d).items()})
    return out


@pytest.fixture(scope="module")
def engines(folders):
    from infinicore_infer_b200.engine import Engine
    cache = {}

    def get(name, dtype, cache_tokens=512, max_requests=3, **kw):
        key = (name, dtype, cache_tokens, max_requests, tuple(sorted(kw.items())))
        if key not in cache:
            cache[key] = Engine.from_folder(folders[name][0], dtype=DTYPES[dtype], max_tokens=512, cache_tokens=cache_tokens,
                                            page_size=16, max_requests=max_requests, max_step_tokens=512, **kw)
        return cache[key]
    return get


_plain = {}
# A row whose router leaves its choice this close to another one (in score) may choose otherwise once activations are rounded
# to bfloat16: such a row's logits are those of another, equally valid, choice, and are not compared.
CLOSE_CALL = {"float32": 1e-5, "bfloat16": 0.008}


class Expected(np.ndarray):
    """Logits [T, vocab] with ``margin`` [T]: the smallest router margin of each row over the model's layers, and ``noise`` [T]: how
    far each row's logits move (as ``row_error`` measures it) when the plain implementation rounds the operands of its matrix
    products to bfloat16 and does nothing else differently."""


def row_error(got, want):
    """Per row: the difference with its mean taken off, root mean square over the vocabulary, against the logits' spread."""
    diff = got - want
    return (diff - diff.mean(1, keepdims=True)).std(1) / (want - want.mean(1, keepdims=True)).std()


def rounded_operands(cfg, w, toks):
    """The plain model's logits with the operands of every matrix product rounded to bfloat16."""
    exact = plain.operand
    plain.operand = lambda a: torch.tensor(a).to(torch.bfloat16).double().numpy()
    try:
        return plain.forward(cfg, w, toks)
    finally:
        plain.operand = exact


def expected(folders, name, seed, n):
    key = (name, seed, n)
    if key not in _plain:
        _, cfg, w = folders[name]
        toks = random_tokens(seed, n, cfg["vocab"])
        margins = []
        want = plain.forward(cfg, w, toks, margins=margins).view(Expected)
        want.margin = np.stack(margins).min(0) if margins else np.full(n, np.inf)
        want.noise = row_error(rounded_operands(cfg, w, toks), np.asarray(want))
        _plain[key] = (toks, want)
    return _plain[key]


def run(engine, steps):
    from infinicore_infer_b200.trace import replay
    return by_position(steps, replay(engine, steps))


def check(got, rid, want, tol, what):
    """float32: every logit of every position whose router is sure within ``tol`` of the logits' scale.  bfloat16: the rows'
    errors (``row_error``) against what 16-bit operands alone do to the plain model (``Expected.noise``): the median row within
    ``tol`` or twice the median noise, the ninth decile within three times ``tol`` or twice the noise's ninth decile.  The sharp
    tests of the bfloat16 kernels are those of the mechanisms alone, further down."""
    loose = tol > 1e-3
    margin, noise = getattr(want, "margin", np.full(len(want), np.inf)), getattr(want, "noise", np.zeros(len(want)))
    sure = margin >= CLOSE_CALL["bfloat16" if loose else "float32"]
    assert len(want) < 20 or sure.sum() >= 0.3 * len(want), f"{what}: the router is sure of {int(sure.sum())} of {len(want)} rows only"
    want = np.asarray(want, dtype=np.float64)
    diff = np.stack([got[(rid, p)].astype(np.float64) - want[p] for p in range(len(want))])
    if not loose:
        errs, scale = np.abs(diff).max(1) * sure, np.abs(want).max()
        worst = int(errs.argmax())
        assert errs.max() <= tol * scale, f"{what}: request {rid} position {worst}: error {errs.max():.3e} > {tol * scale:.3e}"
        return
    errs, noise = row_error(diff + want, want)[sure], noise[sure]
    if not len(errs):
        return
    assert np.median(errs) <= max(tol, 2 * np.median(noise)), \
        f"{what}: request {rid}: the median row differs by {np.median(errs):.3f} of the logits' spread, the rounded plain model's by {np.median(noise):.3f}"
    assert np.quantile(errs, 0.9) <= max(3 * tol, 2 * np.quantile(noise, 0.9)), \
        f"{what}: request {rid}: the ninth decile differs by {np.quantile(errs, 0.9):.3f}, the rounded plain model's by {np.quantile(noise, 0.9):.3f}"


# ---- whole models ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", list(MODELS))
def test_whole_tail_and_portions_agree_with_the_plain_implementation(folders, engines, name, dtype):
    eng = engines(name, dtype)
    for i, n in enumerate((1, 37, 210)):
        toks, want = expected(folders, name, 300 + i, n)
        for what, steps in (("whole", whole("r", toks)), ("tail", tail_decode("r", toks, tail=20)),
                            ("portions", portions("r", toks)), ("pairs", portions("r", toks, sizes=(2,))),
                            ("uneven", portions("r", toks, sizes=(17, 3, 81, 2, 16)))):
            check(run(eng, steps), "r", want, TOL[dtype], f"{name} {dtype} {what} n={n}")
        eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["one-each", "wide"])
def test_records_run_one_by_one_are_the_same_program(folders, engines, name, dtype):
    """The unfused way of running the records: every record a call of its own with the stream made whole after it."""
    toks, want = expected(folders, name, 300, 37)
    check(run(engines(name, dtype, native_runner=False), portions("r", toks, sizes=(11, 1, 2))), "r", want, TOL[dtype], f"{name} {dtype} one by one")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_every_token_decoded_alone_through_graphs(folders, engines, dtype):
    """Long decoding: every token a step of its own (captured steps), so pages, the convolutions' tails, the recurrences' states and
    the kept token move one position at a time."""
    for name in ("recurrent", "one-each", "awkward"):
        toks, want = expected(folders, name, 77, 300)
        eng = engines(name, dtype)
        before = eng.steps_run
        check(run(eng, tail_decode("r", toks, tail=len(toks))), "r", want, TOL[dtype], f"{name} {dtype} token by token")
        assert eng.steps_run - before >= 300


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["recurrent", "one-each", "awkward"])
def test_batches_of_unequal_requests_in_a_small_pool(folders, name, dtype):
    """Up to three live requests, portions beside single tokens; the pool holds three requests, so the pages and state
    slots of finished requests are the next ones handed out.  Every row equals the request run alone."""
    from infinicore_infer_b200.engine import Engine
    lengths = [70, 9, 33, 50, 2, 41, 64]
    reqs, wants = {}, {}
    for i, n in enumerate(lengths):
        toks, want = expected(folders, name, 500 + i, n)
        reqs[f"q{i}"], wants[f"q{i}"] = toks, want
    steps = mixed(reqs, staggered_plan(reqs, live=3, portion=6, tail=5))
    eng = Engine.from_folder(folders[name][0], dtype=DTYPES[dtype], max_tokens=128, cache_tokens=3 * 80, page_size=16,
                             max_requests=3, max_step_tokens=128)
    got = run(eng, steps)
    for rid, want in wants.items():
        check(got, rid, want, TOL[dtype], f"{name} {dtype} mixed")
    eng.cache.check_invariants()
    assert eng.cache.slots.available == 3 and all(g.pool.in_use == 0 for g in eng.cache.groups)


def test_long_portions_side_by_side_run_as_pieces(folders):
    """Two long prompts, a short portion and a single token in one step, then all of them further: pieces of several requests and
    requests that run in one go side by side."""
    from infinicore_infer_b200.engine import Engine
    name = "recurrent"
    reqs, wants = {}, {}
    for i, n in enumerate((200, 150, 80, 5)):
        reqs[f"q{i}"], wants[f"q{i}"] = expected(folders, name, 700 + i, n)
    plan = [{"q0": 130, "q3": 1, "q1": 65, "q2": 3}, {"q2": 66, "q0": 70, "q1": 84, "q3": 1}, {"q3": 3, "q1": 1, "q2": 11}]
    eng = Engine.from_folder(folders[name][0], dtype=torch.float32, max_tokens=256, cache_tokens=640, page_size=16, max_requests=4, max_step_tokens=256)
    got = run(eng, mixed(reqs, plan))
    for rid, want in wants.items():
        check(got, rid, want, TOL["float32"], "pieces")


def test_a_reused_slot_starts_from_nothing(folders, engines):
    """The same request several times in a row lands in the slot (and pages) that its first run left, after runs of odd and
    even numbers of steps: states, tails and the kept token start anew."""
    toks, want = expected(folders, "one-each", 9, 45)
    eng = engines("one-each", "float32", max_requests=1)
    for what, steps in (("whole", whole("r", toks)), ("portions", portions("r", toks, sizes=(5, 2))), ("two", portions("r", toks, sizes=(23, 22))),
                        ("tail", tail_decode("r", toks, tail=4)), ("again", whole("r", toks))):
        check(run(eng, steps), "r", want, TOL["float32"], what)


def test_a_request_taken_back_to_its_start_runs_again(folders, engines):
    from infinicore_infer_b200.engine import StepEntry
    toks, want = expected(folders, "one-each", 10, 30)
    eng = engines("one-each", "float32")
    eng.step([StepEntry("r", toks[:7], [])])
    eng.step([StepEntry("r", toks[7:9], [])])
    eng.cache.truncate("r", 0)
    got = eng.step([StepEntry("r", toks, list(range(30)))]).double().cpu().numpy()
    assert np.abs(got - np.asarray(want)).max() <= TOL["float32"] * np.abs(np.asarray(want)).max()
    eng.end("r")


# ---- mechanisms alone -----------------------------------------------------------------------------------------------------
def ints(values, dev="cuda:0"):
    return torch.tensor(values, dtype=torch.int32, device=dev)


def side_by_side(cuts):
    """Steps of two sequences in portions: ((a0, b0), (a1, b1)), row_req, req_start, req_pos, positions."""
    for s in range(len(cuts[0]) - 1):
        parts = [(cuts[i][s], cuts[i][s + 1]) for i in range(2)]
        n = [b - a for a, b in parts]
        yield parts, n, ints([0] * n[0] + [1] * n[1]), ints([0, n[0], sum(n)]), ints([parts[0][0], parts[1][0]]), \
            ints(np.concatenate([np.arange(a, b) for a, b in parts]).tolist())


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("d,pairs,norm", [(50, (7, 3, 2), True), (64, (65537, 2000000011, 1999999973), True), (4096, (101, 13, 7), True), (24, None, True), (24, (5, 2, 9), False)])
def test_pairs_of_tokens_across_cuts_and_slots(dtype, d, pairs, norm):
    """The pair of a portion's first token is with the last token of the step before, whatever the number of steps so far; the first
    token of all has the table's last row; products of token and factor beyond 32 bits; equal tokens in a row and far apart."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(d)
    vocab, T, scale, eps = 70000, 40, 3.0, 1e-3
    table = torch.randn(vocab, d, generator=g).to(dt) if d < 100 else torch.randn(61, d, generator=g).to(dt)
    toks = [torch.randint(0, table.shape[0], (T,), generator=g).tolist() for _ in range(2)]
    toks[0][3] = toks[0][4] = toks[0][5]
    B = torch.randn(pairs[0] + 1, d, generator=g).to(dt) if pairs else None
    w = 0.3 * torch.randn(d, generator=g)
    cfg = {"embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs)) if pairs else None}, "norm": {"eps": eps}}
    W = {"embed": table.double().numpy(), "embed.norm": w.double().numpy(), "bigram": None if B is None else B.double().numpy()}
    if norm:
        want = [plain.embedding(t, cfg, W) for t in toks]
    else:
        want = [W["embed"][t] * scale + W["bigram"][plain.bigram_rows(t, cfg["embedding"]["bigram"])] for t in toks]
    state = torch.zeros(4, 2, 2, dtype=torch.float32, device=dev)
    state[0] = 7.0
    for parts, n, row_req, req_start, req_pos, pos in side_by_side(([0, 1, 2, 4, 5, 20, T], [0, 2, 3, 4, 17, 18, T])):
        x = torch.empty(sum(n), d, device=dev)
        K.embed_pair(ints(sum((toks[i][a:b] for i, (a, b) in enumerate(parts)), [])), pos, row_req, req_start, req_pos, ints([3, 1]), table.to(dev),
                     None if B is None else B.to(dev), pairs[1] if pairs else 0, pairs[2] if pairs else 0, scale, state,
                     (1.0 + w).to(dev) if norm else None, eps, x)
        got = x.double().cpu().numpy()
        for i, (a, b) in enumerate(parts):
            assert np.abs(got[n[0] * i: n[0] * i + n[i]] - want[i][a:b]).max() < 2e-5 * np.abs(want[i]).max(), f"sequence {i}, rows {a} .. {b}"
    assert torch.all(state[0] == 7.0) and torch.all(state[2] == 0.0)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("d,T", [(50, 3), (64, 300), (2048, 5), (4100, 40)])
def test_joined_outputs_and_a_pair_of_norms_behind_an_added_one(dtype, d, T):
    """Outputs with and without a norm, two or one, with and without a third, into the stream and as activations; then a norm that
    adds with the two norms of the next layer's sublayers."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(d + T)
    r = lambda *s: torch.randn(*s, generator=g)
    x, a, b, c, wa, wb, w, w1, w2 = r(T, d), 5.0 * r(T, d), 0.1 * r(T, d), r(T, d), r(d), r(d), r(d), r(d), r(d)
    D = lambda t: t.double().numpy()
    tol = 2e-5 if dt == torch.float32 else 2e-2
    for two, normed, third, cast in ((True, True, True, True), (True, True, False, False), (False, False, True, True), (False, True, True, False), (True, False, False, True)):
        want = D(x) + (plain.rms_unit(D(a), 1e-3) * D(wa) if normed else D(a))
        if two:
            want = want + (plain.rms_unit(D(b), 1e-2) * D(wb) if normed else D(b))
        if third:
            want = want + D(c)
        got, h = x.to(dev).clone(), torch.zeros(T, d, dtype=dt, device=dev)
        K.join_parts(got, a.to(dev), wa.to(dev) if normed else None, 1e-3, b.to(dev) if two else None, wb.to(dev) if two and normed else None, 1e-2,
                     c.to(dev) if third else None, h if cast else None)
        assert np.abs(D(got.cpu()) - want).max() < 1e-5 * np.abs(want).max()
        assert not cast or np.abs(D(h.cpu()) - want).max() < tol * np.abs(want).max()
    got, h, h2 = x.to(dev).clone(), torch.empty(T, d, dtype=dt, device=dev), torch.empty(T, d, dtype=dt, device=dev)
    K.norm_add(a.to(dev), got, w.to(dev), 1e-3, w1.to(dev), 1e-4, h, w2.to(dev), h2)
    want = D(x) + plain.rms_unit(D(a), 1e-3) * D(w)
    assert np.abs(D(got.cpu()) - want).max() < 1e-5 * np.abs(want).max()
    for out, ww in ((h, w1), (h2, w2)):
        n = plain.rms_unit(want, 1e-4) * D(ww)
        assert np.abs(D(out.cpu()) - n).max() < tol * np.abs(n).max()


def far_rows_error(got, want, a, b):
    """The largest error of rows a .. b, each against its own largest value or that of a middling row, whichever is larger (a row
    that stands out must not hide the others' errors)."""
    size = np.abs(want).max(1)
    return (np.abs(got - want[a:b]).max(1) / np.maximum(size[a:b], np.median(size))).max()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("C,blocks,taps", [(12, 3, 2), (33, 3, 3), (96, 1, 4), (128, 4, 1), (192, 2, 5), (1024, 4, 3)])
def test_the_gated_recurrence_across_cuts_and_slots(dtype, C, blocks, taps):
    """Two sequences in portions (single rows, pairs, rows enough for several pieces) through state slots side by side: the
    convolution with the projection's bias ahead of it (not before the start), the gates from the block-diagonal maps, the
    recurrence and the branch.  Slow channels (lam far below zero: a close to 1) carry a large input from near the start to the end;
    fast ones forget at once."""
    from infinicore_infer_b200 import kernels as K
    from infinicore_infer_b200.parts import LinearAttention
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(C)
    T, n = 330, C // blocks
    r = lambda *s: torch.randn(*s, generator=g)
    bf = lambda t: t.to(torch.bfloat16)
    w_r, w_i = bf(r(blocks, n, n) * 1.5 * n ** -0.5), bf(r(blocks, n, n) * 1.5 * n ** -0.5)
    b_r, b_i, y_b, x_b, c_b = r(blocks, n), r(blocks, n), r(C), 2.0 * r(C), r(C)
    conv, lam = r(C, taps), torch.cat([torch.linspace(-9.0, -8.0, C // 2), torch.linspace(-7.0, 4.0, C - C // 2)])[torch.randperm(C, generator=g)]
    D = lambda t: t.double().numpy()
    us, want, plainer = [], [], []
    for i in range(2):
        u = r(T, 2 * C + 3)
        u[5, C:2 * C] *= 1000.0                   # a large input near the start
        us.append(u)
        y = plain.gelu_tanh(D(u)[:, :C] + D(y_b))
        x = plain.short_conv(D(u)[:, C:2 * C] + D(x_b), D(conv)) + D(c_b)
        gates = [plain.sigmoid(plain.block_maps(x, D(m.float()), D(b))) for m, b in ((w_r, b_r), (w_i, b_i))]
        want.append(plain.gated_linear_scan(x, *gates, D(lam))[0] * y)
        x2 = x.copy()
        x2[5:5 + taps] = 0.0
        plainer.append(plain.gated_linear_scan(x2, *gates, D(lam))[0] * y)
    late = [np.abs(o[T - 20:]).max(0) for o in want]          # per channel
    assert (np.abs(plainer[0] - want[0])[T - 20:].max(0) / late[0]).max() > 0.5          # in some channel the early input is still there at the end
    rate = (-8.0 * torch.logaddexp(lam.double(), torch.zeros_like(lam.double()))).float().to(dev)
    state, tails = torch.zeros(4, C, device=dev), torch.zeros(4, max(taps - 1, 1), C, device=dev)
    state[0] = tails[0] = 7.0
    tol = 3e-5 if dt == torch.float32 else 1.2e-2
    for parts, m, row_req, req_start, req_pos, pos in side_by_side(([0, 1, 2, 4, 30, 31, 95, 96, 300, T], [0, 2, 3, 4, 70, 71, 72, 281, 282, T])):
        u = torch.cat([us[i][a:b] for i, (a, b) in enumerate(parts)]).to(dev)
        v = torch.empty(sum(m), C, device=dev)
        K.causal_conv(u, C, C, conv.to(dev), c_b.to(dev), K.ACT_NONE, tails if taps > 1 else None, row_req, req_start, ints([3, 1]), v, None, in_bias=x_b.to(dev))
        caps = LinearAttention.step_list_capacity(sum(m), 2)
        arrays = {k: np.zeros(max(1, c), dtype=np.int32) for k, c in caps.items()}
        counts = LinearAttention.fill_step_lists(2, 2, m, [a for a, _ in parts], arrays)
        lists = {k: ints(arrays[k].tolist()) for k in arrays}
        out = torch.empty(sum(m), C, dtype=dt, device=dev)
        K.gated_recurrence(v, w_r.to(dt).to(dev), w_i.to(dt).to(dev), b_r.to(dev), b_i.to(dev), rate, u[:, :C], y_b.to(dev), K.ACT_GELU_TANH, state, req_start,
                           ints([3, 1]), out, lists["direct"], counts["direct"][0], lists["pieces"], counts["pieces"][0], lists["piece_reqs"],
                           counts["piece_reqs"][0])
        got = out.double().cpu().numpy()
        for i, (a, b) in enumerate(parts):
            err = far_rows_error(got[m[0] * i: m[0] * i + m[i]], want[i], a, b)
            assert err < tol, f"sequence {i}, rows {a} .. {b}: {err}"
            if b == T:
                err = (np.abs(got[m[0] * i: m[0] * i + m[i]][-20:] - want[i][T - 20:]).max(0) / late[i]).max()
                assert err < (1e-3 if dt == torch.float32 else 2e-2), f"sequence {i}, the last rows channel by channel: {err}"
    assert torch.all(state[0] == 7.0) and torch.all(tails[0] == 7.0) and torch.all(state[2] == 0.0) and torch.all(tails[2] == 0.0)


@pytest.mark.parametrize("dims,dk,half", [(8, 8, True), (6, 10, True), (6, 10, False), (64, 64, True), (128, 128, True)])
def test_rotation_in_place(dims, dk, half):
    from infinicore_infer_b200 import kernels as K
    dev = torch.device("cuda:0")
    H, T, base = 3, 70, 300.0
    g = torch.Generator().manual_seed(dims)
    u = torch.randn(T, 2 * H * dk + 9, generator=g)
    pos = torch.arange(900, 900 + T)
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    want = u.double().numpy().copy()
    order = list(range(dims)) if half else list(range(0, dims, 2)) + list(range(1, dims, 2))
    for off in (2, 4 + H * dk):
        x = want[:, off: off + H * dk].reshape(T, H, dk).copy()
        y = plain.rotate_half(np.concatenate([x[..., order], x[..., dims:]], axis=-1), pos.numpy(), {"dims": dims, "base": base})
        x[..., order], x[..., dims:] = y[..., :dims], y[..., dims:]
        want[:, off: off + H * dk] = x.reshape(T, H * dk)
    got = K.rotate_rows(u.to(dev), 2, 4 + H * dk, H, dk, f.float().to(dev), pos.to(torch.int32).to(dev), half=half)
    assert np.abs(got.double().cpu().numpy() - want).max() < 2e-4          # the angle itself is a float32 of up to a thousand
    only_q = K.rotate_rows(u.to(dev), 2, -1, H, dk, f.float().to(dev), pos.to(torch.int32).to(dev), half=half).double().cpu().numpy()
    assert np.abs(only_q[:, 2 + H * dk:] - u.double().numpy()[:, 2 + H * dk:]).max() == 0.0 and np.abs(only_q[:, :2 + H * dk] - want[:, :2 + H * dk]).max() < 2e-4


def part_context(lens, starts, slots, vocab=3):
    from infinicore_infer_b200.parts import StepContext
    rows, req_start = sum(lens), np.concatenate([[0], np.cumsum(lens)]).tolist()
    pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, lens)]).tolist()
    return StepContext(ntok=rows, nreq=len(lens), tokens=ints([0] * rows), positions=ints(pos), row_req=ints(np.repeat(np.arange(len(lens)), lens).tolist()),
                       req_start=ints(req_start), req_pos=ints(list(starts)), slot_ids=ints(list(slots)), block_tables=[], want_rows=ints([]), n_want=0,
                       host_req_start=req_start, host_req_pos=list(starts), host_slot_ids=list(slots))


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,dk,dv,dims", [(3, 16, 24, 16), (2, 40, 8, 12), (1, 6, 5, 4), (2, 128, 64, 128), (2, 64, 128, 0)])
def test_retention_keeps_far_keys_across_cuts_and_slots(dtype, H, dk, dv, dims):
    """The part alone over two sequences in portions: one row's key and value stand out near the start, and with a decay next to
    one the rows at the end still rest on it; a fast head has forgotten it."""
    from infinicore_infer_b200.cache.manager import StateView
    from infinicore_infer_b200.config import LinearAttentionSpec, PairRotarySpec
    from infinicore_infer_b200.parts import LinearAttention, Runtime
    from infinicore_infer_b200.weights import DictWeights
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    d, T, eps = 64, 300, 1e-6
    decay = tuple(np.linspace(0.9995, 0.5, H).tolist())
    g = torch.Generator().manual_seed(dk)
    bf = lambda t: t.to(torch.bfloat16).double()
    W = {n: bf(torch.randn(c, d, generator=g) * d ** -0.5).numpy() for n, c in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv))}
    W["o"] = bf(torch.randn(d, H * dv, generator=g) * (H * dv) ** -0.5).numpy()
    m = {"heads": H, "dim": dk, "vdim": dv, "decay": decay, "rot": {"dims": dims, "base": 3e4}}
    hs, want = [], []
    for i in range(2):
        h = torch.randn(T, d, generator=g)
        h[4] *= 25.0                              # a row whose key and value stand out
        hs.append(bf(h).numpy() if dt == torch.bfloat16 else h.double().numpy())
        want.append(plain.retention(hs[i], m, W, "", eps))
    lost = hs[0].copy()
    lost[4] = 0.0
    assert np.abs(plain.retention(lost, m, W, "", eps) - want[0])[T - 20:].max() > 0.3 * np.abs(want[0])[T - 20:].max()
    spec = LinearAttentionSpec(hidden_size=d, num_heads=H, head_dim=dk, v_head_dim=dv, norm_eps=eps, decay=decay, q_scale=dk ** -0.5, norm_per_head=True,
                               norm_name=None, gate_act="silu", position=PairRotarySpec(dims=dims, base=3e4, layout="halves") if dims else None)
    part = LinearAttention(spec, DictWeights({n: torch.tensor(a) for n, a in W.items()}, dt, dev), "", Runtime(dt, dev))
    state = torch.zeros(4, H, dk, dv, device=dev)
    state[0] = 7.0
    tol = 1e-4 if dt == torch.float32 else 3e-2
    cuts = ([0, 1, 2, 4, 30, 31, 95, 96, 270, T], [0, 2, 3, 4, 70, 71, 72, 251, 252, T])
    for s in range(len(cuts[0]) - 1):
        parts = [(cuts[i][s], cuts[i][s + 1]) for i in range(2)]
        h = torch.tensor(np.concatenate([hs[i][a:b] for i, (a, b) in enumerate(parts)])).to(dt).to(dev)
        got = part.forward(h, part_context([b - a for a, b in parts], [a for a, _ in parts], [3, 1]), StateView(state)).double().cpu().numpy()
        n0 = parts[0][1] - parts[0][0]
        for i, (a, b) in enumerate(parts):
            err = far_rows_error(got[n0 * i: n0 * i + b - a], want[i], a, b)
            assert err < tol, f"sequence {i}, rows {a} .. {b}: {err}"
    assert torch.all(state[0] == 7.0) and torch.all(state[2] == 0.0)


def paged(k, v, page, dev, dtype):
    """Keys [T, G, dk] and values [T, G, dv] of one request into pages handed out in a scrambled order; what lies beyond its end is
    what another request left."""
    T, G, dk = k.shape
    blocks = (T + page - 1) // page
    order = torch.randperm(blocks, generator=torch.Generator().manual_seed(3)) + 1
    kp = torch.full((blocks + 1, G, page, dk), 3.0, dtype=dtype, device=dev)
    vp = torch.full((blocks + 1, G, page, v.shape[-1]), 50.0, dtype=dtype, device=dev)
    for t in range(T):
        kp[order[t // page], :, t % page] = k[t].to(dtype)
        vp[order[t // page], :, t % page] = v[t].to(dtype)
    return kp, vp, order.to(torch.int32).view(1, -1).to(dev)


@pytest.mark.parametrize("dk,dv", [(56, 96), (96, 40), (64, 128), (128, 64), (8, 40), (40, 8), (120, 128), (72, 16), (64, 56)])
@pytest.mark.parametrize("heads,page", [((4, 2), 16), ((8, 1), 8), ((3, 3), 64), ((20, 1), 16)])
def test_keys_and_values_of_unlike_sizes_on_the_tensor_cores(dk, dv, heads, page):
    """The bfloat16 kernels of the generation path: tiles of a prompt's rows (a whole prompt, and a portion that starts in the middle
    of a page behind cached keys) and single rows whose keys are cut into ranges, with and without the gate per element.  For chosen
    rows one key scores above all others: the row's own, the first of all, one at a page's border, one far back."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), torch.bfloat16
    T, (H, G) = 333, heads
    g = torch.Generator().manual_seed(dk + dv)
    q = torch.randn(T, H, dk, generator=g, dtype=F)
    k = 2.0 * dk ** -0.5 * torch.randn(T, G, dk, generator=g, dtype=F)
    v = torch.randn(T, G, dv, generator=g, dtype=F)
    rests = {T - 1: 0, 300: 300, 200: 15, 201: 16, 128: 127, 255: 64, 90: 3, 17: 17}
    for j, (row, key) in enumerate(rests.items()):        # queries of these rows next to orthogonal to one another
        q[row, H - 1] *= 0.1
        q[row, H - 1, j] = 4.0
        k[key, G - 1] = 18.0 * q[row, H - 1] / (q[row, H - 1] @ q[row, H - 1])
    gate = 2.0 * torch.randn(T, H * dv, generator=g, dtype=F)
    q, k, v, gate = (t.to(dt).double() for t in (q, k, v, gate))
    out = np.zeros((T, H, dv))
    for hd in range(H):
        out[:, hd] = plain.causal_softmax(q[:, hd].numpy() @ k[:, hd // (H // G)].numpy().T) @ v[:, hd // (H // G)].numpy()
    for row, key in rests.items():
        assert np.abs(out[row, H - 1] - v[key, G - 1].numpy()).max() < 0.2, "the row rests on its key"
    gated = out * plain.sigmoid(gate.numpy()).reshape(T, H, dv)
    kp, vp, table = paged(k, v, page, dev, dt)
    qd = q.to(dt).to(dev).contiguous()
    wide = torch.zeros(T, H * dv + 7)
    wide[:, 3:3 + H * dv] = gate.float()
    wide = wide.to(dev)[:, 3:3 + H * dv]
    for gr, want in ((None, out), (wide, gated)):
        for start in (0, 203):
            n = T - start
            tiles = ints([[0, r0] for r0 in range(0, n, K.TILE_ROWS)])
            got = torch.full((n, H, dv), 9.0, dtype=dt, device=dev)
            K.attention_tcgen05(qd[start:].contiguous(), kp, vp, got, tiles, len(tiles), n, ints([0, n]), ints([start]), table, H, 1.0,
                                gate=None if gr is None else gr[start:], gate_elem=gr is not None)
            K.check_gemm_status(dev)
            err = np.abs(got.double().cpu().numpy() - want[start:]).max()
            assert err <= 4e-2, f"tiles from position {start}, gate {gr is not None}: {err}"
        pos = torch.arange(T, dtype=torch.int32, device=dev)
        some = ints(sorted(rests) + [0, 1, 7])
        for splits in (1, 2, 5):
            got = torch.full((T, H, dv), 9.0, dtype=dt, device=dev)
            K.attention_decode(qd, kp, vp, got, some, len(some), pos, torch.zeros_like(pos), table, H, 1.0, 0, splits, gate=gr, gate_elem=gr is not None)
            got = got.double().cpu().numpy()
            for i in some.tolist():
                assert np.abs(got[i] - want[i]).max() <= 4e-2, f"single row {i}, {splits} ranges, gate {gr is not None}"


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("experts,top,ff,shared,scale", [(5, 2, 40, 24, 2.25), (3, 3, 24, None, 0.5), (16, 1, 16, 8, 1.0), (60, 6, 9, 33, 1.75)])
def test_renormalised_scaled_scores_and_the_gated_shared_unit(dtype, experts, top, ff, shared, scale):
    from infinicore_infer_b200.config import GLUSpec, RoutedExpertsSpec
    from infinicore_infer_b200.parts import RoutedExperts, Runtime
    from infinicore_infer_b200.weights import DictWeights
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(experts)
    d = 48
    bf = lambda t: t.to(torch.bfloat16).double().numpy()
    W = {"router": bf(torch.randn(experts, d, generator=g) * 0.3)}
    units = [(f"e{e}.", ff) for e in range(experts)] + ([("shared.", shared)] if shared else [])
    for p, n in units:
        W[p + "gate"], W[p + "up"] = (bf(torch.randn(n, d, generator=g) * 1.5 * d ** -0.5) for _ in range(2))
        W[p + "down"] = bf(torch.randn(d, n, generator=g) * 2.0 * n ** -0.5)
    if shared:
        W["shared.sg"] = bf(torch.randn(1, d, generator=g) * 0.3)
    mlp = {"router": {"experts": experts, "top": top, "scale": scale}, "shared": {"ff": shared} if shared else None}
    spec = RoutedExpertsSpec(hidden_size=d, num_experts=experts, top=top, expert_size=ff, act="silu", scale_input=False, score_form="softmax_renorm",
                             score_scale=scale, shared=GLUSpec(hidden_size=d, intermediate_size=shared, act="silu") if shared else None,
                             shared_gate_name="sg" if shared else None)
    part = RoutedExperts(spec, DictWeights({n: torch.tensor(a) for n, a in W.items()}, dt, dev), "", Runtime(dt, dev))
    for T in (1, 5, 200, 600):
        h = torch.randn(T, d, generator=g, dtype=F) * 2.0
        if dt == torch.bfloat16:
            h = h.to(dt).double()
        margins = []
        want = plain.experts_ff(h.numpy(), mlp, W, "", margins)
        sure = margins[0] >= {"float32": 1e-6, "bfloat16": 1e-4}[dtype]        # the inputs are the same bits: only the sums' order differs
        got = part.forward(h.to(dt).to(dev).contiguous(), None).double().cpu().numpy()
        err = (np.abs(got - want).max(1) * sure).max() / np.abs(want).max()
        assert err <= (2e-5 if dt == torch.float32 else 2e-2), f"{T} rows: {err}"


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("dim,width,layer", [(8, 64, 2), (5, 50, 0), (24, 96, 1)])
def test_a_tokens_own_vector_multiplies_the_activated_gate(dtype, dim, width, layer):
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(dim)
    T, vocab, layers = 77, 31, 3
    table, z = torch.randn(vocab, layers * dim, generator=g).to(dt), 2.0 * torch.randn(T, dim, generator=g)
    toks = torch.randint(0, vocab, (T,), generator=g)
    out = torch.empty(T, dim, dtype=dt, device=dev)
    K.act_rows(z.to(dev), out, K.ACT_GELU_TANH, table.to(dev), layer * dim, toks.to(torch.int32).to(dev))
    want = plain.gelu_tanh(z.double().numpy()) * table.double().numpy()[toks.numpy()][:, layer * dim: (layer + 1) * dim]
    assert np.abs(out.double().cpu().numpy() - want).max() < (1e-5 if dt == torch.float32 else 1e-2) * np.abs(want).max()


# ---- generation through the scheduler ---------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler_matches_the_plain_model(folders):
    """Requests of unequal length through ``Generator`` (admission, portions of 16 tokens, decoding beside prompts, three
    slots for five requests): every generated token is the plain model's argmax given the tokens before it."""
    from infinicore_infer_b200.engine import Engine, Generator
    d, cfg, w = folders["recurrent"]
    eng = Engine.from_folder(d, dtype=torch.float32, max_tokens=160, cache_tokens=3 * 96, page_size=16, max_requests=3, max_step_tokens=64)
    gen = Generator(eng, chunk_size=16)
    prompts = [random_tokens(900 + i, n, cfg["vocab"]) for i, n in enumerate((40, 3, 25, 61, 12))]
    outs = gen.generate(prompts, max_new_tokens=12)
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits = plain.forward(cfg, w, p + o)
        for j, tok in enumerate(o):
            row = logits[len(p) + j - 1]
            best = int(row.argmax())
            assert tok == best or row[best] - row[tok] < 1e-4 * np.abs(row).max(), f"token {j} of a prompt of {len(p)}"
    eng.cache.check_invariants()


def test_command_line_runs_a_small_model_with_random_weights(tmp_path):
    """``--random piratar-tiny`` with three prompts through the scheduler, greedy: the printed tokens are the plain model's."""
    import re
    import subprocess
    import sys
    from infinicore_infer_b200.config import PRESETS, PiratarConfig
    from infinicore_infer_b200.weights import index_directory, read_tensor, write_model_folder
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    preset = PRESETS["piratar-tiny"]
    proc = subprocess.run([sys.executable, "-m", "infinicore_infer_b200.jiuge", "--nvidia", "--random", "piratar-tiny", "--seed", "3",
                           "--prompt-lens", "2,19,40", "--chunk-size", "11", "--num-pages", "24", "--max-batch", "3",
                           "--max-tokens-per-step", "24", "--temperature", "0", "--max-steps", "8", "--dtype", "float32"],
                          capture_output=True, text=True, cwd=root, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = {int(m.group(1)): [int(t) for t in m.group(2).split()] for m in re.finditer(r"request (\d+): ([\d ]*)", proc.stdout)}
    assert sorted(got) == [0, 1, 2]
    cfg = PiratarConfig.from_dict(preset.config)
    write_model_folder(cfg, str(tmp_path), seed=3, std=preset.std, norm_std=preset.norm_std)
    w = {n: read_tensor(i).double().numpy() for n, i in index_directory(str(tmp_path)).items()}
    for k, n in enumerate((2, 19, 40)):
        prompt = torch.randint(0, cfg.vocab, (n,), generator=torch.Generator().manual_seed(3 + k)).tolist()
        assert len(got[k]) == 8
        logits = plain.forward(cfg.to_dict(), w, prompt + got[k])
        for j, tok in enumerate(got[k]):
            row = logits[n + j - 1]
            assert tok == int(row.argmax()) or row.max() - row[tok] < 1e-4 * np.abs(row).max(), f"request {k}, token {j}"
