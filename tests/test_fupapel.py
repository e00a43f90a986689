"""Fupapel through the engine against the plain implementation (tests/plain_fupapel.py): each mechanism alone, whole models of
several sizes and layer orders, prompts cut in every way, batches, reused pages and state slots, keys at the borders of chunks
and far away, long decoding, and greedy generation through the scheduler."""
import json
import os

import numpy as np
import pytest
import torch

from conftest import random_tokens
import plain_fupapel as plain
from trace_helpers import by_position, mixed, portions, staggered_plan, tail_decode, whole

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 1e-5, "bfloat16": 4e-2}
F = torch.float64


def rotation(dims, base=1e4, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def chunked(heads, kv_heads, dim, vdim, scale, chunk, rot):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}, "rot": rot}


def convolved(heads, kv_heads, dim, vdim, scale, chunk, rot, taps, kv_from=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}, "rot": rot, "conv": taps}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return "attention_2", out


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=1e5):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def moe(experts, identity, top, ff, groups):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "groups": dict(zip(("count", "keep"), groups))},
            "expert": {"ff": ff}}


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(width, vocab, layers, mult=1.0, eps=1e-5):
    return {"architecture": "Fupapel", "norm": {"eps": eps}, "vocab": vocab, "width": width, "residual_mult": mult, "layers": layers}


# Sizes that differ from one another in everything: every order of the three mixers, key and value sizes that are unequal in
# both directions, one key head, several and as many as query heads, rotation of a part of a head and of all of it, with and
# without stretched frequencies, chunks shorter than a page, no multiple of one and longer than every prompt here, one to five
# taps, borrowed keys under a wider and a narrower mask and twice from one layer, one expert a row, several and all, no identity,
# a few, and more than experts, one group, several, all kept, layers without feed-forward, residual factors of one and not.
MODELS = {
    "one-each": config(64, 97, [layer(convolved(4, 2, 16, 24, 0.3, 21, rotation(8, scaling=(8.0, 1.0, 4.0, 32)), 3), moe(5, 3, 2, 40, (4, 1))),
                                layer(chunked(6, 1, 24, 16, 0.3, 37, rotation(24)), moe(4, 2, 3, 24, (2, 1))),
                                layer(latent(3, 16, 8, 24, 40, 28, 0.25), None)], mult=0.6),
    "borrowed": config(96, 211, [layer(latent(4, 8, 16, 16, 24, 40, 0.3, 300.0), moe(6, 2, 4, 32, (4, 3))),
                                 layer(convolved(6, 3, 16, 16, 0.35, 40, rotation(16, 5e4, (4.0, 1.0, 2.0, 64)), 4), moe(3, 1, 1, 24, (1, 1))),
                                 layer(convolved(6, 3, 16, 16, 0.2, 64, rotation(16, 5e4, (4.0, 1.0, 2.0, 64)), 2, kv_from=1), None),
                                 layer(chunked(2, 2, 32, 48, 0.25, 300, rotation(12, 2.5e5)), moe(4, 0, 2, 24, (2, 2))),
                                 layer(convolved(6, 3, 16, 16, 0.3, 9, rotation(16, 5e4, (4.0, 1.0, 2.0, 64)), 5, kv_from=1), moe(2, 4, 2, 40, (3, 2)))],
                      mult=0.75, eps=3e-6),
    "latents": config(80, 77, [layer(latent(5, 8, 24, 8, 12, 9, 0.4), moe(7, 1, 3, 24, (2, 1))),
                               layer(latent(2, 40, 8, 24, 64, 48, 0.2, 1e3), None),
                               layer(chunked(5, 5, 16, 16, 0.3, 50, rotation(16)), moe(2, 1, 2, 48, (1, 1)))], mult=1.0),
    # nothing a multiple of anything: odd width, odd sizes everywhere, a prime vocabulary, one tap
    "awkward": config(50, 61, [layer(chunked(3, 1, 10, 7, 0.4, 13, rotation(6, 555.0)), moe(2, 1, 2, 11, (3, 2))),
                               layer(convolved(3, 3, 14, 9, 0.4, 5, rotation(10, 77.0, (3.0, 1.0, 3.0, 20)), 1), moe(3, 2, 1, 13, (5, 1))),
                               layer(latent(3, 6, 4, 9, 11, 7, 0.5), moe(3, 0, 3, 7, (1, 1))),
                               layer(convolved(3, 3, 14, 9, 0.3, 7, rotation(10, 77.0, (3.0, 1.0, 3.0, 20)), 1, kv_from=1), None)], mult=0.9),
    # heads of 64 and 128, as the tensor-core kernels take them; experts of a width that the tiles share
    "wide": config(256, 333, [layer(chunked(4, 1, 64, 64, 0.125, 48, rotation(32)), moe(6, 2, 2, 128, (4, 2))),
                              layer(convolved(4, 2, 128, 128, 0.09, 100, rotation(128, scaling=(4.0, 1.0, 4.0, 64)), 3), moe(4, 4, 3, 64, (2, 1))),
                              layer(latent(4, 64, 32, 64, 160, 96, 0.1), None),
                              layer(convolved(4, 2, 128, 128, 0.09, 130, rotation(128, scaling=(4.0, 1.0, 4.0, 64)), 3, kv_from=1), moe(3, 1, 1, 64, (2, 1)))],
                  mult=0.8),
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
        d = str(tmp_path_factory.mktemp("fupapel_" + name))
        write_model_folder(config_class_for(cfg).from_dict(cfg), d, seed=seed + 51, std=STDS.get(name, STD), norm_std=0.2)
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
    """Logits [T, vocab] with ``margin`` [T]: the smallest router margin of each row (and of the row before it, which the token
    shift carries into it) over the model's layers, and ``noise`` [T]: how far each row's logits move (as ``row_error``
    measures it) when the plain implementation rounds the operands of its matrix products to bfloat16 and does nothing else
    differently."""


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
        margin = np.stack(margins).min(0)
        want.margin = np.minimum(margin, np.concatenate([[np.inf], margin[:-1]]))
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
    for i, n in enumerate((1, 37, 150)):
        toks, want = expected(folders, name, 300 + i, n)
        for what, steps in (("whole", whole("r", toks)), ("tail", tail_decode("r", toks, tail=20)),
                            ("portions", portions("r", toks)), ("pairs", portions("r", toks, sizes=(2,))),
                            ("uneven", portions("r", toks, sizes=(17, 3, 31, 2, 16)))):
            check(run(eng, steps), "r", want, TOL[dtype], f"{name} {dtype} {what} n={n}")
        eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["borrowed", "wide"])
def test_records_run_one_by_one_are_the_same_program(folders, engines, name, dtype):
    """The unfused way of running the records: every record a call of its own with the stream made whole after it."""
    toks, want = expected(folders, name, 300, 37)
    check(run(engines(name, dtype, native_runner=False), portions("r", toks, sizes=(11, 1, 2))), "r", want, TOL[dtype], f"{name} {dtype} one by one")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_every_token_decoded_alone_through_graphs(folders, engines, dtype):
    """Long decoding: every token a step of its own (captured steps), so pages, the convolutions' tails and the kept rows move
    one position at a time, and chunk borders pass over decoded tokens."""
    for name in ("borrowed", "one-each", "awkward"):
        toks, want = expected(folders, name, 77, 300)
        eng = engines(name, dtype)
        before = eng.steps_run
        check(run(eng, tail_decode("r", toks, tail=len(toks))), "r", want, TOL[dtype], f"{name} {dtype} token by token")
        assert eng.steps_run - before >= 300


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["borrowed", "one-each", "awkward"])
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


def test_a_reused_slot_starts_from_a_row_of_zeros_and_empty_tails(folders, engines):
    """The same request several times in a row lands in the slot (and pages) that its first run left, after runs of odd and
    even numbers of steps: whichever of the two kept rows was the last one, the first row's row before is zeros again."""
    toks, want = expected(folders, "borrowed", 9, 45)
    eng = engines("borrowed", "float32", max_requests=1)
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


# ---- mechanisms alone, with inputs made so that one key decides ------------------------------------------------------------
def paged(k, v, page, dev, dtype):
    """Keys [T, G, dk] and values [T, G, dv] of one request into pages handed out in a scrambled order."""
    T, G, dk = k.shape
    blocks = (T + page - 1) // page
    order = torch.randperm(blocks, generator=torch.Generator().manual_seed(3)) + 1
    kp = torch.zeros(blocks + 1, G, page, dk, dtype=dtype, device=dev)
    vp = torch.zeros(blocks + 1, G, page, v.shape[-1], dtype=dtype, device=dev)
    for t in range(T):
        kp[order[t // page], :, t % page] = k[t].to(dtype)
        vp[order[t // page], :, t % page] = v[t].to(dtype)
    return kp, vp, order.to(torch.int32).view(1, -1).to(dev)


def border_case(T, H, G, dk, dv, chunk, seed, bf16):
    """Queries, keys, values, sinks and gates in which, for chosen rows, head 0 scores the last key of the chunk before (just
    outside) above the first key of its own chunk (just inside) above all others; the last row of every chunk scores, with its
    last head, the chunk's second key above everything (a key far back among all the others); and the sinks, one above the
    strongest score of most rows and one far below all, each move their heads' outputs."""
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(T, H, dk, generator=g, dtype=F)
    k = 0.3 * torch.randn(T, G, dk, generator=g, dtype=F)
    v = torch.randn(T, G, dv, generator=g, dtype=F)
    rows = [i for i in range(chunk + 2, T, 7) if i % chunk not in (0, 1)]
    for i in rows:
        start = i // chunk * chunk
        unit = q[i, 0] / (q[i, 0] @ q[i, 0])
        k[start - 1, 0], k[start, 0] = 14.0 * unit, 9.0 * unit
    far = []
    for start in range(0, T, chunk):
        last = min(start + chunk, T) - 1
        if last - start >= 8:
            k[start + 1, G - 1] = 16.0 * q[last, H - 1] / (q[last, H - 1] @ q[last, H - 1])
            far.append((last, start + 1))
    sinks = torch.linspace(7.0, -3.0, H, dtype=F)
    if H > 1:
        sinks[1] = 20.0
    gate = 2.0 * torch.randn(T, H * dv, generator=g, dtype=F)
    if bf16:
        q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
    return q, k, v, sinks.float().double(), gate.float().double(), rows, far


def plain_chunks(q, k, v, chunk, positions, sinks, gate=None, shift=0):
    see = np.array([[j <= i and (i + shift) // chunk == (j + shift) // chunk for j in positions] for i in positions])
    out = plain.attend(q.numpy(), k.numpy(), v.numpy(), 1.0, see, sinks)
    return out if gate is None else out * plain.sigmoid(gate.numpy()).reshape(out.shape)


def gate_rows(gate, dev):
    """The gate as columns of wider float32 rows, as the fused projection leaves them (its first column on no 16-byte boundary)."""
    wide = torch.zeros(gate.shape[0], gate.shape[1] + 7, dtype=torch.float32)
    wide[:, 3:3 + gate.shape[1]] = gate.float()
    return wide.to(dev)[:, 3:3 + gate.shape[1]]


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("chunk,page", [(7, 8), (16, 16), (33, 8), (64, 16)])
def test_chunk_borders_sinks_and_element_gates_of_the_row_attention(dtype, chunk, page):
    """The kernel of one warp a row and head: whole prompts and single decoded rows, values of another size than keys."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    T, H, G, dk, dv = 150, 4, 2, 24, 40
    q, k, v, sinks, gate, rows, far = border_case(T, H, G, dk, dv, chunk, chunk, dt == torch.bfloat16)
    at = np.arange(T)
    want = plain_chunks(q, k, v, chunk, at, sinks.numpy(), gate)
    for row, key in far:                          # rows that rest on a far key: its value, the sink's share off, times the gate
        assert np.abs(plain_chunks(q, k, v, chunk, at, sinks.numpy() - 1e3)[row, -1] - v[key, G - 1].numpy()).max() < 0.05
    for other in (plain_chunks(q, k, v, chunk, at, sinks.numpy(), gate, shift=1), plain_chunks(q, k, v, chunk, at, sinks.numpy(), gate, shift=-1),
                  plain_chunks(q, k, v, chunk, at, np.zeros(H), gate), plain_chunks(q, k, v, chunk, at, sinks.numpy())):
        assert np.abs(other - want)[rows].max() > 0.05       # the inputs tell a border that is one off, a lost sink, a lost gate
    kp, vp, table = paged(k, v, page, dev, dt)
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    out = torch.empty(T, H, dv, dtype=dt, device=dev)
    sw, gr = sinks.float().to(dev), gate_rows(gate, dev)
    K.attention_rows(q.to(dt).to(dev).contiguous(), kp, vp, out, pos, torch.zeros_like(pos), table, T, H, 1.0, -chunk, sink=True, gate=gr,
                     sink_w=sw, gate_elem=True)
    tol = 2e-5 if dt == torch.float32 else 3e-2
    err = np.abs(out.double().cpu().numpy() - want).max()
    assert err <= tol, f"prompt rows differ by {err}"
    for i in rows[-4:] + [0, chunk - 1, chunk, chunk + 1] + [row for row, _ in far]:
        one = torch.empty(1, H, dv, dtype=dt, device=dev)
        K.attention_rows(q[i:i + 1].to(dt).to(dev).contiguous(), kp, vp, one, pos[i:i + 1], torch.zeros(1, dtype=torch.int32, device=dev), table,
                         1, H, 1.0, -chunk, sink=True, gate=gr[i:i + 1], sink_w=sw, gate_elem=True)
        assert np.abs(one.double().cpu().numpy()[0] - want[i]).max() <= tol, f"decoded row {i}"


@pytest.mark.parametrize("dh", [32, 48, 64, 128])
@pytest.mark.parametrize("chunk,heads", [(17, (4, 2)), (64, (8, 1)), (130, (4, 2)), (200, (3, 3))])
def test_chunk_borders_sinks_and_element_gates_on_the_tensor_cores(dh, chunk, heads):
    """The bfloat16 kernels of the generation path: tiles of a prompt's rows (a whole prompt, and a portion that starts in
    the middle of a page and of a chunk behind cached keys), and single rows whose keys are cut into ranges; with the gate
    per element, with the sinks alone, and with a gate per head."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), torch.bfloat16
    T, page, (H, G) = 333, 16, heads
    q, k, v, sinks, gate, rows, far = border_case(T, H, G, dh, dh, chunk, chunk + dh, True)
    at = np.arange(T)
    rows = rows + [row for row, _ in far]
    kp, vp, table = paged(k, v, page, dev, dt)
    qd, sw = q.to(dt).to(dev).contiguous(), sinks.float().to(dev)
    plain_out = plain_chunks(q, k, v, chunk, at, sinks.numpy())
    per_head = plain.sigmoid(gate.numpy()[:, :H])[:, :, None]
    for form, gr, elem, want in (("element gate", gate_rows(gate, dev), True, plain_chunks(q, k, v, chunk, at, sinks.numpy(), gate)),
                                 ("sinks alone", None, False, plain_out), ("head gate", gate_rows(gate, dev)[:, :H], False, plain_out * per_head)):
        kernels = [("legacy tiles", K.attention_prefill)]
        if K.attention_tcgen05_supports(dh, page):
            kernels.append(("tcgen05 tiles", None))
        for start in (0, 203):                    # the rows of positions start .. T - 1 as one portion
            n = T - start
            tiles = torch.tensor([[0, r0] for r0 in range(0, n, K.TILE_ROWS)], dtype=torch.int32, device=dev)
            req_start = torch.tensor([0, n], dtype=torch.int32, device=dev)
            req_pos = torch.tensor([start], dtype=torch.int32, device=dev)
            how = dict(sink=True, gate=None if gr is None else gr[start:], sink_w=sw, gate_elem=elem)
            for name, fn in kernels:
                out = torch.zeros(n, H, dh, dtype=dt, device=dev)
                if fn is None:
                    K.attention_tcgen05(qd[start:].contiguous(), kp, vp, out, tiles, len(tiles), n, req_start, req_pos, table, H, 1.0, -chunk, **how)
                    K.check_gemm_status(dev)
                else:
                    fn(qd[start:].contiguous(), kp, vp, out, tiles, len(tiles), req_start, req_pos, table, H, 1.0, -chunk, **how)
                err = np.abs(out.double().cpu().numpy() - want[start:]).max()
                assert err <= 3e-2, f"{form}: {name} from position {start}: {err}"
        pos = torch.arange(T, dtype=torch.int32, device=dev)
        some = torch.tensor(rows[-6:] + [0, chunk - 1, chunk, chunk + 1], dtype=torch.int32, device=dev)
        for splits in (1, 3, 8):
            out = torch.zeros(T, H, dh, dtype=dt, device=dev)
            K.attention_decode(qd, kp, vp, out, some, len(some), pos, torch.zeros_like(pos), table, H, 1.0, -chunk, splits, sink=True, gate=gr,
                               sink_w=sw, gate_elem=elem)
            got = out.double().cpu().numpy()
            for i in some.tolist():
                assert np.abs(got[i] - want[i]).max() <= 3e-2, f"{form}: single row {i}, {splits} ranges"


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("taps,borrows", [(1, False), (2, False), (3, False), (5, False), (3, True)])
def test_convolved_queries_and_keys_across_cuts(dtype, taps, borrows):
    """Two sequences in portions of several sizes, single rows and pairs among them, through state slots side by side: the
    convolutions from the kept tails (whether the row's own block or the tails' kernel moved them on), the norm over the whole
    projection, the rotation in halves by stretched frequencies, each head's factor on its queries; keys and values land in the
    pages at the rows' positions.  A layer that borrows its keys makes queries only, from tails of its own."""
    from infinicore_infer_b200 import kernels as K
    from infinicore_infer_b200.config import FrequencyBandSpec, PairRotarySpec
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    H, G, dk, dv, dims, page, eps, T = 4, 2, 24, 16, 16, 8, 1e-3, 90
    rot = rotation(dims, 300.0, (4.0, 1.0, 4.0, 32))
    f, mag = PairRotarySpec(dims=dims, base=300.0, scaling=FrequencyBandSpec(4.0, 32.0, 1.0, 4.0), layout="halves").frequencies()
    g = torch.Generator().manual_seed(taps)
    nq, nk, nv = H * dk, (0 if borrows else G * dk), (0 if borrows else G * dv)
    C, ld = nq + nk + nv, nq + nk + nv + 5
    us = [(2.0 * torch.randn(T, ld, generator=g, dtype=F)).float().double().numpy() for _ in range(2)]
    conv = torch.randn(C, taps, generator=g, dtype=F).float()
    wq, wk = (1 + 0.5 * torch.randn(nq, generator=g, dtype=F)).float(), (1 + 0.5 * torch.randn(max(nk, 1), generator=g, dtype=F)).float()
    temp = (1 + 0.5 * torch.randn(H, generator=g, dtype=F)).float()
    want = []
    for u in us:
        y = plain.short_conv(u[:, :C], conv.double().numpy())
        q = plain.rotate_half(plain.norm_plain(y[:, :nq], wq.double().numpy(), eps).reshape(T, H, dk), np.arange(T), rot) * temp.double().numpy()[:, None]
        k = v = None
        if not borrows:
            k = plain.rotate_half(plain.norm_plain(y[:, nq:nq + nk], wk.double().numpy(), eps).reshape(T, G, dk), np.arange(T), rot)
            v = y[:, nq + nk:].reshape(T, G, dv)
        want.append((q, k, v))
    blocks = (T + page - 1) // page
    table = torch.tensor([[2 * b + 2 for b in range(blocks)], [2 * b + 1 for b in range(blocks)]], dtype=torch.int32, device=dev)
    kp = torch.zeros(2 * blocks + 1, G, page, dk, dtype=dt, device=dev)
    vp = torch.zeros(2 * blocks + 1, G, page, dv, dtype=dt, device=dev)
    tails = torch.zeros(4, taps - 1, C, dtype=torch.float32, device=dev) if taps > 1 else None
    if tails is not None:
        tails[0] = 7.0                            # slot 0 is nobody's
    cv = conv.to(dev)
    convs = (cv[:nq].contiguous(), cv[nq:nq + nk].contiguous(), cv[nq + nk:].contiguous()) if not borrows else (cv, None, None)
    tol = 2e-5 if dt == torch.float32 else 2e-2
    cuts = ([0, 1, 2, 4, 30, 31, 32, 61, 63, T], [0, 3, 4, 5, 6, 29, 31, 32, 62, T])      # steps of unequal portions side by side
    for s in range(len(cuts[0]) - 1):
        parts = [(cuts[i][s], cuts[i][s + 1]) for i in range(2)]
        n = [b - a for a, b in parts]
        u = torch.tensor(np.concatenate([us[i][a:b] for i, (a, b) in enumerate(parts)]), dtype=torch.float32, device=dev)
        q_out = torch.empty(sum(n), H, dk, dtype=dt, device=dev)
        pos = torch.tensor(np.concatenate([np.arange(a, b) for a, b in parts]), dtype=torch.int32, device=dev)
        K.conv_qkv(u, (0, nq, nq + nk), H, G, dk, dv, not borrows, convs, taps, (wq.to(dev), None if borrows else wk.to(dev)), eps,
                   torch.tensor(f, dtype=torch.float32, device=dev), dims, tails, pos,
                   torch.tensor([0] * n[0] + [1] * n[1], dtype=torch.int32, device=dev), torch.tensor([0, n[0], sum(n)], dtype=torch.int32, device=dev),
                   torch.tensor([3, 1], dtype=torch.int32, device=dev), table, page, q_out, kp, vp, rot_half=True, rot_mag=mag, temp=temp.to(dev))
        got = q_out.double().cpu().numpy()
        for i, (a, b) in enumerate(parts):
            q = want[i][0][a:b]
            assert np.abs(got[n[0] * i: n[0] * i + n[i]] - q).max() < tol * np.abs(want[i][0]).max(), f"queries of sequence {i}, rows {a} .. {b}"
    for i in range(2 if not borrows else 0):
        for t in range(T):
            pg, at = table[i, t // page].item(), t % page
            assert np.abs(kp[pg, :, at].double().cpu().numpy() - want[i][1][t]).max() < tol * np.abs(want[i][1]).max(), f"key {t} of sequence {i}"
            assert np.abs(vp[pg, :, at].double().cpu().numpy() - want[i][2][t]).max() < tol * np.abs(want[i][2]).max(), f"value {t} of sequence {i}"
    if tails is not None:
        assert torch.all(tails[0] == 7.0) and torch.all(tails[2] == 0.0)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("d,T", [(50, 40), (64, 700), (96, 1300), (256, 90), (2052, 700), (4096, 1300), (8192, 650), (8200, 12)])
def test_a_pair_of_norms_with_a_token_shift_across_cuts_and_slots(dtype, d, T):
    """Two norms of one stream, the first mixed with the row before it: sequences in portions (whole, single rows, pairs, more
    rows than blocks take at once) through state slots, the row before a portion's first row from the step before whatever
    the number of steps so far.  Large rows before small ones, so that a lost or repeated row shows."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(d)
    eps, eps2 = 1e-4, 1e-2
    w, w2 = (1 + 0.3 * torch.randn(d, generator=g)), (1 + 0.3 * torch.randn(d, generator=g))
    mu = 0.5 + 0.4 * torch.randn(d, generator=g)
    xs = [torch.randn(T, d, generator=g) * (0.1 + (torch.arange(T) % 5)[:, None].float()) for _ in range(2)]
    norm = [plain.norm_plain(x.double().numpy(), w.double().numpy(), eps) for x in xs]
    want = [plain.token_shift(n, mu.double().numpy()) for n in norm]
    want2 = [plain.norm_plain(x.double().numpy(), w2.double().numpy(), eps2) for x in xs]
    kept = K.norm_pair_kept_floats(d)
    state = torch.zeros(4, 2, kept, dtype=torch.float32, device=dev)
    state[0] = 7.0
    slots = torch.tensor([3, 1], dtype=torch.int32, device=dev)
    tol = 1e-5 if dt == torch.float32 else 1e-2
    cuts = ([0, 1, 2, 4, 5, T - 1, T], [0, 2, 3, 4, T - 3, T - 2, T])
    for a0, b0, a1, b1 in zip(cuts[0], cuts[0][1:], cuts[1], cuts[1][1:]):
        n0, n1 = b0 - a0, b1 - a1
        x = torch.cat([xs[0][a0:b0], xs[1][a1:b1]]).to(dev)
        h, h2 = torch.empty(n0 + n1, d, dtype=dt, device=dev), torch.empty(n0 + n1, d, dtype=dt, device=dev)
        ints = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        K.norm_pair(x, w.to(dev), eps, h, mu.to(dev), state, ints([0] * n0 + [1] * n1), ints([0, n0, n0 + n1]), ints([a0, a1]), slots,
                    w2.to(dev), eps2, h2)
        got, got2 = h.double().cpu().numpy(), h2.double().cpu().numpy()
        for i, (a, b, rows) in enumerate(((a0, b0, slice(0, n0)), (a1, b1, slice(n0, n0 + n1)))):
            assert np.abs(got[rows] - want[i][a:b]).max() < tol * np.abs(want[i]).max(), f"sequence {i}, rows {a} .. {b}"
            assert np.abs(got2[rows] - want2[i][a:b]).max() < tol * np.abs(want2[i]).max(), f"second norm of sequence {i}, rows {a} .. {b}"
    assert torch.all(state[0] == 7.0) and torch.all(state[2] == 0.0)
    h = torch.empty(T, d, dtype=dt, device=dev)          # without a shift and without a second norm
    K.norm_pair(xs[0].to(dev), w.to(dev), eps, h)
    assert np.abs(h.double().cpu().numpy() - norm[0]).max() < tol * np.abs(norm[0]).max()


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_latent_queries_with_a_rotated_part_and_cache_rows(dtype):
    """Both forms of the kernel ahead of the latent attention: the queries' latent normed beside the cache row with its rotated
    key part, and the heads' queries split and rotated (in halves; in pairs; fewer elements than the part)."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    H, dn, dr, R, Q, page, eps, n = 3, 10, 12, 28, 20, 8, 1e-3, 30
    g = torch.Generator().manual_seed(1)
    start = 13
    u = torch.randn(n, Q + R + dr + 3, generator=g)
    qu = torch.randn(n, H * (dn + dr), generator=g)
    wq, wc = 1 + 0.4 * torch.randn(Q, generator=g), 1 + 0.4 * torch.randn(R, generator=g)
    pos = torch.arange(start, start + n, dtype=torch.int32, device=dev)
    zero = torch.zeros_like(pos)
    blocks = (start + n + page - 1) // page
    table = torch.tensor([[blocks - b for b in range(blocks)]], dtype=torch.int32, device=dev)
    tol = 2e-5 if dt == torch.float32 else 2e-2
    for dims, half in ((12, True), (8, True), (12, False), (6, False)):
        f = torch.tensor([200.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32, device=dev)
        pages = torch.zeros(blocks + 1, page, R + dr, dtype=dt, device=dev)
        c_q = torch.empty(n, Q, dtype=dt, device=dev)
        K.latent_qkv(u.to(dev), 0, Q, H, dn, dr, R, dims, f, 1.0, wc.to(dev), eps, pos, zero, table, page, c_q, None, pages, q_norm=wq.to(dev),
                     q_rank=Q, rot_half=half)
        q_plain = torch.empty(n, H * dn, dtype=dt, device=dev)
        q_full = torch.full((n, H, R + dr), 9.0, dtype=dt, device=dev)
        K.latent_qkv(qu.to(dev), 0, -1, H, dn, dr, R, dims, f, 1.0, None, eps, pos, zero, None, page, q_plain, q_full, None, rot_half=half)

        def turn(x):
            if half:
                return plain.rotate_half(x, np.arange(start, start + n), rotation(dims, 200.0))
            order = list(range(0, dims, 2)) + list(range(1, dims, 2))            # neighbours side by side become halves
            y = plain.rotate_half(np.concatenate([x[..., order], x[..., dims:]], axis=-1), np.arange(start, start + n), rotation(dims, 200.0))
            out = y.copy()
            out[..., order] = y[..., :dims]
            return out
        un, qn = u.double().numpy(), qu.double().numpy().reshape(n, H, dn + dr)
        assert np.abs(c_q.double().cpu().numpy() - plain.norm_plain(un[:, :Q], wq.double().numpy(), eps)).max() < 4 * tol
        c, r = plain.norm_plain(un[:, Q:Q + R], wc.double().numpy(), eps), turn(un[:, None, Q + R:Q + R + dr])[:, 0]
        for t in range(n):
            p = start + t
            row = pages[table[0, p // page].item(), p % page].double().cpu().numpy()
            assert np.abs(row - np.concatenate([c[t], r[t]])).max() < 4 * tol, f"cache row {p} ({dims} of {dr}, halves {half})"
        assert np.abs(q_plain.double().cpu().numpy() - qn[..., :dn].reshape(n, H * dn)).max() < 4 * tol
        assert np.abs(q_full.double().cpu().numpy()[..., R:] - turn(qn[..., dn:])).max() < 4 * tol
        assert torch.all(q_full[..., :R] == 9.0)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,R,dr,page", [(3, 20, 8, 8), (8, 64, 32, 16), (2, 96, 5, 16), (16, 128, 64, 16), (5, 24, 16, 8), (4, 512, 64, 16)])
def test_sinks_and_far_keys_of_the_latent_attention(dtype, H, R, dr, page):
    """All heads over one cached row per position, on the row kernel and (bfloat16) the tensor-core kernel, whole prompts, a
    portion behind cached keys, and single rows with their keys cut into ranges: the last head of chosen rows rests on the
    sequence's second key, far back; a sink above all other scores and one below each move their heads."""
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    T, D = 210, R + dr
    g = torch.Generator().manual_seed(R + dr)
    q = torch.randn(T, H, D, generator=g, dtype=F) * 3.0 / D ** 0.5
    c = torch.randn(T, D, generator=g, dtype=F)
    far = [T - 1, T - 2, 100]
    for i in far:
        q[i, H - 1] = q[T - 1, H - 1]
    c[1] = 22.0 * q[T - 1, H - 1] / (q[T - 1, H - 1] @ q[T - 1, H - 1])
    sinks = torch.linspace(4.0, -2.0, H, dtype=F).float().double()
    if dt == torch.bfloat16:
        q, c = q.to(dt).double(), c.to(dt).double()
    see = plain.visibility(np.arange(T), plain.sees_all)
    how = lambda s: plain.attend(q.numpy(), c.numpy()[:, None], c.numpy()[:, None, :R], 1.0, see, s)
    want = how(sinks.numpy())
    assert np.abs(how(sinks.numpy() - 1e3)[far, -1] - c[1, :R].numpy()).max() < 0.05 * np.abs(c[1].numpy()).max()
    assert np.abs(how(np.zeros(H)) - want).max() > 0.1 and np.abs(how(sinks.numpy() - 1e3) - want)[:, -1].max() > 0.01
    kp, _, table = paged(c[:, None], c[:, None], page, dev, dt)
    pages, sw = kp[:, 0].contiguous(), sinks.float().to(dev)
    tol = (2e-5 if dt == torch.float32 else 2e-2) * np.abs(want).max()
    for start in (0, 77):
        n = T - start
        pos = torch.arange(start, T, dtype=torch.int32, device=dev)
        req_start = torch.tensor([0, n], dtype=torch.int32, device=dev)
        for with_tiles in (False, True):
            out = torch.empty(n, H, R, dtype=dt, device=dev)
            K.latent_attention(q[start:].to(dt).to(dev).contiguous(), pages, out, pos, torch.zeros_like(pos), table, H, R, dr, 1.0,
                               req_start=req_start if with_tiles else None, sink_w=sw)
            err = np.abs(out.double().cpu().numpy() - want[start:]).max()
            assert err <= tol, f"rows from {start} (tiles {with_tiles}): {err}"
    for i in far + [0, 1, 33]:
        for splits in (1, 4):
            one = torch.empty(1, H, R, dtype=dt, device=dev)
            p1 = torch.tensor([i], dtype=torch.int32, device=dev)
            K.latent_attention(q[i:i + 1].to(dt).to(dev).contiguous(), pages, one, p1, torch.zeros_like(p1), table, H, R, dr, 1.0, splits=splits,
                               req_start=torch.tensor([0, 1], dtype=torch.int32, device=dev), sink_w=sw)
            assert np.abs(one.double().cpu().numpy()[0] - want[i]).max() <= tol, f"single row {i}, {splits} ranges"


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,n,k,T", [(3, 20, 12, 5), (4, 64, 128, 70), (2, 40, 96, 1)])
def test_a_product_per_head_times_the_heads_gate(dtype, H, n, k, T):
    from infinicore_infer_b200 import kernels as K
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(T, H, k, generator=g).to(dt), (torch.randn(H, n, k, generator=g) * k ** -0.5).to(dt)
    gate = torch.randn(T, H + 5, generator=g) * 2.0
    out = torch.empty(T, H, n, dtype=dt, device=dev)
    K.head_linear(x.to(dev), w.to(dev), out, n, gate=gate.to(dev)[:, 2:], gate_ld=H + 5, gate_head=True)
    want = np.einsum("thk,hnk->thn", x.double().numpy(), w.double().numpy()) * plain.sigmoid(gate.double().numpy()[:, 2:2 + H])[:, :, None]
    assert np.abs(out.double().cpu().numpy() - want).max() < (2e-5 if dt == torch.float32 else 2e-2) * np.abs(want).max()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("experts,identity,top,ff,groups", [(5, 3, 2, 40, (4, 2)), (3, 0, 3, 24, (1, 1)), (6, 6, 4, 88, (3, 2)), (60, 12, 5, 9, (9, 4)),
                                                            (2, 6, 2, 16, (2, 1)), (7, 1, 8, 24, (2, 2)), (40, 24, 6, 32, None)])
def test_corrected_choice_within_groups_and_identity_units(dtype, experts, identity, top, ff, groups):
    """The score plus correction chooses, within the groups whose best choice score is largest; the score itself weighs; an
    identity returns its input.  The corrections reach below zero (a group that is not kept must count as minus infinity, not
    as zero) and change choices.  The sum goes into a stream with a factor, on top of a product that waits for it, or is left
    as it is."""
    from infinicore_infer_b200 import kernels as K
    from infinicore_infer_b200.config import RoutedExpertsSpec
    from infinicore_infer_b200.parts import RoutedExperts, Runtime
    from infinicore_infer_b200.weights import DictWeights
    dev, dt = torch.device("cuda:0"), DTYPES[dtype]
    g = torch.Generator().manual_seed(experts + identity)
    d, N = 48, experts + identity
    bf = lambda t: t.to(torch.bfloat16).double()
    W = {"router": bf(torch.randn(N, d, generator=g) * 0.3).numpy(), "correction": bf(0.2 * torch.randn(N, generator=g) - 0.4).numpy()}
    for e in range(experts):
        W[f"e{e}.gate"], W[f"e{e}.up"] = (bf(torch.randn(ff, d, generator=g) * 1.5 * d ** -0.5).numpy() for _ in range(2))
        W[f"e{e}.down"] = bf(torch.randn(d, ff, generator=g) * 2.0 * ff ** -0.5).numpy()
    router = {"experts": experts, "identity": identity, "top": top}
    if groups:
        router["groups"] = dict(zip(("count", "keep"), groups))
    mlp = {"router": router, "expert": {"ff": ff}}
    spec = RoutedExpertsSpec(hidden_size=d, num_experts=experts, num_identity=identity, top=top, expert_size=ff, act="silu", scale_input=False,
                             score_form="softmax", correction_name="correction", groups=groups)
    part = RoutedExperts(spec, DictWeights({n: torch.tensor(a) for n, a in W.items()}, dt, dev), "", Runtime(dt, dev))
    told = {"correction": False, "groups": False, "identity": False}
    for T in (1, 5, 200):
        h = torch.randn(T, d, generator=g, dtype=F) * 2.0
        if dt == torch.bfloat16:
            h = bf(h)
        margins = []
        want = plain.experts_ff(h.numpy(), mlp, W, "", margins)
        chosen, _ = plain.route(h.numpy(), W, "", router)
        told["identity"] |= bool((chosen >= experts).any())
        told["correction"] |= bool((chosen != plain.route(h.numpy(), dict(W, correction=0 * W["correction"]), "", router)[0]).any())
        told["groups"] |= bool((chosen != plain.route(h.numpy(), W, "", {"top": top})[0]).any())
        sure = margins[0] >= {"float32": 1e-6, "bfloat16": 1e-4}[dtype]        # the inputs are the same bits: only the sums' order differs
        tol = (2e-5 if dt == torch.float32 else 2e-2) * np.abs(want).max()
        got = part.forward(h.to(dt).to(dev).contiguous(), None).double().cpu().numpy()
        err = (np.abs(got - want).max(1) * sure).max()
        assert err <= tol, f"{T} rows: {err}"
        x, pend = torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
        for waits in (False, True):
            xd = x.to(dev).clone()
            K.routed_experts(h.to(dt).to(dev).contiguous(), part.router, part.w_gate_up, part.w_down, torch.empty(T, d, device=dev), False, experts, top,
                             K.ACT_SILU, score_form=2, identity=identity, groups=groups or (0, 0), correction=part.correction, x=xd, x_scale=0.3,
                             pending=pend.to(dev) if waits else None, pending_scale=0.7)
            into = x.double().numpy() + 0.3 * want + (0.7 * pend.double().numpy() if waits else 0.0)
            err = (np.abs(xd.double().cpu().numpy() - into).max(1) * sure).max()
            assert err <= tol + 1e-6, f"{T} rows into the stream: {err}"
    assert told["correction"] or top == N
    assert told["groups"] or groups is None or groups[1] in (groups[0], top)       # the best `top` lie in the best `top` groups
    assert told["identity"] or identity == 0


# ---- generation through the scheduler ---------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler_matches_the_plain_model(folders):
    """Requests of unequal length through ``Generator`` (admission, portions of 16 tokens, decoding beside prompts, three
    slots for five requests): every generated token is the plain model's argmax given the tokens before it."""
    from infinicore_infer_b200.engine import Engine, Generator
    d, cfg, w = folders["borrowed"]
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
    """``--random fupapel-tiny`` with three prompts through the scheduler, greedy: the printed tokens are the plain model's."""
    import re
    import subprocess
    import sys
    from infinicore_infer_b200.config import PRESETS, FupapelConfig
    from infinicore_infer_b200.weights import index_directory, read_tensor, write_model_folder
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    preset = PRESETS["fupapel-tiny"]
    proc = subprocess.run([sys.executable, "-m", "infinicore_infer_b200.jiuge", "--nvidia", "--random", "fupapel-tiny", "--seed", "3",
                           "--prompt-lens", "2,19,40", "--chunk-size", "11", "--num-pages", "24", "--max-batch", "3",
                           "--max-tokens-per-step", "24", "--temperature", "0", "--max-steps", "8", "--dtype", "float32"],
                          capture_output=True, text=True, cwd=root, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = {int(m.group(1)): [int(t) for t in m.group(2).split()] for m in re.finditer(r"request (\d+): ([\d ]*)", proc.stdout)}
    assert sorted(got) == [0, 1, 2]
    cfg = FupapelConfig.from_dict(preset.config)
    write_model_folder(cfg, str(tmp_path), seed=3, std=preset.std, norm_std=preset.norm_std)
    w = {n: read_tensor(i).double().numpy() for n, i in index_directory(str(tmp_path)).items()}
    for k, n in enumerate((2, 19, 40)):
        prompt = torch.randint(0, cfg.vocab, (n,), generator=torch.Generator().manual_seed(3 + k)).tolist()
        assert len(got[k]) == 8
        logits = plain.forward(cfg.to_dict(), w, prompt + got[k])
        for j, tok in enumerate(got[k]):
            row = logits[n + j - 1]
            assert tok == int(row.argmax()) or row.max() - row[tok] < 1e-4 * np.abs(row).max(), f"request {k}, token {j}"
