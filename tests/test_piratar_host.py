"""Piratar without a GPU: the configuration, the manifest, what is kept per request, and the plain implementation's own small
cases."""
import numpy as np
import pytest

import plain_piratar as plain
from infinicore_infer_b200.config import ConfigError, PiratarConfig, config_class_for
from infinicore_infer_b200.parts import cache_needs, model_manifest, state_needs


def cfg():
    layers = [
        {"type": "parallel", "mixer": {
            "left": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.3, "conv": 3, "rot": {"base": 100.0, "dims": 4}},
            "right": {"heads": 3, "dim": 8, "vdim": 5, "decay": [0.5, 0.75, 0.99], "rot": {"base": 50.0, "dims": 8}}},
         "mlp": {"kind": "moe", "router": {"experts": 5, "top": 2, "scale": 1.25}, "expert": {"ff": 8}, "shared": {"ff": 12}}},
        {"type": "rglru", "mixer": {"width": 24, "blocks": 3, "conv": 4}, "mlp": {"kind": "dense", "ff": 20}},
        {"type": "parallel", "mixer": {
            "left": {"heads": 2, "kv_heads": 2, "dim": 4, "vdim": 4, "scale": 0.5, "conv": 1},
            "right": {"heads": 1, "dim": 4, "vdim": 6, "decay": [0.9], "rot": {"base": 10.0, "dims": 2}}},
         "mlp": {"kind": "moe", "router": {"experts": 3, "top": 3}, "expert": {"ff": 4}}},
        {"type": "rglru", "mixer": {"width": 10, "blocks": 1, "conv": 1}, "mlp": None},
    ]
    return {"architecture": "Piratar", "norm": {"eps": 1e-5}, "vocab": 40, "width": 16, "embedding": {"scale": 3.0, "bigram": {"buckets": 11, "mul_prev": 5, "mul_cur": 3}},
            "token_side": {"dim": 6}, "layers": layers}


def test_the_registry_finds_the_configuration_and_it_reads_back():
    c = config_class_for(cfg())
    assert c is PiratarConfig
    typed = c.from_dict(cfg(), max_tokens=48)
    assert typed.max_positions == 48 and typed.embed_scale == 3.0 and not typed.tie_word_embeddings
    assert PiratarConfig.from_dict(typed.to_dict(), max_tokens=48) == typed
    spec = typed.model_spec()
    assert all(b.joined and b.shift_name is None and b.mixer_norm.one_plus for b in spec.layers) and spec.embed_norm.one_plus
    assert (spec.pairs.buckets, spec.pairs.mul_prev, spec.pairs.mul_cur) == (11, 5, 3)
    m = spec.layers[0].mixer
    assert m.left_scale == m.right_scale == 0.5 and not m.left_norm.one_plus and m.left.element_gate and m.left.conv_taps == 3
    assert m.left.window is None and m.left.position.layout == "halves" and m.left.position.dims == 4
    assert m.right.decay == (0.5, 0.75, 0.99) and m.right.q_scale == 8 ** -0.5 and m.right.norm_name is None and m.right.position.base == 50.0
    e = spec.layers[0].feed_forward
    assert (e.num_experts, e.top, e.score_form, e.score_scale, e.shared_gate_name, e.shared.intermediate_size) == (5, 2, "softmax_renorm", 1.25, "sg", 12)
    assert spec.layers[2].mixer.left.position is None and spec.layers[2].feed_forward.shared is None and spec.layers[2].feed_forward.score_scale == 1.0
    assert spec.layers[1].mixer.rate == 8.0 and spec.layers[1].feed_forward.intermediate_size == 20 and spec.layers[3].feed_forward is None
    assert [(e.after.offset, e.after.table_width, e.after.gate_name) for e in spec.order] == [(6 * i, 24, f"l{i}.side.gate") for i in range(4)]


def test_what_a_request_keeps():
    spec = PiratarConfig.from_dict(cfg()).model_spec()
    needs, states = cache_needs(spec), state_needs(spec)
    assert (needs[0].num_kv_heads, needs[0].head_dim, needs[0].v_head_dim, needs[0].window) == (2, 6, 10, None)
    assert (needs[2].num_kv_heads, needs[2].head_dim, needs[2].v_head_dim) == (2, 4, None)
    assert needs[1].shape == (24,) and needs[3].shape == (10,)
    # left: the tails of [q | k | v]; right: S per head; a recurrence's tails; last of all the embedding's token
    assert [s.shape for s in states[0].slots] == [(2, 24 + 12 + 20), (3, 8, 5)]
    assert states[1].shape == (3, 24) and [s.shape for s in states[2].slots] == [(1, 4, 6)] and states[3] is None
    assert len(states) == 5 and states[4].shape == (2, 2)
    plainer = cfg()
    plainer["embedding"]["bigram"] = None
    plainer["token_side"] = None
    spec = PiratarConfig.from_dict(plainer).model_spec()
    assert len(state_needs(spec)) == 4 and all(e.after is None for e in spec.order)
    assert not any(n.startswith(("bigram", "side.")) or ".side." in n for n in model_manifest(spec))


def test_manifest_names_every_tensor_once():
    names = model_manifest(PiratarConfig.from_dict(cfg()).model_spec())
    shape = lambda n: names[n].shape
    assert shape("embed") == shape("head") == (40, 16) and shape("bigram") == (12, 16) and shape("side.embed") == (40, 24)
    assert shape("embed.norm") == shape("final.norm") == shape("l0.norm1") == shape("l0.norm2") == (16,)
    assert shape("l0.mix.left.q") == (24, 16) and shape("l0.mix.left.k") == (12, 16) and shape("l0.mix.left.v") == (20, 16)
    assert shape("l0.mix.left.v.conv") == (20, 3) and shape("l0.mix.left.g") == (40, 16) and shape("l0.mix.left.o") == (16, 40)
    assert shape("l0.mix.left.out") == shape("l0.mix.right.out") == (16,) and "l0.mix.right.norm" not in names
    assert shape("l0.mix.right.q") == shape("l0.mix.right.k") == (24, 16) and shape("l0.mix.right.v") == shape("l0.mix.right.g") == (15, 16)
    assert shape("l0.mlp.router") == (5, 16) and shape("l0.mlp.e4.down") == (16, 8) and shape("l0.mlp.shared.sg") == (1, 16)
    assert shape("l0.side.gate") == (6, 16) and shape("l0.side.proj") == (16, 6) and shape("l0.side.norm") == (16,)
    assert shape("l1.mix.y") == shape("l1.mix.x") == (24, 16) and shape("l1.mix.y.b") == shape("l1.mix.conv.b") == shape("l1.mix.lam") == (24,)
    assert shape("l1.mix.conv") == (24, 4) and shape("l1.mix.ra") == shape("l1.mix.ri") == (3, 8, 8) and shape("l1.mix.ri.b") == (3, 8)
    assert shape("l1.mlp.gate") == (20, 16) and "l2.mlp.shared.sg" not in names and "l3.norm2" not in names and "l3.side.proj" in names


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["right"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "experts"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "heads"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][1]["mixer"].update(blocks=5), "parts"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c["embedding"]["bigram"].update(mul_prev=-1), "mul_prev"),
    (lambda c: c["token_side"].pop("dim"), "dim"),
])
def test_what_the_configuration_refuses(change, what):
    c = cfg()
    change(c)
    with pytest.raises(ConfigError, match=what):
        PiratarConfig.from_dict(c)


def test_pairs_of_tokens_by_hand():
    pairs = {"buckets": 10, "mul_prev": 7, "mul_cur": 3}
    assert plain.bigram_rows([4, 5, 5], pairs).tolist() == [10, (28 + 15) % 10, (35 + 15) % 10]
    assert plain.bigram_rows([5, 5], pairs, before=4).tolist() == plain.bigram_rows([4, 5, 5], pairs)[1:].tolist()


def test_retention_and_the_gated_recurrence_by_hand():
    q, k, v = np.array([[[1.0, 0.0]], [[2.0, 1.0]]]), np.array([[[3.0, 1.0]], [[0.0, 2.0]]]), np.array([[[5.0]], [[7.0]]])
    out, S = plain.retention_scan(q, k, v, [0.5])
    # S_1 = (15, 5); S_2 = (7.5, 2.5 + 14)
    assert out.ravel().tolist() == [15.0, 2 * 7.5 + 16.5] and S.ravel().tolist() == [7.5, 16.5]
    later, _ = plain.retention_scan(q[1:], k[1:], v[1:], [0.5], state=np.array([[[15.0], [5.0]]]))
    assert later.ravel().tolist() == [31.5]
    lam = np.array([0.3])
    a = np.exp(-8.0 * 0.25 * np.log1p(np.exp(0.3)))
    got, last = plain.gated_linear_scan(np.array([[2.0], [1.0]]), np.full((2, 1), 0.25), np.array([[0.5], [1.0]]), lam)
    s1 = np.sqrt(1 - a * a) * 0.5 * 2.0
    assert np.allclose(got.ravel(), [s1, a * s1 + np.sqrt(1 - a * a)]) and last == got[-1]
    blocks = plain.block_maps(np.array([[1.0, 2.0, 3.0, 4.0]]), np.array([[[1.0, 1.0], [0.0, 1.0]], [[2.0, 0.0], [0.0, 3.0]]]), np.array([[0.0, 1.0], [0.0, 0.0]]))
    assert blocks.tolist() == [[3.0, 3.0, 6.0, 12.0]]


def test_renormalised_and_scaled_scores_by_hand():
    W = {"router": np.log(np.array([[1.0], [2.0], [5.0]]))}
    chosen, weight = plain.route(np.array([[1.0]]), W, "", {"top": 2, "scale": 3.0})
    assert chosen.tolist() == [[2, 1]] and np.allclose(weight, [[15.0 / 7.0, 6.0 / 7.0]])
