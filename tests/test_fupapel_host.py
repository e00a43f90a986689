"""Fupapel without a GPU: the configuration, borrowed caches, the manifest, what is kept per request, the stretched
frequencies, and the plain implementation's own small cases."""
import numpy as np
import pytest

import plain_fupapel as plain
from infinicore_infer_b200.config import ConfigError, FrequencyBandSpec, FupapelConfig, PairRotarySpec, config_class_for
from infinicore_infer_b200.parts import cache_needs, model_manifest, state_needs


def cfg():
    layers = [
        {"type": "attention_2", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.3, "conv": 3, "mask": {"size": 5},
                                          "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 16}}},
         "mlp": {"kind": "moe", "router": {"experts": 5, "identity": 3, "top": 2, "groups": {"count": 4, "keep": 2}}, "expert": {"ff": 8}}},
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 4, "scale": 0.4, "mask": {"size": 7}, "rot": {"base": 50.0, "dims": 8}},
         "mlp": None},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 4, "rot_dim": 6, "vdim": 10, "kv_rank": 8, "q_rank": 12, "scale": 0.4,
                                               "rot": {"base": 1000.0, "dims": 6}},
         "mlp": {"kind": "moe", "router": {"experts": 2, "identity": 0, "top": 2, "groups": {"count": 1, "keep": 1}}, "expert": {"ff": 4}}},
        {"type": "attention_2", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.3, "conv": 2, "mask": {"size": 9}, "kv_from": 0,
                                          "rot": {"base": 100.0, "dims": 4}},
         "mlp": None},
    ]
    return {"architecture": "Fupapel", "norm": {"eps": 1e-5}, "vocab": 40, "width": 16, "residual_mult": 0.4, "layers": layers}


def test_the_registry_finds_the_configuration_and_it_reads_back():
    c = config_class_for(cfg())
    assert c is FupapelConfig
    typed = c.from_dict(cfg(), max_tokens=48)
    assert typed.max_positions == 48 and typed.residual_mult == 0.4 and not typed.tie_word_embeddings
    assert FupapelConfig.from_dict(typed.to_dict(), max_tokens=48) == typed
    spec = typed.model_spec()
    assert [b.residual_scale for b in spec.layers] == [0.4] * 4 and all(b.shift_name == "shift" for b in spec.layers)
    assert spec.layers[1].feed_forward is None and spec.layers[1].ffn_norm is None
    e = spec.layers[0].feed_forward
    assert (e.num_experts, e.num_identity, e.top, e.groups, e.score_form, e.correction_name) == (5, 3, 2, (4, 2), "softmax", "correction")
    a, b = spec.layers[1].mixer, spec.layers[0].mixer
    assert a.element_gate and a.sink and a.sink_name is None and a.temp_name is None and a.chunk == 7 and a.conv_taps == 0 and a.qk_norm
    assert b.sink_name == "sink" and b.temp_name == "temp" and not b.element_gate and b.conv_taps == 3 and b.position.scaling.high == 4.0
    assert spec.layers[2].mixer.output_gate == "head" and spec.layers[2].mixer.position.layout == "halves"


def test_a_layer_that_borrows_its_keys_reads_the_writers_cache():
    spec = FupapelConfig.from_dict(cfg()).model_spec()
    assert [(e.layer, e.cache, e.writes_cache) for e in spec.order] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 0, False)]
    needs, states = cache_needs(spec), state_needs(spec)
    assert (needs[0].num_kv_heads, needs[0].head_dim, needs[0].v_head_dim, needs[0].window) == (2, 6, 10, 9)      # kept for the wider mask
    assert (needs[1].num_kv_heads, needs[1].head_dim, needs[1].v_head_dim, needs[1].window) == (3, 8, 4, 7)
    assert (needs[2].head_dim, needs[2].v_head_dim, needs[2].window, needs[2].values_in_keys) == (14, 8, None, True)
    # every layer keeps the rows of its shift (two that take turns, each with a word behind it); convolutions their tails
    shapes = [[s.shape for s in st.slots] for st in states]
    assert shapes == [[(2, 20), (2, 24 + 12 + 20)], [(2, 20)], [(2, 20)], [(2, 20), (1, 24)]]


def test_manifest_names_every_tensor_once():
    names = model_manifest(FupapelConfig.from_dict(cfg()).model_spec())
    assert names["embed"].shape == (40, 16) and names["head"].shape == (40, 16) and names["final.norm"].shape == (16,)
    assert names["l0.mix.q"].shape == (24, 16) and names["l0.mix.k"].shape == (12, 16) and names["l0.mix.v"].shape == (20, 16)
    assert names["l0.mix.q.norm"].shape == (24,) and names["l0.mix.k.norm"].shape == (12,) and names["l0.mix.v.conv"].shape == (20, 3)
    assert names["l0.mix.temp"].shape == (4,) and names["l0.mix.sink"].shape == (4,) and names["l0.mix.o"].shape == (16, 40)
    assert names["l0.mlp.router"].shape == (8, 16) and names["l0.mlp.correction"].shape == (8,) and names["l0.mlp.e4.down"].shape == (16, 8)
    assert "l0.mlp.e5.down" not in names and "l0.mix.g" not in names and names["l0.shift"].shape == (16,)
    assert names["l1.mix.g"].shape == (24, 16) and "l1.mix.sink" not in names and "l1.mix.q.conv" not in names and "l1.norm2" not in names
    assert names["l2.mix.dq"].shape == (12, 16) and names["l2.mix.dq.norm"].shape == (12,) and names["l2.mix.uq"].shape == (20, 12)
    assert names["l2.mix.dkv"].shape == (14, 16) and names["l2.mix.dkv.norm"].shape == (8,) and names["l2.mix.uk"].shape == (8, 8)
    assert names["l2.mix.uv"].shape == (20, 8) and names["l2.mix.g"].shape == (2, 16) and names["l2.mix.sink"].shape == (2,)
    assert names["l3.mix.q.conv"].shape == (24, 2) and not any(n.startswith(("l3.mix.k", "l3.mix.v")) for n in names)


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "experts"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
])
def test_what_the_configuration_refuses(change, what):
    c = cfg()
    change(c)
    with pytest.raises(ConfigError, match=what):
        FupapelConfig.from_dict(c)


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, (4.0, 1.0, 4.0, 64)), (64, 5e5, (8.0, 1.0, 4.0, 8192)), (8, 100.0, (2.0, 1.0, 3.0, 40)), (6, 7.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    rot = {"dims": dims, "base": base}
    spec = None
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        factor, low, high, original = scaling
        spec = FrequencyBandSpec(factor=factor, original=original, low=low, high=high)
    got, magnitude = PairRotarySpec(dims=dims, base=base, scaling=spec, layout="halves").frequencies()
    want = plain.rotary_frequencies(rot)
    assert magnitude == 1.0 and np.allclose(got, want, rtol=1e-12)
    if scaling:
        plain_f = plain.rotary_frequencies({"dims": dims, "base": base})
        kinds = {"kept": np.isclose(want, plain_f), "divided": np.isclose(want, plain_f / factor)}
        assert kinds["kept"].any() and kinds["divided"].any()
        between = ~(kinds["kept"] | kinds["divided"])
        assert np.all(want[between] < plain_f[between]) and np.all(want[between] > plain_f[between] / factor)


def test_the_two_kept_rows_take_turns_whatever_the_cuts():
    """The rule by which a step finds the row that the step before left, and where it leaves its own: the row marked with the
    step's first position, and the other one.  Both start marked 0."""
    r = np.random.default_rng(0)
    for _ in range(200):
        marks, holds, pos = [0, 0], [None, None], 0
        for _ in range(12):
            n = int(r.integers(1, 4))
            second = marks[0] != pos
            assert pos == 0 or holds[int(second)] == pos - 1, "the row read is the sequence's last one"
            other = 0 if second else 1
            assert marks[1 - other] != pos + n        # the first row's block cannot take the new mark for its own
            marks[other], holds[other] = pos + n, pos + n - 1
            pos += n


def test_shift_convolution_and_identity_by_hand():
    h = np.array([[4.0, 8.0], [2.0, 2.0], [6.0, 0.0]])
    out = plain.token_shift(h, np.array([0.5, 1.0]))
    assert out.tolist() == [[2.0, 0.0], [3.0, 8.0], [4.0, 2.0]]
    assert np.allclose(plain.token_shift(h[1:], np.array([0.5, 1.0]), before=h[0]), out[1:])
    W = {"router": np.zeros((4, 2)), "correction": np.array([-0.5, -0.9, -0.4, -0.45])}
    # equal scores of 1/4: the group of outputs 2 and 3 is the better one although every choice score is negative
    chosen, weight = plain.route(h, W, "", {"top": 2, "groups": {"count": 2, "keep": 1}})
    assert chosen.tolist() == [[2, 3]] * 3 and np.allclose(weight, 0.25)
    got = plain.experts_ff(h, {"router": {"experts": 2, "identity": 2, "top": 2, "groups": {"count": 2, "keep": 1}}, "expert": {"ff": 1}}, W, "")
    assert np.allclose(got, 0.5 * h)


def test_the_sink_takes_its_share():
    s = np.array([[1.0, -np.inf]])
    assert np.allclose(plain.softmax_with_sink(s, 1.0), [[0.5, 0.0]])
    assert np.allclose(plain.softmax_with_sink(s, 0.0)[0, 0], np.e / (1 + np.e))
    assert np.allclose(plain.softmax_with_sink(s, -50.0), [[1.0, 0.0]])
