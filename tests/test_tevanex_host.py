"""Tevanex decoders on the host: the plain statement of the mechanisms by hand, the configuration reader and the checkpoint audit.
No GPU."""
import importlib
import json

import numpy as np
import pytest

from oracle import mixers
import mixer_cases as mc


@pytest.fixture(scope="module")
def eng(mk):
    return importlib.import_module("macllm_infer_b200.engine")


@pytest.fixture(scope="module")
def capi(mk):
    return importlib.import_module("macllm_infer_b200._capi")


# ------------------------------------------------------------------------------------------------ the plain statement

def test_mlstm_rule_by_hand():
    # one head, key width 2, value width 1
    q, k = np.array([[[1.0, 0.0]], [[0.5, 2.0]]]), np.array([[[2.0, 1.0]], [[0.0, 1.0]]])
    v, i, f = np.array([[[3.0]], [[5.0]]]), np.log(np.array([[4.0], [0.5]])), np.log(np.array([[0.5], [0.25]]))
    o, (S, n, m) = mixers.mlstm_rule(q, k, v, i, f)
    # without the maximum S1 = 4 k1 3 = (24, 12), n1 = (8, 4); S2 = S1 / 4 + 0.5 k2 5 = (6, 5.5), n2 = (2, 1.5)
    # the maxima are 4 and max(4 / 4, 1/2) = 1, so the floor of the denominators is 1/4 and 1
    assert np.allclose(o[0, 0], 24 / 4 / (8 / 4 + 1e-6)) and np.allclose(o[1, 0], (3 + 11) / (1 + 3 + 1e-6))
    assert np.allclose(m, 0) and np.allclose(S[0, :, 0], [6, 5.5]) and np.allclose(n[0], [2, 1.5])


def test_mlstm_starts_from_a_maximum_of_zero_and_has_a_floor():
    one = np.ones((1, 1, 1))
    # a write of e^-9 against a starting maximum of 0 that decays to -2: the floor e^2 is what divides
    o, (S, n, m) = mixers.mlstm_rule(one, one, 7 * one, np.full((1, 1), -9.0), np.full((1, 1), -2.0))
    assert np.allclose(m, -2) and np.allclose(S, 7 * np.exp(-7)) and np.allclose(o, 7 * np.exp(-7) / (np.exp(2) + 1e-6))


def test_mlstm_gates_and_carried_state():
    i, f = mixers.mlstm_gates(np.array([0.0, 1e9]), np.array([0.0, 1e9]), 3.0)
    assert np.allclose(i, [0, 3]) and np.allclose(f, [np.log(0.5), -np.log1p(np.exp(-3))])
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3))
    i, f = 4 * rng.standard_normal((9, 2)), -rng.uniform(0, 3, (9, 2))
    whole, _ = mixers.mlstm_rule(q, k, v, i, f)
    a, state = mixers.mlstm_rule(q[:4], k[:4], v[:4], i[:4], f[:4])
    b, _ = mixers.mlstm_rule(q[4:], k[4:], v[4:], i[4:], f[4:], state)
    assert np.allclose(np.concatenate([a, b]), whole)


def test_chunked_attention_by_hand():
    q, k = np.ones((3, 1, 1)), np.log(np.array([1.0, 3.0, 5.0])).reshape(3, 1, 1)
    v = np.array([4.0, 8.0, 2.0]).reshape(3, 1, 1)
    o = mixers.chunked_attention(q, k, v, 1.0, 2)
    assert np.allclose(o[:, 0, 0], [4, (4 + 24) / 4, 2])
    o = mixers.chunked_attention(q, k, v, 1.0, 2, sink=np.log([4.0]))
    assert np.allclose(o[:, 0, 0], [4 / 5, 28 / 8, 10 / 9])
    o = mixers.chunked_attention(q, 1e6 * k, v, 1.0, 3, softcap=np.log(3.0))       # scores 0 and two of log 3
    assert np.allclose(o[2, 0, 0], (4 + 24 + 6) / 7)


def test_rotation_turns_halves():
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    out = mixers.rotate_half(x, [2], 4, np.array([np.pi / 4, np.pi / 2]))          # pairs (0, 2) and (1, 3): quarter and half turns
    assert np.allclose(out[0, 0], [-3, -2, 1, -4, 5, 6])


def test_clamped_expert_and_routing_by_hand():
    W = {"gate": np.array([[2.0]]), "up": np.array([[-3.0]]), "down": np.array([[10.0]])}
    s = 1 / (1 + np.exp(-1.702 * 1.5))
    assert np.allclose(mixers.clamped_mlp(np.array([[1.0], [-1.0]]), W, 1.5), [[1.5 * s * -0.5 * 10], [-2 / (1 + np.exp(1.702 * 2)) * 2.5 * 10]])
    chosen, weight = mixers.routed(np.array([[1.0]]), {"router": np.array([[0.0], [2.0], [-1.0], [2.0]])}, 3)
    assert chosen.tolist() == [[1, 3, 0]] and np.allclose(weight, [mixers.sigmoid(np.array([2.0, 2.0, 0.0]))])


def test_a_weight_in_front_of_the_activation_is_a_weight_on_the_input():
    """What the kernels do: the weight times the gate and up sums."""
    rng = np.random.default_rng(1)
    W = {"gate": rng.standard_normal((5, 4)), "up": rng.standard_normal((5, 4)), "down": rng.standard_normal((4, 5))}
    h = rng.standard_normal((3, 4))
    scaled = {**W, "gate": 0.3 * W["gate"], "up": 0.3 * W["up"]}
    assert np.allclose(mixers.clamped_mlp(0.3 * h, W, 0.4), mixers.clamped_mlp(h, scaled, 0.4))
    assert not np.allclose(mixers.clamped_mlp(0.3 * h, W, 0.4), 0.3 * mixers.clamped_mlp(h, W, 0.4))


@pytest.mark.parametrize("dims,base,scaling", [(32, 500.0, mc.YARN), (10, 1e5, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                                               (64, 1e4, dict(factor=2.0, original=300, fast=4.0, slow=4.0)), (8, 50.0, dict(factor=40.0, original=20, fast=1e4, slow=1e-4))])
def test_stretched_frequencies_of_the_loader(capi, dims, base, scaling):
    out, amplitude = np.empty(dims // 2), np.empty(1)
    capi.check(capi.lib().mk_rotary_frequencies_yarn(dims, base, scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"], out.ctypes.data, amplitude.ctypes.data))
    want, m = mixers.yarn_frequencies(dims, base, **scaling)
    assert np.allclose(out, want, rtol=1e-14) and np.isclose(amplitude[0], m)


def test_stretched_frequencies_have_three_regimes():
    f, m = mixers.yarn_frequencies(32, 500.0, 4.0, 64, 8.0, 1.0)
    ratio = f / mixers.rope_frequencies(32, 500.0)
    assert np.isclose(ratio[0], 1) and np.isclose(ratio[-1], 1 / 4) and np.any((ratio > 0.26) & (ratio < 0.99)) and np.isclose(m, 1 + 0.1 * np.log(4))


# ------------------------------------------------------------------------------------------------ configuration, audit

MLP = mc.experts(3, 2, 20, 0.9, (28, 1.1))
LAYERS = [mc.mlstm(2, 12, 10, mlp=MLP), mc.sink_attention(4, 2, 16, 20, 8, 24), mc.capped_attention(2, 1, 24, 12, 24, 40, mlp=mc.experts(5, 1, 16))]
LAYERS = LAYERS + [mc.again(LAYERS, 2), mc.again(LAYERS, 0)]


def folder(tmp_path, change_cfg=None, change_w=None):
    cfg = json.loads(json.dumps(mc.tevanex(LAYERS, width=40)))
    w = mc.weights(cfg)
    if change_cfg:
        change_cfg(cfg)
    if change_w:
        change_w(w)
    return mc.write(tmp_path / "m", cfg, w)


def test_inspect_reads_the_description(eng, tmp_path):
    s = eng.Model.inspect_mixer(folder(tmp_path))
    w = mc.weights(mc.tevanex(LAYERS, width=40))
    assert (s["architecture"], s["vocab_size"], s["hidden_size"], s["n_layers"], s["layer_runs"]) == ("Tevanex", 131, 40, 5, 5)
    assert (s["mlstm_layers"], s["attention_layers"], s["ffn_layers"], s["experts"]) == (2, 3, 4, 5)
    assert s["tensors_in_file"] == s["tensors_read"] == len(w)
    assert s["parameters"] == sum(a.size for a in w.values())


@pytest.mark.parametrize("change,message", [
    (lambda w: w.pop("l0.mlp.e2.up"), "`l0.mlp.e2.up` is missing"),
    (lambda w: w.pop("l1.mix.sink"), "`l1.mix.sink` is missing"),
    (lambda w: w.pop("l2.mix.g"), "`l2.mix.g` is missing"),
    (lambda w: w.pop("l0.mlp.shared.sg"), "`l0.mlp.shared.sg` is missing"),
    (lambda w: w.update({"l1.mix.q.norm": np.zeros(16, np.float32)}), "`l1.mix.q.norm` has shape [16], expected [64]"),
    (lambda w: w.update({"l0.mix.f.b": np.zeros(3, np.float32)}), "`l0.mix.f.b` has shape [3], expected [2]"),
    (lambda w: w.update({"l2.mlp.router": np.zeros((4, 40), np.float32)}), "`l2.mlp.router` has shape [4, 40], expected [5, 40]"),
])
def test_audit_names_the_tensor(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(folder(tmp_path, change_w=change))
    assert message in str(e.value)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="wkv"), "config.layers[0].type `wkv` is not a known mixer"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "config.layers[1].mixer.mask is missing"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "config.layers[1].mixer.mask.size is out of range"),
    (lambda c: c["layers"][2]["mixer"].pop("softcap"), "config.layers[2].mixer.softcap is missing"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("fast"), "config.layers[2].mixer.rot.scaling.fast is missing"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(scaling=mc.YARN), "config.layers[1].mixer.rot.scaling is not supported here"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "heads must be a multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0), "gate_cap must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind `dense` is not supported"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), "config.layers[0].mlp.router.top is out of range"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "config.layers[0].mlp.expert.limit is missing"),
    (lambda c: c["layers"][3].update(weights_of=5), "config.layers[3].weights_of is out of range"),
    (lambda c: c["layers"][3].update(weights_of=0), "config.layers[3].weights_of names a layer of another kind"),
    (lambda c: c["layers"][3].update(weights_of=3), "config.layers[3].weights_of goes round in a circle"),
    (lambda c: c.pop("logit_softcap"), "config.logit_softcap is missing"),
    (lambda c: c["embedding"].pop("scale"), "config.embedding.scale is missing"),
])
def test_reader_names_the_setting(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(folder(tmp_path, change_cfg=change))
    assert message in str(e.value)

