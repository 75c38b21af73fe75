"""Mamivik decoders on the host: the plain statement of the mechanisms by hand, the configuration reader and the checkpoint audit.
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

def test_windowed_attention_by_hand():
    q, k = np.ones((3, 1, 1)), np.log(np.array([1.0, 3.0, 5.0])).reshape(3, 1, 1)
    v = np.array([4.0, 8.0, 2.0]).reshape(3, 1, 1)
    assert np.allclose(mixers.windowed_attention(q, k, v, 1.0, 2)[:, 0, 0], [4, (4 + 24) / 4, (24 + 10) / 8])
    assert np.allclose(mixers.windowed_attention(q, k, v, 1.0, 1)[:, 0, 0], [4, 8, 2])
    assert np.allclose(mixers.windowed_attention(q, k, v, 1.0, 9, sink=np.log([4.0]))[:, 0, 0], [4 / 5, 28 / 8, 38 / 13])


def test_values_are_the_keys_before_they_turn():
    # width 2, one head of 2 dimensions that turn by a quarter per position; a window of one: the output is the key itself
    W = {"q": np.eye(2), "k": np.array([[1.0, 0.0], [0.0, 2.0]]), "q.b": np.zeros(2), "k.b": np.array([0.5, 0.0]), "o": np.eye(2)}
    cfg = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=1.0, rot=dict(dims=2, base=1e4), mask=dict(size=1))
    h = np.array([[1.0, 1.0], [3.0, -1.0]])
    assert np.allclose(mixers.shared_kv_attention(h, W, cfg), [[1.5, 2.0], [3.5, -2.0]])


def test_channel_delta_rule_by_hand():
    # one head of two key channels; a second value column stays empty
    r = np.array([[[1.0, 1.0]], [[2.0, 1.0]]])
    k = np.array([[[3.0, 4.0]], [[0.0, 2.0]]])
    v = np.array([[[1.0, 0.0]], [[5.0, 0.0]]])
    w = np.array([[[0.9, 0.9]], [[0.5, 0.25]]])
    a = np.array([[[0.7, 0.7]], [[0.1, 0.5]]])
    o, S = mixers.channel_delta_rule(r, k, v, w, a)
    # S1 = (3, 4); the second unit key is (0, 1) and sees 4: S2 = (3 / 2 - 0, 4 / 4 - 0.5 * 4 + 2 * 5)
    assert np.allclose(S[0, :, 0], [1.5, 9.0], atol=1e-5) and np.allclose(S[0, :, 1], 0)
    assert np.allclose(o[:, 0, 0], [7, 12], atol=1e-5)


def test_removal_by_the_projected_key():
    """What the kernels do: a k / (sum k^2 + 1e-6) times (k^T S)."""
    rng = np.random.default_rng(0)
    k, a, S = rng.standard_normal(5), rng.uniform(0, 1, 5), rng.standard_normal((5, 3))
    u = mixers.unit(k)
    assert np.allclose(np.outer(a * u, u @ S), np.outer(a * k / (np.sum(k * k) + 1e-6), k @ S))


def test_channel_delta_state_is_carried():
    rng = np.random.default_rng(0)
    r, k, v = (rng.standard_normal((9, 2, 4)) for _ in range(3))
    w, a = rng.uniform(0.5, 1, (9, 2, 4)), rng.uniform(0, 1, (9, 2, 4))
    whole, S = mixers.channel_delta_rule(r, k, v, w, a)
    x, S1 = mixers.channel_delta_rule(r[:4], k[:4], v[:4], w[:4], a[:4])
    y, S2 = mixers.channel_delta_rule(r[4:], k[4:], v[4:], w[4:], a[4:], S1)
    assert np.allclose(np.concatenate([x, y]), whole) and np.allclose(S, S2)


def test_bounded_decay_has_its_bounds():
    one = np.ones((1, 1))
    assert np.allclose(mixers.bounded_decay(one, 0 * one, one, np.array([-50.0, 0.0, 50.0]))[0], [1, np.exp(-0.5 * np.exp(-0.5)), np.exp(-np.exp(-0.5))])


def test_rotated_latents_by_hand():
    # one head, latent of one value, one unrotated dimension, two that turn; a window of one: scores do not matter but for the sink
    W = {"dq": np.array([[1.0]]), "dq.norm": np.ones(1), "uq": np.array([[1.0], [0.5], [0.0]]), "dkv": np.array([[2.0], [1.0], [0.0]]), "dkv.norm": np.array([3.0]),
         "uk": np.array([[1.0]]), "uv": np.array([[4.0]]), "sink": np.array([0.0]), "g": np.array([[0.0]]), "o": np.array([[1.0]])}
    cfg = dict(heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, rot_dim=2, scale=0.1, mask=dict(size=1), rot=dict(dims=2, base=1e4, scaling=None))
    # c_q = 1, c = 3; the score is (1 * 3 + 0.5 * 1 at the same angle) / 10, the value 12, the gate 1/2
    out = mixers.rotated_latent_attention(np.array([[1.0], [1.0]]), W, cfg, 0.0)
    assert np.allclose(out, 6 * np.exp(0.35) / (np.exp(0.35) + 1))
    cfg["mask"]["size"] = 2
    turned = np.array([0.35, 0.3 + 0.05 * np.cos(1.0)])   # the second token's scores: itself, and the first one an angle of 1 away
    out = mixers.rotated_latent_attention(np.array([[1.0], [1.0]]), W, cfg, 0.0)[1, 0]
    assert np.allclose(out, 6 * np.exp(turned).sum() / (np.exp(turned).sum() + 1))


def test_convolution_adds_to_its_input():
    cfg = mc.mamivik([mc.scaled_parallel((1, 1, 4, 2), (1, 4), 3)], width=8, vocab=5, taps=3)
    w = mc.weights(cfg)
    d = mixers.decoder(cfg, w)
    for t in ([1], [1, 2, 3, 4]):
        x = d.embedding_output(np.array(t))
        h = x / np.sqrt(np.mean(x * x, axis=1, keepdims=True) + cfg["norm"]["eps"]) * d.w["l0.norm1"]
        want = h.copy()
        for i in range(len(t)):
            for j in range(3):
                if i - 2 + j >= 0:
                    want[i] += d.w["l0.canon1"][:, j] * h[i - 2 + j]
        got = mixers.scaled_parallel_mixer(want, d._sub("l0.mix."), cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
        assert np.allclose(d.residuals(t)[0], x + got)


# ------------------------------------------------------------------------------------------------ configuration, audit

LAYERS = [mc.scaled_parallel((4, 2, 16, 8), (2, 12), 24, ff=30), mc.rotated_latent(3, 16, 20, 12, 10, 6, 40), mc.scaled_parallel((2, 1, 8, 8), (3, 8), 5)]


def folder(tmp_path, change_cfg=None, change_w=None):
    cfg = json.loads(json.dumps(mc.mamivik(LAYERS, width=40)))
    w = mc.weights(cfg)
    if change_cfg:
        change_cfg(cfg)
    if change_w:
        change_w(w)
    return mc.write(tmp_path / "m", cfg, w)


def test_inspect_reads_the_description(eng, tmp_path):
    s = eng.Model.inspect_mixer(folder(tmp_path))
    w = mc.weights(mc.mamivik(LAYERS, width=40))
    assert (s["architecture"], s["vocab_size"], s["hidden_size"], s["n_layers"], s["layer_runs"]) == ("Mamivik", 131, 40, 3, 3)
    assert (s["parallel_layers"], s["latent_layers"], s["ffn_layers"], s["attention_layers"]) == (2, 1, 1, 0)
    assert s["tensors_in_file"] == s["tensors_read"] == len(w)
    assert s["parameters"] == sum(a.size for a in w.values())


@pytest.mark.parametrize("change,message", [
    (lambda w: w.pop("l0.canon1"), "`l0.canon1` is missing"),
    (lambda w: w.pop("l1.mix.sink"), "`l1.mix.sink` is missing"),
    (lambda w: w.pop("l2.mix.left.k.b"), "`l2.mix.left.k.b` is missing"),
    (lambda w: w.pop("l0.mix.right.a.b"), "`l0.mix.right.a.b` is missing"),
    (lambda w: w.pop("l0.mlp.gate"), "`l0.mlp.gate` is missing"),
    (lambda w: w.update({"l0.norm1": np.zeros(40, np.float32)}), "`l0.norm1` has shape [40], expected []"),
    (lambda w: w.update({"l1.mix.dkv": np.zeros((10, 40), np.float32)}), "`l1.mix.dkv` has shape [10, 40], expected [16, 40]"),
    (lambda w: w.update({"l1.mix.uq": np.zeros((48, 12), np.float32)}), "`l1.mix.uq` has shape [48, 12], expected [66, 12]"),
    (lambda w: w.update({"l1.mix.g": np.zeros((3, 40), np.float32)}), "`l1.mix.g` has shape [3, 40], expected [60, 40]"),
    (lambda w: w.update({"l0.mix.right.w1": np.zeros(40, np.float32)}), "`l0.mix.right.w1` must be a matrix"),
    (lambda w: w.update({"l0.canon1": np.zeros((40, 4), np.float32)}), "`l0.canon1` has shape [40, 4], expected [40, 3]"),
])
def test_audit_names_the_tensor(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(folder(tmp_path, change_w=change))
    assert message in str(e.value)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="wkv"), "config.layers[0].type `wkv` is not a known mixer"),
    (lambda c: c.pop("canon"), "config.canon is missing"),
    (lambda c: c["canon"].update(taps=0), "config.canon.taps is out of range"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "config.layers[0].mixer.left_scale is missing"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=12), "config.layers[0].mixer.left.vdim must be dim"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "heads must be a multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("mask"), "config.layers[0].mixer.left.mask is missing"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling=mc.YARN), "config.layers[0].mixer.left.rot.scaling is not supported here"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "config.layers[1].mixer.mask.size is out of range"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "config.layers[1].mixer.rot.dims is out of range"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "config.layers[1].mixer.rot.scaling.slow is missing"),
    (lambda c: c["layers"][1]["mixer"].pop("rot_dim"), "config.layers[1].mixer.rot_dim is missing"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind `moe` is not supported"),
])
def test_reader_names_the_setting(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(folder(tmp_path, change_cfg=change))
    assert message in str(e.value)
