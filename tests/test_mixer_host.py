"""Mixer-built decoders on the host: the plain statement of the mechanisms against itself, the configuration reader and the
checkpoint audit, recurrent-state slots in the session and reservation protocol.  No GPU."""
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

def test_delta_rule_by_hand():
    # one head, key width 2, value width 1; the read-out sees the current token's write
    q = np.array([[[1.0, 0.0]], [[0.0, 1.0]]])
    k = np.array([[[1.0, 0.0]], [[0.6, 0.8]]])
    v, g, beta = np.array([[[2.0]], [[3.0]]]), np.array([[0.5], [0.25]]), np.array([[0.5], [1.0]])
    o, S = mixers.delta_rule(q, k, v, g, beta)
    # S1 = k1 * 0.5 * 2 = (1, 0); decayed (0.25, 0); u = 3 - 0.15 = 2.85; S2 = (0.25 + 1.71, 2.28)
    assert np.allclose(o[:, 0, 0], [1.0, 2.28]) and np.allclose(S[0, :, 0], [1.96, 2.28])


def test_wkv_rule_by_hand():
    r = np.array([[[1.0, 2.0]], [[1.0, 1.0]]])
    k = np.array([[[1.0, -1.0]], [[0.5, 0.0]]])
    v = np.array([[[3.0, 0.0]], [[1.0, 1.0]]])
    w, u = np.array([[[0.5, 0.1]], [[0.5, 0.5]]]), np.array([[2.0, 1.0]])
    o, S = mixers.wkv_rule(r, k, v, w, u)
    # o1 = r1 . (u k1) v1 = (2 - 2) * 3 = 0;  S1 = k1 v1^T: the first decay meets an empty state
    # o2 = (S1 + u k2 v2)^T r2 = (3 + 1 - 3 + 0, 0 + 1) = (1, 1)
    assert np.allclose(o[0, 0], [0, 0]) and np.allclose(o[1, 0], [1.0, 1.0])
    assert np.allclose(S[0], [[2.0, 0.5], [-1.5, 0.0]])


def test_recurrences_carry_their_state():
    rng = np.random.default_rng(1)
    T, H, d, e = 11, 4, 5, 3
    q, k, v = rng.standard_normal((T, 2, d)), rng.standard_normal((T, 2, d)), rng.standard_normal((T, H, e))
    g, beta = rng.uniform(0.5, 1, (T, H)), rng.uniform(0, 1, (T, H))
    whole, S = mixers.delta_rule(q, k, v, g, beta)
    a, S1 = mixers.delta_rule(q[:4], k[:4], v[:4], g[:4], beta[:4])
    b, S2 = mixers.delta_rule(q[4:], k[4:], v[4:], g[4:], beta[4:], S1)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(S, S2)
    r, k, v = (rng.standard_normal((T, H, d)) for _ in range(3))
    w, u = rng.uniform(0.5, 1, (T, H, d)), rng.standard_normal((H, d))
    whole, S = mixers.wkv_rule(r, k, v, w, u)
    a, S1 = mixers.wkv_rule(r[:7], k[:7], v[:7], w[:7], u)
    b, S2 = mixers.wkv_rule(r[7:], k[7:], v[7:], w[7:], u, S1)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(S, S2)


def test_causal_conv_and_token_shift_start_from_zeros():
    x = np.array([[1.0], [2.0], [4.0]])
    assert np.allclose(mixers.causal_conv(x, np.array([[10.0, 100.0, 1000.0]]))[:, 0], [1000, 2100, 4210])
    assert np.allclose(mixers.causal_conv(x, np.array([[3.0]]))[:, 0], [3, 6, 12])
    assert np.allclose(mixers.token_shift(x, np.array([0.25]))[:, 0], [0.75, 1.75, 3.5])


def test_rotation_turns_adjacent_pairs():
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    out = mixers.rotate_interleaved(x, [2], 4, np.array([np.pi / 4, np.pi / 2]))     # quarter and half turns
    assert np.allclose(out[0, 0], [-2, 1, -3, -4, 5, 6])


def test_dyn_tanh_and_unit_and_gelu():
    assert np.allclose(mixers.dyn_tanh(np.array([0.0, 2.0]), 0.5, np.array([3.0, 2.0]), np.array([1.0, -1.0])), [1.0, 2 * np.tanh(1) - 1])
    assert np.allclose(mixers.unit(np.array([3.0, 4.0])), np.array([0.6, 0.8]), atol=1e-7)
    assert np.allclose(mixers.gelu_tanh(np.array([0.0, 10.0, -10.0])), [0, 10, 0])


@pytest.mark.parametrize("dims,base,scaling", [(8, 10000.0, None), (64, 500.0, mc.SCALING), (10, 1e6, dict(factor=2.0, low=0.5, high=6.0, original=4096))])
def test_rotary_frequencies_of_the_loader(capi, dims, base, scaling):
    out = np.empty(dims // 2)
    args = None if scaling is None else np.array([scaling[k] for k in ("factor", "low", "high", "original")])
    capi.check(capi.lib().mk_rotary_frequencies(dims, base, None if args is None else args.ctypes.data, out.ctypes.data))
    want = mixers.rope_frequencies(dims, base, scaling)
    assert np.allclose(out, want, rtol=1e-14)
    if scaling:     # all three regimes are there
        plain = mixers.rope_frequencies(dims, base)
        ratio = want / plain
        assert np.isclose(ratio.max(), 1) and np.isclose(ratio.min(), 1 / scaling["factor"])


# ------------------------------------------------------------------------------------------------ configuration, audit

LAYERS = [mc.wkv(2, 24), mc.parallel((4, 2, 16, 20, 8, True), (4, 2, 12, 10, 3), ff=40), mc.wkv(1, 40, ff=24)]


def broken(tmp_path, change_cfg=None, change_w=None):
    cfg = json.loads(json.dumps(mc.config(LAYERS, width=40)))
    w = mc.weights(cfg)
    if change_cfg:
        change_cfg(cfg)
    if change_w:
        change_w(w)
    return mc.write(tmp_path / "m", cfg, w)


def test_inspect_reads_the_description(eng, tmp_path):
    s = eng.Model.inspect_mixer(broken(tmp_path))
    assert (s["architecture"], s["vocab_size"], s["hidden_size"], s["n_layers"]) == ("Sizilorn", 131, 40, 3)
    assert (s["wkv_layers"], s["parallel_layers"], s["ffn_layers"], s["side_dim"]) == (2, 1, 2, 12)
    w = mc.weights(mc.config(LAYERS, width=40))
    assert s["tensors_in_file"] == s["tensors_read"] == len(w)
    assert s["parameters"] == sum(a.size for a in w.values())


@pytest.mark.parametrize("change,message", [
    (lambda w: w.pop("l0.mix.u"), "`l0.mix.u` is missing"),
    (lambda w: w.update({"l1.mix.right.v.conv": np.zeros((40, 4), np.float32)}), "`l1.mix.right.v.conv` has shape [40, 4], expected [40, 3]"),
    (lambda w: w.update({"head": np.zeros((131, 40), np.int32)}), "`head` is not a floating-point tensor"),
    (lambda w: w.update({"l2.norm2.alpha": np.zeros(1, np.float32)}), "`l2.norm2.alpha` has shape [1], expected []"),
    (lambda w: w.update({"l0.mix.w1": np.zeros(40, np.float32)}), "`l0.mix.w1` must be a matrix"),
])
def test_audit_names_the_tensor(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(broken(tmp_path, change_w=change))
    assert message in str(e.value)


@pytest.mark.parametrize("change,message", [
    (lambda c: c.update(architecture="Other"), "architecture `Other` is not supported"),
    (lambda c: c["layers"][0].update(type="conv"), "config.layers[0].type `conv` is not a known mixer"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "heads must be a multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "dims must be even"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "dims is out of range"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind `sparse` is not supported"),
    (lambda c: c["layers"][2]["mixer"].pop("heads"), "config.layers[2].mixer.heads is missing"),
    (lambda c: c.update(vocab=1.5), "config.vocab must be an integer"),
    (lambda c: c.update(layers=[]), "config lists no layers"),
])
def test_reader_names_the_setting(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(broken(tmp_path, change_cfg=change))
    assert message in str(e.value)


@pytest.mark.parametrize("raw,message", [
    (b"", "cannot be mapped"),
    (b"\xff" * 16, "header length is out of range"),
    (b"\x04\0\0\0\0\0\0\0{\"a\"", "malformed JSON"),
    (b"\x44\0\0\0\0\0\0\0" + b'{"embed":{"dtype":"BF16","shape":[131,40],"data_offsets":[0,10480]}} ', "lies outside the file"),
])
def test_container_refuses_broken_files(eng, capi, tmp_path, raw, message):
    d = broken(tmp_path)
    (d / "model.safetensors").write_bytes(raw)
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(d)
    assert message in str(e.value)


# ------------------------------------------------------------------------------------------------ state slots

def fake(eng, slots, **kw):
    return eng.Model.fake(vocab=32, kv_capacity_tokens=1024, state_slots=slots, **kw)


def test_slots_are_taken_at_the_first_forward_and_given_back(eng):
    m = fake(eng, 3)
    a, b = m.new_session(), m.new_session()
    assert m.state_slots() == (3, 0)
    m.forward_batch([(a, [1, 2, 3], 0), (b, [4], 0)])
    assert m.state_slots() == (3, 2)
    m.forward_batch([(a, [5], 3)])
    assert m.state_slots() == (3, 2)
    a.clear()
    assert m.state_slots() == (3, 1) and len(a) == 0
    m.forward_batch([(a, [1], 0)])
    b.close()
    assert m.state_slots() == (3, 1)


def test_a_reservation_without_a_slot_is_exhausted_and_changes_nothing(eng, capi):
    m = fake(eng, 2)
    s = [m.new_session() for _ in range(3)]
    m.forward_batch([(s[0], [1], 0)])
    before = m.pool_stats()
    with pytest.raises(capi.KvExhausted) as e:
        m.forward_batch([(s[1], [1], 0), (s[2], [1], 0)])
    assert "recurrent-state slot" in str(e.value)
    assert m.state_slots() == (2, 1) and m.pool_stats() == before
    m.forward_batch([(s[1], [1], 0)])
    assert m.state_slots() == (2, 2)


def test_a_failed_forward_keeps_no_slot(eng, capi):
    m = fake(eng, 2, fail_forward_at=0)
    s = m.new_session()
    with pytest.raises(capi.MkError):
        m.forward_batch([(s, [1, 2], 0)])
    assert m.state_slots() == (2, 0) and len(s) == 0
    m.forward_batch([(s, [1, 2], 0)])
    assert m.state_slots() == (2, 1)


def test_forks_of_recurrent_sessions(eng, capi):
    m = fake(eng, 2)
    s = m.new_session()
    m.forward_batch([(s, [1, 2, 3], 0)])
    with pytest.raises(capi.MkError) as e:
        s.fork_prefix(2)
    assert "current length only" in str(e.value)
    f = s.fork_prefix(3)
    assert m.state_slots() == (2, 2) and len(f) == 3
    with pytest.raises(capi.MkError):
        s.fork_prefix(3)


def test_recurrent_models_have_no_prefix_cache(eng, capi):
    with pytest.raises(capi.MkError) as e:
        fake(eng, 2, prefix_capacity_tokens=64)
    assert "recurrent layers" in str(e.value)


def test_engine_fits_its_active_set_to_the_slots(eng, capi):
    m = fake(eng, 2)
    with pytest.raises(capi.MkError) as e:
        eng.Engine(m, max_active_sequences=3)
    assert "recurrent-state slots" in str(e.value)
    e = eng.Engine(m, max_active_sequences=2, queue_capacity=8)
    ids = e.submit([eng.Request([1, 2, 3 + i], 4) for i in range(6)])
    e.run()
    assert all(e.result(i)["state"] == "done" and len(e.result(i)["tokens"]) == 4 for i in ids)
    assert m.state_slots() == (2, 0)


def test_logit_rows_are_checked(eng, capi):
    m = fake(eng, 2)
    s = m.new_session()
    for rows in ([[3]], [[-1]]):
        with pytest.raises(capi.MkError) as e:
            m.forward_batch([(s, [1, 2, 3], 0)], want_tokens=False, rows=rows)
        assert "outside its lane" in str(e.value)
    with pytest.raises(capi.MkError) as e:
        m.forward_batch([(s, [1, 2, 3], 0)], rows=[[0]])
    assert "last row" in str(e.value)
    with pytest.raises(capi.MkError) as e:
        m.forward_batch([(s, [1, 2, 3], 0)], want_tokens=False, rows=[[0], [0]])
    assert "another number of lanes" in str(e.value)
    assert len(s) == 0
