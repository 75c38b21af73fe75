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


def test_layer_norm_and_poly_norm_by_hand():
    assert np.allclose(mixers.layer_norm(np.array([1.0, 3.0]), np.array([2.0, 0.5]), 0.0), [-2.0, 0.5])
    assert np.allclose(mixers.layer_norm(np.array([1.0, 3.0]), np.ones(2), 3.0), [-0.5, 0.5])     # eps inside the root
    z = np.array([3.0, -1.0])
    # roots of the mean squares: sqrt(5), sqrt(41), sqrt(365)
    want = 2.0 * z / np.sqrt(5) + 3.0 * z ** 2 / np.sqrt(41) - z ** 3 / np.sqrt(365) + 0.25
    assert np.allclose(mixers.poly_norm(z, (2.0, 3.0, -1.0, 0.25), 0.0), want)


def test_sinusoid_by_hand():
    s = mixers.sinusoid([0, 1, 2000], 5)
    assert np.allclose(s[0], [0, 1, 0, 1, 0])
    f = 10000.0 ** -0.4
    assert np.allclose(s[1], [np.sin(1), np.cos(1), np.sin(f), np.cos(f), np.sin(f * f)])
    assert np.allclose(s[2, 2:4], [np.sin(2000 * f), np.cos(2000 * f)])


def test_min_gru_by_hand():
    z, u = np.array([[0.5], [0.25], [1.0]]), np.array([[1.5], [0.0], [-np.log(3.0)]])
    out, S = mixers.min_gru(z, u)
    # candidates 2, 1/2 and sigmoid(-log 3) = 1/4
    assert np.allclose(out[:, 0], [1.0, 0.875, 0.25]) and np.allclose(S, [0.25])
    rest, _ = mixers.min_gru(z[1:], u[1:], out[0])
    assert np.allclose(rest, out[1:])


def test_latent_attention_equals_attention_in_the_latent_space():
    """Queries taken to the latent space and values taken out of it: the same numbers (what the kernels rely on)."""
    rng = np.random.default_rng(0)
    cfg = mc.latent(3, 7, 5, 6, 4)["mixer"]
    W = {k[len("l0.mix."):]: v for k, v in mc.kunonex_weights(mc.kunonex([mc.latent(3, 7, 5, 6, 4)], width=10, vocab=11), 3).items() if k.startswith("l0.mix.")}
    h = rng.standard_normal((9, 10))
    want = mixers.latent_attention(h, W, cfg, 1e-5)
    q = ((mixers.rms(h @ W["dq"].T, 1e-5) * W["dq.norm"]) @ W["uq"].T).reshape(9, 3, 7)
    c = mixers.rms(h @ W["dkv"].T, 1e-5) * W["dkv.norm"]
    lat = np.einsum("thd,hdr->thr", q, W["uk"].reshape(3, 7, 4))
    o = mixers.causal_attention(lat, c[:, None, :], c[:, None, :], cfg["scale"])
    v = np.einsum("thr,her->the", o, W["uv"].reshape(3, 5, 4)) * mixers.sigmoid(h @ W["g"].T)[:, :, None]
    assert np.allclose(v.reshape(9, -1) @ W["o"].T, want)


def test_looped_layers_run_in_order():
    cfg = mc.kunonex([mc.mingru(3)] * 4, width=6, vocab=9, loop=(1, 3, 2))
    m = mixers.decoder(cfg, mc.weights(cfg))
    assert m.schedule() == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)]
    cfg["loop"] = None
    assert mixers.decoder(cfg, {}).schedule() == [(i, None) for i in range(4)]


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


BESIDE = [mc.mingru(24), mc.latent(4, 16, 20, 12, 10, ff=40), mc.mingru(40, ff=24)]


def broken_beside(tmp_path, change_cfg=None, change_w=None):
    cfg = json.loads(json.dumps(mc.kunonex(BESIDE, width=40, loop=(1, 3, 3))))
    w = mc.weights(cfg)
    if change_cfg:
        change_cfg(cfg)
    if change_w:
        change_w(w)
    return mc.write(tmp_path / "m", cfg, w)


@pytest.mark.parametrize("loop,runs", [((1, 3, 3), 7), ((0, 3, 2), 6), ((0, 1, 1), 3), (None, 3)])
def test_inspect_reads_layers_with_one_norm(eng, tmp_path, loop, runs):
    cfg = mc.kunonex(BESIDE, width=40, loop=loop)
    w = mc.weights(cfg)
    s = eng.Model.inspect_mixer(mc.write(tmp_path / "m", cfg, w))
    assert (s["architecture"], s["vocab_size"], s["hidden_size"], s["n_layers"], s["layer_runs"]) == ("Kunonex", 131, 40, 3, runs)
    assert (s["mingru_layers"], s["latent_layers"], s["wkv_layers"], s["parallel_layers"], s["ffn_layers"], s["side_dim"]) == (2, 1, 0, 0, 2, 0)
    assert s["tensors_in_file"] == s["tensors_read"] == len(w)
    assert s["parameters"] == sum(a.size for a in w.values())


@pytest.mark.parametrize("change,message", [
    (lambda w: w.pop("l1.mix.uk"), "`l1.mix.uk` is missing"),
    (lambda w: w.pop("embed.norm"), "`embed.norm` is missing"),
    (lambda w: w.pop("l2.shift"), "`l2.shift` is missing"),
    (lambda w: w.update({"loop.step": np.zeros((2, 40), np.float32)}), "`loop.step` has shape [2, 40], expected [3, 40]"),
    (lambda w: w.update({"l1.mlp.act": np.zeros(3, np.float32)}), "`l1.mlp.act` has shape [3], expected [4]"),
    (lambda w: w.update({"l0.mix.z.b": np.zeros(40, np.float32)}), "`l0.mix.z.b` has shape [40], expected [24]"),
])
def test_audit_names_the_tensor_of_layers_with_one_norm(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(broken_beside(tmp_path, change_w=change))
    assert message in str(e.value)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="wkv"), "config.layers[0].type `wkv` is not a known mixer"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "config.layers[1].mixer.q_rank is missing"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind `sparse` is not supported"),
    (lambda c: c["loop"].update(stop=4), "config.loop.stop is out of range"),
    (lambda c: c["loop"].update(stop=1), "config.loop.stop is out of range"),
    (lambda c: c["loop"].update(times=0), "config.loop.times is out of range"),
    (lambda c: c.pop("logit_scale"), "config.logit_scale is missing"),
])
def test_reader_names_the_setting_of_layers_with_one_norm(eng, capi, tmp_path, change, message):
    with pytest.raises(capi.MkError) as e:
        eng.Model.inspect_mixer(broken_beside(tmp_path, change_cfg=change))
    assert message in str(e.value)


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
