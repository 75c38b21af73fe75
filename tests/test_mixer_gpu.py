"""Mixer-built decoders on the GPU against the plain statement of their mechanisms (oracle/mixers.py), in 32-bit and in
bfloat16: every mechanism alone, whole prompts, portions, decoding, mixed batches, pages and slots used again, far keys and
page borders, sampling and generation through the engine, and the trace replay program."""
import importlib
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import mixer_cases as mc
from oracle import mixers

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def eng(mk):
    return importlib.import_module("macllm_infer_b200.engine")


@pytest.fixture(scope="module")
def capi(mk):
    return importlib.import_module("macllm_infer_b200._capi")


def checkpoint(tmp_path, cfg, seed=0, rank=5, change=None):
    w = mc.weights(cfg, seed, rank)
    if change:
        change(w)
        w = {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in w.items()}
    return mc.write(tmp_path / "m", cfg, w), mixers.decoder(cfg, w)


def tokens_of(n, vocab, seed=3):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


# ------------------------------------------------------------------------------------------------ mechanisms alone

def silence(*names):
    def change(w):
        for n in names:
            w[n] = np.zeros_like(w[n])
    return change


ALONE = {
    # name: (layer, width, side, what is silenced, rank)
    "wkv": (mc.wkv(3, 64), 96, 0, (), 16),
    "wkv narrow odd heads": (mc.wkv(2, 43), 70, 0, (), 3),
    "wkv one wide head": (mc.wkv(1, 136), 64, 0, (), 130),
    "wkv 128": (mc.wkv(2, 128), 128, 0, (), 8),
    "delta": (mc.parallel((2, 1, 16, 16, 8, False), (4, 2, 32, 64, 4)), 96, 0, ("l0.mix.left.out",), 5),
    "delta ungrouped, two taps": (mc.parallel((2, 1, 16, 16, 8, False), (3, 3, 21, 38, 2)), 72, 0, ("l0.mix.left.out",), 5),
    "delta without convolution history": (mc.parallel((2, 1, 16, 16, 8, False), (6, 2, 64, 128, 1)), 96, 0, ("l0.mix.left.out",), 5),
    "delta wide keys": (mc.parallel((2, 1, 16, 16, 8, False), (2, 1, 200, 72, 5)), 96, 0, ("l0.mix.left.out",), 5),
    "attention 64, scaled rotation": (mc.parallel((4, 2, 64, 64, 64, True), (1, 1, 8, 8, 2)), 96, 0, ("l0.mix.right.out",), 5),
    "attention narrow values": (mc.parallel((8, 2, 48, 24, 24, True), (1, 1, 8, 8, 2)), 96, 0, ("l0.mix.right.out",), 5),
    "attention wide values, three heads per key": (mc.parallel((6, 2, 20, 36, 20, False), (1, 1, 8, 8, 2)), 96, 0, ("l0.mix.right.out",), 5),
    "attention without rotation": (mc.parallel((4, 4, 128, 96, 0, False), (1, 1, 8, 8, 2)), 96, 0, ("l0.mix.right.out",), 5),
    "attention one key head": (mc.parallel((8, 1, 128, 128, 64, True), (1, 1, 8, 8, 2)), 96, 0, ("l0.mix.right.out",), 5),
    "both branches": (mc.parallel((4, 2, 40, 56, 16, True), (4, 2, 24, 40, 3)), 100, 0, (), 5),
    "feed-forward": (mc.wkv(1, 8, ff=200), 66, 0, ("l0.mix.o",), 5),
    "token input": (mc.wkv(1, 8), 100, 37, ("l0.mix.o",), 5),
}


ALONE_BESIDE = {
    # name: (layer, width, what is silenced)
    "minGRU": (mc.mingru(70), 96, ()),
    "minGRU wide state": (mc.mingru(300), 40, ()),
    "minGRU few odd channels": (mc.mingru(5), 67, ()),
    "minGRU beside a feed-forward": (mc.mingru(33, ff=90), 100, ()),
    "latent odd sizes": (mc.latent(3, 40, 24, 33, 50), 70, ()),
    "latent 128, wide values": (mc.latent(5, 20, 100, 12, 128), 96, ()),
    "latent 256, twenty heads": (mc.latent(20, 16, 30, 40, 200), 64, ()),
    "latent 512, one head": (mc.latent(1, 130, 70, 7, 300), 64, ()),
    "latent 512, thirty heads": (mc.latent(30, 8, 8, 24, 512), 64, ()),
    "latent, more than one head group": (mc.latent(37, 9, 12, 20, 30), 64, ()),
    "latent, heads too wide to expand": (mc.latent(2, 270, 20, 30, 64), 64, ()),
    "latent above the tensor-core kernel": (mc.latent(2, 24, 32, 30, 600), 64, ()),
    "latent beside a feed-forward": (mc.latent(4, 64, 64, 50, 70, ff=130), 96, ()),
    "feed-forward": (mc.mingru(8, ff=200), 66, ("l0.mix.o",)),
    "feed-forward, odd width": (mc.latent(1, 8, 8, 8, 8, ff=37), 67, ("l0.mix.o",)),
}


ALONE_OUTPUT = {
    # name: (layer, width, what is silenced)
    "mLSTM": (mc.mlstm(3, 64, 64), 96, ()),
    "mLSTM odd sizes": (mc.mlstm(2, 43, 37), 70, ()),
    "mLSTM 128, tight cap": (mc.mlstm(2, 128, 128, cap=0.8), 96, ()),
    "mLSTM narrow keys, wide values": (mc.mlstm(1, 12, 200), 64, ()),
    "mLSTM wide keys": (mc.mlstm(2, 200, 72, cap=12.0), 64, ()),
    "mLSTM two values": (mc.mlstm(5, 9, 2), 64, ()),
    "sink, chunk of a page": (mc.sink_attention(4, 2, 64, 64, 64, 16), 96, ()),
    "sink, odd chunk, partly turned": (mc.sink_attention(8, 2, 48, 24, 22, 33), 96, ()),
    "sink, three heads per key": (mc.sink_attention(6, 2, 20, 36, 20, 10), 70, ()),
    "sink, chunk of one": (mc.sink_attention(2, 2, 128, 96, 64, 1), 64, ()),
    "sink, one chunk for all": (mc.sink_attention(8, 1, 32, 128, 30, 4096), 64, ()),
    "capped, chunk of a tile": (mc.capped_attention(4, 2, 64, 64, 64, 32), 96, ()),
    "capped, odd chunk, partly turned": (mc.capped_attention(8, 4, 40, 24, 26, 27, softcap=0.7), 96, ()),
    "capped, odd width, five heads": (mc.capped_attention(5, 5, 21, 33, 12, 50, softcap=30.0), 67, ()),
    "capped, 256 wide": (mc.capped_attention(2, 1, 200, 130, 128, 7, yarn=dict(factor=16.0, original=512, fast=32.0, slow=2.0)), 64, ()),
    "experts, one of five": (mc.mlstm(1, 8, 8, mlp=mc.experts(5, 1, 37, 0.5)), 66, ("l0.norm1",)),
    "experts, seven of forty and a shared one": (mc.mlstm(1, 8, 8, mlp=mc.experts(40, 7, 24, 2.0, (90, 0.3))), 96, ("l0.norm1",)),
    "experts, all of three": (mc.mlstm(1, 8, 8, mlp=mc.experts(3, 3, 130, 0.7, (20, 3.0))), 130, ("l0.norm1",)),
    "experts behind a mixer": (mc.sink_attention(2, 1, 16, 16, 8, 12, mlp=mc.experts(6, 2, 64, 1.0, (64, 1.0))), 64, ()),
}


ALONE_CONV = {
    # name: (layer, width, taps, what is silenced, rank)
    "shared keys and values": (mc.scaled_parallel((4, 2, 64, 32), (1, 8), 20), 96, 4, ("l0.mix.right.o",), 5),
    "shared keys and values, three heads per key": (mc.scaled_parallel((6, 2, 20, 8), (1, 8), 9), 70, 3, ("l0.mix.right.o",), 5),
    "shared keys and values, window of one": (mc.scaled_parallel((2, 2, 32, 32), (1, 8), 1), 64, 2, ("l0.mix.right.o",), 5),
    "shared keys and values, 128, one key head": (mc.scaled_parallel((8, 1, 128, 64), (1, 8), 33), 96, 4, ("l0.mix.right.o",), 5),
    "shared keys and values, odd head": (mc.scaled_parallel((5, 5, 21, 6), (1, 8), 300), 67, 5, ("l0.mix.right.o",), 5),
    "shared keys and values, no turning": (mc.scaled_parallel((4, 4, 40, 0), (1, 8), 16), 64, 1, ("l0.mix.right.o",), 5),
    "channel delta": (mc.scaled_parallel((2, 1, 16, 8), (3, 64), 9), 96, 4, ("l0.mix.left.o",), 16),
    "channel delta, odd heads": (mc.scaled_parallel((2, 1, 16, 8), (5, 43), 9), 70, 3, ("l0.mix.left.o",), 3),
    "channel delta, one head": (mc.scaled_parallel((2, 1, 16, 8), (1, 24), 9), 64, 2, ("l0.mix.left.o",), 7),
    "channel delta 128": (mc.scaled_parallel((2, 1, 16, 8), (2, 128), 9), 128, 4, ("l0.mix.left.o",), 64),
    "channel delta, wide head, wide rank": (mc.scaled_parallel((2, 1, 16, 8), (2, 136), 9), 96, 1, ("l0.mix.left.o",), 130),
    "channel delta 256": (mc.scaled_parallel((2, 1, 16, 8), (1, 256), 9), 64, 4, ("l0.mix.left.o",), 4),
    "channel delta, many small heads": (mc.scaled_parallel((2, 1, 16, 8), (19, 12), 9), 64, 4, ("l0.mix.left.o",), 8),
    "both scaled branches": (mc.scaled_parallel((4, 2, 40, 16), (4, 24), 20, scales=(-0.7, 1.6)), 100, 4, (), 5),
    "rotated latents": (mc.rotated_latent(4, 32, 48, 40, 56, 16, 24), 96, 4, (), 5),
    "rotated latents, odd sizes": (mc.rotated_latent(3, 37, 24, 33, 45, 10, 17), 70, 3, (), 5),
    "rotated latents, turned part wider": (mc.rotated_latent(5, 12, 100, 12, 64, 60, 300), 96, 2, (), 5),
    "rotated latents behind 128": (mc.rotated_latent(2, 40, 20, 30, 128, 32, 40), 64, 4, (), 5),
    "rotated latents, whole extra chunk": (mc.rotated_latent(2, 64, 64, 30, 128, 96, 40), 64, 4, (), 5),
    "rotated latents behind 256, twenty heads": (mc.rotated_latent(20, 16, 30, 40, 250, 24, 50), 64, 4, (), 5),
    "rotated latents behind 384": (mc.rotated_latent(2, 16, 16, 20, 384, 64, 19), 64, 4, (), 5),
    "rotated latents behind 512, 192 wide": (mc.rotated_latent(3, 128, 128, 64, 512, 64, 48), 96, 4, (), 5),
    "rotated latents behind 512, more than one head group": (mc.rotated_latent(37, 9, 12, 20, 512, 8, 60), 64, 4, (), 5),
    "rotated latents above the tensor-core kernel": (mc.rotated_latent(2, 24, 32, 30, 600, 16, 30), 64, 4, (), 5),
    "rotated latents, heads too wide to expand": (mc.rotated_latent(2, 250, 20, 30, 64, 16, 30), 64, 4, (), 5),
    "rotated latents, window of one": (mc.rotated_latent(2, 16, 16, 20, 40, 8, 1), 64, 4, (), 5),
    "rotated latents, plain rotation": (mc.rotated_latent(4, 24, 24, 32, 40, 24, 40, scaling=None), 64, 4, (), 5),
    "gelu feed-forward": (mc.scaled_parallel((2, 1, 16, 8), (1, 8), 9, ff=200), 66, 4, ("l0.mix.left.o", "l0.mix.right.o"), 5),
}


def check_alone(folder, oracle, compute):
    """The residual stream after a layer with one mechanism at work, for a whole prompt, portions and single tokens."""
    toks = tokens_of(75, oracle.cfg["vocab"])
    base = oracle.embedding_output(toks)
    want = oracle.residuals(toks)[0]
    delta = want - base          # what the layer adds: the part under test
    model = mc.load(folder, compute)
    model.capture_residuals(True)
    for portions in ([75], mc.cut(75, [2, 17, 1, 5, 33]), mc.cut(75, [34, 2, 39]), mc.cut(75, [1])):
        s, at, got = model.new_session(), 0, []
        for k in portions:
            model.forward_batch([(s, toks[at:at + k], at)], want_logits=False, want_tokens=False, rows=[[]])
            got.append(model.residuals(k)[0])
            at += k
        s.close()
        got = np.concatenate(got) - base
        e = np.sqrt(np.mean((got - delta) ** 2, axis=1) / np.mean(delta ** 2))
        assert e.max() <= mc.LIMIT[compute], f"{portions[:5]}: token {int(e.argmax())} off by {e.max():.2e}"
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism_alone(mk, tmp_path, name, compute):
    layer, width, side, silenced, rank = ALONE[name]
    cfg = mc.config([layer], width=width, side=side)
    check_alone(*checkpoint(tmp_path, cfg, seed=7, rank=rank, change=silence(*silenced)), compute)


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", ALONE_BESIDE)
def test_mechanism_alone_in_layers_with_one_norm(mk, tmp_path, name, compute):
    layer, width, silenced = ALONE_BESIDE[name]
    check_alone(*checkpoint(tmp_path, mc.kunonex([layer], width=width), seed=7, change=silence(*silenced)), compute)


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", ALONE_OUTPUT)
def test_mechanism_alone_in_layers_with_norms_on_outputs(mk, tmp_path, name, compute):
    layer, width, silenced = ALONE_OUTPUT[name]
    check_alone(*checkpoint(tmp_path, mc.tevanex([layer], width=width), seed=7, change=silence(*silenced)), compute)


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", ALONE_CONV)
def test_mechanism_alone_in_layers_behind_a_convolution(mk, tmp_path, name, compute):
    layer, width, taps, silenced, rank = ALONE_CONV[name]
    check_alone(*checkpoint(tmp_path, mc.mamivik([layer], width=width, taps=taps), seed=7, rank=rank, change=silence(*silenced)), compute)


@pytest.mark.parametrize("compute", DTYPES)
def test_token_shift_reaches_the_mixer_only(mk, tmp_path, compute):
    """A shift of one: the mixer sees nothing but the token before (zeros at first), the feed-forward nothing but the token."""
    cfg = mc.kunonex([mc.mingru(20, ff=30)], width=50, vocab=40)

    def change(w):
        w["l0.shift"][:] = 1.0

    folder, oracle = checkpoint(tmp_path, cfg, seed=9, change=change)
    check_alone(folder, oracle, compute)


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("width", [64, 67])
def test_sinusoidal_positions_far_out(mk, tmp_path, width, compute):
    """The embedding output at positions up to the thousands: the layer adds nothing, so the stream after it is that output."""
    cfg = mc.kunonex([mc.mingru(4)], width=width, vocab=20)
    folder, oracle = checkpoint(tmp_path, cfg, seed=2, change=silence("l0.mix.o"))
    toks = tokens_of(3000, 20)
    model = mc.load(folder, compute, capacity=3008)
    model.capture_residuals(True)
    s = model.new_session()
    model.forward_batch([(s, toks, 0)], want_logits=False, want_tokens=False, rows=[[]])
    assert np.abs(model.residuals(3000)[0] - oracle.embedding_output(toks)).max() < 1e-5
    model.close()


# ------------------------------------------------------------------------------------------------ whole models

_EXPERTS = [mc.mlstm(4, 32, 48, mlp=mc.experts(6, 2, 40, 0.8, (60, 1.2))), mc.sink_attention(4, 2, 64, 40, 64, 24, mlp=mc.experts(12, 1, 64)),
            mc.capped_attention(8, 2, 64, 64, 32, 48, mlp=mc.experts(4, 4, 33, 1.5, (33, 1.5))), mc.mlstm(2, 64, 130)]

MODELS = {
    "first": (mc.config([mc.wkv(3, 40), mc.parallel((4, 2, 64, 64, 32, True), (4, 2, 32, 48, 4), ff=150), mc.wkv(2, 64, ff=90)], width=104), 9),
    "second": (mc.config([mc.parallel((6, 2, 36, 20, 12, False), (3, 3, 48, 40, 2)), mc.wkv(5, 16), mc.parallel((8, 1, 32, 32, 32, True), (2, 2, 64, 64, 3), ff=64)],
                         width=67, vocab=201, side=5, eps=1e-5), 4),
    "looped": (mc.kunonex([mc.mingru(40, ff=50), mc.latent(4, 32, 48, 30, 60, ff=150), mc.mingru(72), mc.latent(6, 20, 36, 24, 90)], width=104,
                          loop=(1, 3, 3)), 0),
    "loop over all layers": (mc.kunonex([mc.latent(2, 70, 20, 48, 130), mc.mingru(33, ff=41)], width=67, vocab=201, loop=(0, 2, 2), eps=1e-5,
                                        logit_scale=1.3), 0),
    "no loop": (mc.kunonex([mc.mingru(24, ff=60), mc.latent(20, 16, 16, 64, 40, ff=60)], width=64, logit_scale=1.0), 0),
    "a loop of one pass": (mc.kunonex([mc.latent(3, 24, 24, 24, 24), mc.mingru(50, ff=32)], width=48, loop=(1, 2, 1)), 0),
    "experts": (mc.tevanex(_EXPERTS + [mc.again(_EXPERTS, 1), mc.again(_EXPERTS, 0)], width=104), 0),
    "experts, odd sizes": (mc.tevanex([mc.capped_attention(6, 2, 44, 36, 28, 50, mlp=mc.experts(5, 3, 37)), mc.mlstm(3, 40, 21, mlp=mc.experts(9, 2, 50, 0.6, (70, 0.4))),
                                       mc.sink_attention(8, 1, 32, 80, 32, 20)], width=67, vocab=201, eps=1e-5, embed=2.3, mult=0.35, logit_scale=1.4, softcap=3.0), 0),
    "convolved": (mc.mamivik([mc.scaled_parallel((4, 2, 64, 16), (3, 48), 37, ff=150), mc.rotated_latent(4, 32, 40, 30, 56, 16, 50, ff=90),
                              mc.scaled_parallel((8, 2, 32, 32), (2, 64), 21, scales=(1.3, 0.4))], width=104, taps=4), 9),
    "convolved, odd sizes": (mc.mamivik([mc.rotated_latent(6, 20, 36, 24, 130, 14, 23), mc.scaled_parallel((6, 2, 36, 12), (3, 40), 60, ff=37),
                                         mc.rotated_latent(2, 70, 20, 48, 90, 40, 100, ff=64, scaling=None)], width=67, vocab=201, taps=6, eps=1e-5), 4),
    "time mixing only": (mc.config([mc.wkv(2, 32), mc.wkv(1, 72)], width=64, side=64), 20),
}


@pytest.fixture(scope="module")
def built(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg, rank = MODELS[name]
            w = mc.weights(cfg, seed=11, rank=rank)
            made[name] = (mc.write(tmp_path_factory.mktemp("mixer") / "m", cfg, w), mixers.decoder(cfg, w), cfg)
        return made[name]
    return get


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", MODELS)
def test_prompt_portions_and_decoding_agree(mk, built, name, compute):
    folder, oracle, cfg = built(name)
    toks = tokens_of(150, cfg["vocab"])
    want = oracle.logits(toks)
    model = mc.load(folder, compute)
    for portions in ([150], [149, 1], mc.cut(150, [2]), mc.cut(150, [3, 64, 5, 16, 31]), mc.cut(150, [1]), [100] + [1] * 50):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:6]}")
    assert model.state_slots()[1] == 0 and model.pool_stats()["live_blocks"] == 0
    model.close()


BOTH = ["first", "looped", "experts", "convolved"]   # a model of each layer form


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", BOTH)
def test_unequal_batches_against_each_alone(mk, built, name, compute):
    """Four sequences of different lengths, portions of some beside single tokens of others, one of them paused for a while."""
    folder, oracle, cfg = built(name)
    seqs = [tokens_of(n, cfg["vocab"], seed=20 + n) for n in (130, 40, 3, 77)]
    want = [oracle.logits(t) for t in seqs]
    model = mc.load(folder, compute)
    alone = [mc.run_portions(model, t, [len(t)]) for t in seqs]
    sessions = [model.new_session() for _ in seqs]
    got = [[] for _ in seqs]
    plans = [mc.cut(130, [33, 2, 1, 1, 50]), [1] * 40, [3], mc.cut(77, [16, 1, 2])]
    tick = 0
    while any(plans):
        lanes, who = [], []
        for i, plan in enumerate(plans):
            if plan and not (i == 3 and tick in (1, 2)):
                k, at = plan.pop(0), len(sessions[i])
                lanes.append((sessions[i], seqs[i][at:at + k], at))
                who.append(i)
        if lanes:
            rows, _ = model.forward_batch(lanes, want_tokens=False, rows=[range(len(l[1])) for l in lanes])
            at = 0
            for i, l in zip(who, lanes):
                got[i].append(rows[at:at + len(l[1])])
                at += len(l[1])
        tick += 1
    for i in range(len(seqs)):
        g = np.concatenate(got[i])
        mc.assert_rows(g, want[i], compute, f"sequence {i}")
        assert mc.row_errors(g, alone[i]).max() <= mc.LIMIT[compute]
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", BOTH)
def test_pages_and_slots_are_used_again(mk, built, name, compute):
    """A pool and a slot array that only just hold the live sequences: every later one runs in what an earlier one left."""
    folder, oracle, cfg = built(name)
    model = mc.load(folder, compute, capacity=128, lanes=2, slots=2)
    held = model.new_session()
    a = tokens_of(40, cfg["vocab"], seed=1)
    wa, got_a = oracle.logits(a), []
    for round_ in range(8):
        b = tokens_of(70 - round_, cfg["vocab"], seed=50 + round_)
        s = model.new_session()
        rows, _ = model.forward_batch([(held, a[5 * round_:5 * round_ + 5], 5 * round_), (s, b[:61], 0)], want_tokens=False, rows=[range(5), [60]])
        got_a.append(rows[:5])
        rows2, _ = model.forward_batch([(s, b[61:], 61)], want_tokens=False, rows=[range(len(b) - 61)])
        mc.assert_rows(np.concatenate([rows[5:], rows2]), oracle.logits(b)[60:], compute, f"round {round_}")
        s.close()
    mc.assert_rows(np.concatenate(got_a), wa, compute, "the sequence that stayed")
    assert model.state_slots() == (2, 1)
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("left", [(4, 2, 64, 64, 32, True), (6, 2, 24, 40, 8, False)])
def test_one_far_key_stands_out(mk, tmp_path, left, compute):
    """A query projects the other half of the embedding's channels with the key's matrix, and the asking token's embedding is the
    sought one's with its halves exchanged: in the dimensions that do not turn the query meets exactly that key, and the
    softmax is nearly all on it.  The sought token sits at the first place, at both sides of page borders and next to the
    query; the asking one follows at once, at a page border, or hundreds of tokens later, in a prompt and decoded."""
    layer = mc.parallel(left, (1, 1, 8, 8, 2))
    cfg = mc.config([layer], width=80, vocab=60, side=0)
    heads, group, dim, turned = left[0], left[0] // left[1], left[2], left[4]

    def change(w):
        w["l0.mix.right.out"] *= 0
        q = w["l0.mix.left.q"].reshape(heads, dim, 80)
        k = w["l0.mix.left.k"].reshape(left[1], dim, 80)
        q[:] = np.repeat(np.roll(k, 40, axis=2), group, axis=0)
        w["embed"][1] = np.roll(w["embed"][0], 40)
        w["l0.norm1"][:] = 1.0
        w["l0.norm1.b"][:] = 0.0
        for n in ("q", "k"):
            w[f"l0.mix.left.{n}.norm"][:turned] = 0.05
            w[f"l0.mix.left.{n}.norm"][turned:] = 4.0

    folder, oracle = checkpoint(tmp_path, cfg, seed=5, change=change)
    model = mc.load(folder, compute)
    sought, asking, filler = 0, 1, np.random.default_rng(2).integers(2, 60, 500)
    for key, query in ((0, 499), (15, 32), (16, 31), (31, 33), (16, 400), (63, 64), (128, 447), (0, 15), (0, 16)):
        toks = filler[:query + 1].copy()
        toks[key], toks[query] = sought, asking
        want = oracle.logits(toks.tolist())[query]
        without = toks.copy()
        without[key] = 2
        assert mc.row_errors(oracle.logits(without.tolist())[query], want) > 0.2      # a lost key shows
        for portions in ([query + 1], [query, 1], mc.cut(query + 1, [48, 2])):
            got = mc.run_portions(model, toks.tolist(), portions)[query]
            assert mc.row_errors(got, want) <= mc.LIMIT[compute], (key, query, portions[:3])
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("latent", [(4, 32, 48, 40, 40), (20, 24, 24, 100, 100), (2, 64, 64, 300, 300)])
def test_one_far_key_stands_out_of_the_latents(mk, tmp_path, latent, compute):
    """As above for latent attention: the query latent is the key latent of the embedding with its halves exchanged, and the
    embeddings are large against the positions.  Histories of more than a few hundred keys are cut into shares when decoded."""
    heads, dim, vdim, q_rank, kv_rank = latent
    cfg = mc.kunonex([mc.latent(*latent)], width=80, vocab=60)

    def change(w):
        w["l0.mix.dq"][:] = np.roll(w["l0.mix.dkv"], 40, axis=1)
        w["l0.mix.dq.norm"][:] = w["l0.mix.dkv.norm"]
        w["l0.mix.uq"][:] = 2.0 * w["l0.mix.uk"]
        w["embed"] *= 8.0
        w["embed"][1] = np.roll(w["embed"][0], 40)
        w["l0.norm1"][:] = 1.0
        w["embed.norm"][:] = 1.0
        w["l0.shift"][:] = 0.0

    folder, oracle = checkpoint(tmp_path, cfg, seed=5, change=change)
    model = mc.load(folder, compute, capacity=1200)
    sought, asking, filler = 0, 1, np.random.default_rng(2).integers(2, 60, 1100)
    for key, query in ((0, 1099), (15, 32), (16, 31), (31, 33), (32, 63), (16, 400), (255, 700), (256, 700), (63, 64), (128, 447), (0, 15), (0, 1), (7, 7)):
        toks = filler[:query + 1].copy()
        toks[key], toks[query] = sought, asking
        want = oracle.logits(toks.tolist())[query]
        if key < query:
            without = toks.copy()
            without[key] = 2
            assert mc.row_errors(oracle.logits(without.tolist())[query], want) > 0.2      # a lost key shows
        for portions in ([query + 1], [query, 1] if query else [1], mc.cut(query + 1, [48, 2])):
            got = mc.run_portions(model, toks.tolist(), portions)[query]
            assert mc.row_errors(got, want) <= mc.LIMIT[compute], (key, query, portions[:3])
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
def test_one_far_write_stays_in_the_mingru_state(mk, tmp_path, compute):
    """Gates that hardly open but for one token: what it wrote is read hundreds of tokens later."""
    cfg = mc.kunonex([mc.mingru(48)], width=64, vocab=50)

    def change(w):
        w["embed"] *= 8.0
        w["embed"][:, 0] = -30.0
        w["embed"][0, 0] = 30.0
        w["embed.norm"][:] = 1.0
        w["l0.norm1"][:] = 1.0
        w["l0.shift"][:] = 0.0
        w["l0.mix.z"] *= 0.05
        w["l0.mix.z"][:, 0] = 4.0
        w["l0.mix.z.b"][:] = -1.0

    folder, oracle = checkpoint(tmp_path, cfg, seed=6, change=change)
    toks = [0] + (1 + np.random.default_rng(4).integers(0, 49, 399)).tolist()
    want = oracle.logits(toks)
    lost = oracle.logits([1] + toks[1:])
    assert mc.row_errors(lost[-40:], want[-40:]).min() > 10 * mc.LIMIT["float32"]
    model = mc.load(folder, compute)
    for portions in ([400], mc.cut(400, [37, 1, 2, 100]), mc.cut(400, [128, 129, 127, 8]), [64] + [1] * 336):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("lanes", [2, 9])
def test_long_histories_decoded_in_shares(mk, built, lanes):
    """A few sequences with a thousand tokens of history each, unequal, decoded together: their keys are shared out over CTAs."""
    folder, oracle, cfg = built("looped")
    seqs = [tokens_of(1000 - 111 * i, cfg["vocab"], seed=90 + i) for i in range(lanes)]
    model = mc.load(folder, "bfloat16", capacity=lanes * 1008, lanes=lanes, slots=lanes)
    sessions = [model.new_session() for _ in seqs]
    for s, q in zip(sessions, seqs):
        model.forward_batch([(s, q[:-4], 0)], want_logits=False, want_tokens=False, rows=[[]])
    got = []
    for t in range(4, 0, -1):
        rows, _ = model.forward_batch([(s, [q[-t]], len(q) - t) for s, q in zip(sessions, seqs)], want_tokens=False)
        got.append(rows)
    for i, q in enumerate(seqs):
        mc.assert_rows(np.stack([g[i] for g in got]), oracle.logits(q)[-4:], "bfloat16", f"sequence {i}")
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
def test_one_far_write_stays_in_the_recurrent_state(mk, tmp_path, compute):
    """Hardly any decay, no overwriting: what the first token wrote is read hundreds of tokens later by both recurrences."""
    cfg = mc.config([mc.wkv(2, 32), mc.parallel((2, 1, 16, 16, 8, False), (2, 1, 32, 32, 3))], width=64, vocab=50, side=0)

    def change(w):
        w["l0.mix.w0"][:] = -9.0
        w["l1.mix.right.dt_bias"][:] = -9.0
        w["l1.mix.right.b"] *= 0.0
        w["l1.mix.left.out"] *= 0
        w["embed"][0] *= 6.0

    folder, oracle = checkpoint(tmp_path, cfg, seed=6, change=change)
    toks = [0] + (1 + np.random.default_rng(4).integers(0, 49, 399)).tolist()
    want = oracle.logits(toks)
    lost = oracle.logits([1] + toks[1:])
    assert mc.row_errors(lost[-40:], want[-40:]).min() > 10 * mc.LIMIT["float32"]
    model = mc.load(folder, compute)
    for portions in ([400], mc.cut(400, [37, 1, 2, 100]), [64] + [1] * 336):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("name", BOTH)
def test_long_decoding_in_a_full_batch(mk, built, name):
    """Four sequences decoded one token a tick for 300 ticks (the one-token kernels all the way), in bfloat16."""
    folder, oracle, cfg = built(name)
    seqs = [tokens_of(300, cfg["vocab"], seed=70 + i) for i in range(4)]
    model = mc.load(folder, "bfloat16", capacity=4 * 304)
    sessions = [model.new_session() for _ in seqs]
    got = [[] for _ in seqs]
    for t in range(300):
        rows, _ = model.forward_batch([(s, [q[t]], t) for s, q in zip(sessions, seqs)], want_tokens=False)
        for i in range(4):
            got[i].append(rows[i])
    for q, g in zip(seqs, got):
        mc.assert_rows(np.stack(g), oracle.logits(q), "bfloat16")
    model.close()


# ------------------------------------------------------------------------------------------------ sessions, sampling, engine

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", BOTH)
def test_a_fork_carries_pages_and_state(mk, built, name, compute):
    folder, oracle, cfg = built(name)
    toks = tokens_of(60, cfg["vocab"], seed=8)
    model = mc.load(folder, compute)
    a = model.new_session()
    model.forward_batch([(a, toks[:37], 0)], want_tokens=False)
    b = a.fork_prefix(37)
    ta, tb = toks[37:], toks[37:][::-1]
    rows, _ = model.forward_batch([(a, ta, 37), (b, tb, 37)], want_tokens=False, rows=[range(23)] * 2)
    mc.assert_rows(rows[:23], oracle.logits(toks[:37] + ta)[37:], compute)
    mc.assert_rows(rows[23:], oracle.logits(toks[:37] + tb)[37:], compute)
    model.close()


@pytest.mark.parametrize("name", ["second", "looped", "experts", "convolved"])
def test_a_refused_forward_leaves_the_state_alone(mk, built, capi, name):
    folder, oracle, cfg = built(name)
    toks = tokens_of(50, cfg["vocab"], seed=9)
    model = mc.load(folder, "float32", capacity=128, lanes=1)
    s, other = model.new_session(), model.new_session()
    model.forward_batch([(s, toks[:20], 0)], want_tokens=False)
    for bad in ([(s, [cfg["vocab"]], 20)], [(s, toks[:1], 20), (other, toks[:1], 0)], [(s, toks[:1], 19)]):
        with pytest.raises(capi.MkError):
            model.forward_batch(bad, want_tokens=False)
    assert model.state_slots()[1] == 1
    rows, _ = model.forward_batch([(s, toks[20:], 20)], want_tokens=False, rows=[range(30)])
    mc.assert_rows(rows, oracle.logits(toks)[20:], "float32")
    model.close()


@pytest.mark.parametrize("name", ["first", "second", "looped", "loop over all layers", "no loop", "experts", "experts, odd sizes", "convolved", "convolved, odd sizes"])
def test_greedy_generation_through_the_engine(mk, eng, built, name):
    """Requests of unequal length through the scheduler, more of them than slots; 32-bit, so that the plain statement's own
    argmax must come out wherever its first two logits are not a near-tie."""
    folder, oracle, cfg = built(name)
    model = mc.load(folder, "float32", capacity=512, lanes=3, slots=3)
    e = eng.Engine(model, max_active_sequences=3, scheduler_token_budget=48, prefill_token_quantum=20, queue_capacity=8)
    prompts = [tokens_of(n, cfg["vocab"], seed=n) for n in (1, 33, 90, 7, 52)]
    ids = e.submit([eng.Request(p, 12) for p in prompts])
    e.run()
    for p, i in zip(prompts, ids):
        r = e.result(i)
        assert r["state"] == "done" and len(r["tokens"]) == 12
        logits = oracle.logits(p + [int(t) for t in r["tokens"][:-1]])[len(p) - 1:]
        for row, t in zip(logits, r["tokens"]):
            assert row.max() - row[t] <= 1e-4 * np.abs(row).max()
    assert model.state_slots() == (3, 0)
    e.close()
    model.close()


@pytest.mark.parametrize("name", BOTH)
def test_device_sampling_and_recorded_logits(mk, eng, built, name):
    """Temperature / top-k / top-p on the device gives the same tokens as the host sampler on read-back logits."""
    folder, oracle, cfg = built(name)
    outs = []
    for host in (False, True):
        model = mc.load(folder, "bfloat16")
        e = eng.Engine(model, max_active_sequences=4, scheduler_token_budget=64, prefill_token_quantum=32, host_sampling=host)
        ids = e.submit([eng.Request(tokens_of(20 + i, cfg["vocab"], seed=i), 10, temperature=0.8, top_k=20, top_p=0.9, seed=100 + i) for i in range(3)])
        e.run()
        outs.append([e.result(i)["tokens"].tolist() for i in ids])
        e.close()
        model.close()
    assert outs[0] == outs[1]


@pytest.mark.parametrize("name", ["second", "looped", "loop over all layers", "experts", "experts, odd sizes", "convolved", "convolved, odd sizes"])
def test_residuals_after_every_layer(mk, built, name):
    """A looped layer counts once per pass."""
    folder, oracle, cfg = built(name)
    toks = tokens_of(30, cfg["vocab"], seed=12)
    model = mc.load(folder, "float32")
    model.capture_residuals(True)
    s = model.new_session()
    model.forward_batch([(s, toks, 0)], want_tokens=False)
    got, want = model.residuals(30), oracle.residuals(toks)
    assert got.shape == want.shape
    for l in range(len(want)):
        assert np.abs(got[l] - want[l]).max() <= 2e-5 * np.abs(want[l]).max()
    model.close()


def test_logit_rows_of_a_gguf_model(mk, eng, tmp_path):
    """Chosen rows work the same for the GGUF families: the rows of one forward equal the last rows of shorter ones."""
    seed = importlib.import_module("macllm_infer_b200.seed_gguf")
    spec = seed.scaled("tinyllama-1.1b", layers=1, vocab=512)
    seed.write_seed_gguf(tmp_path / "m.gguf", spec, seed=0)
    model = eng.Model.load(tmp_path / "m.gguf", kv_dtype="f32", matmul_path=1, max_batch_tokens=64, max_batch_lanes=4, kv_capacity_tokens=512)
    toks = tokens_of(12, 512)
    s = model.new_session()
    rows, _ = model.forward_batch([(s, toks, 0)], want_tokens=False, rows=[[2, 11, 7]])
    for row, at in zip(rows, (2, 11, 7)):
        one = model.new_session()
        last, _ = model.forward_batch([(one, toks[:at + 1], 0)], want_tokens=False)
        assert np.abs(last[0] - row).max() <= 1e-4
        one.close()
    model.close()


# ------------------------------------------------------------------------------------------------ the replay program

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", BOTH)
def test_trace_replay(mk, built, tmp_path, name, compute):
    folder, oracle, cfg = built(name)
    a, b, c = (tokens_of(n, cfg["vocab"], seed=n) for n in (45, 20, 60))
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": []}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b, "want": [0, 19]}, {"id": "a", "tokens": a[17:18], "want": [0]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "c", "tokens": c, "want": [59, 3]}], "end": ["c"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[18:], "want": [26]}, {"id": "b2", "tokens": b[:2], "want": [1]}], "end": ["a", "b2"]},
    ]
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", compute, "--out", str(tmp_path),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "0.f32").exists()
    la, lb, lc = oracle.logits(a), oracle.logits(b), oracle.logits(c)
    for step, want in ((1, [lb[0], lb[19], la[17]]), (2, [lc[59], lc[3]]), (3, [la[44], lb[1]])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(want), cfg["vocab"])
        mc.assert_rows(got, np.stack(want), compute, f"step {step}")
