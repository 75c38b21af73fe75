"""Mamivik decoders on the GPU: what random weights would hide - window edges, sinks, biases, branch constants, far writes of the delta
rule, its removals, the convolution's history, stretched rotations far out - each made to stand out, against the plain statement
(oracle/mixers.py).  tests/test_mixer_gpu.py runs each mechanism alone and whole models of the design beside the others."""
import copy
import importlib

import numpy as np
import pytest

import mixer_cases as mc
from oracle import mixers

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def checkpoint(tmp_path, cfg, seed=0, rank=5, change=None):
    w = mc.weights(cfg, seed, rank)
    if change:
        change(w)
        w = {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in w.items()}
    return mc.write(tmp_path / "m", cfg, w), mixers.decoder(cfg, w), w


def tokens_of(n, vocab, seed=3):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


# ------------------------------------------------------------------------------------------------ window edges

EDGES = {
    "shared keys, window of three pages": mc.scaled_parallel((4, 2, 64, 16), (1, 8), 48, scales=(1.0, 0.0)),
    "shared keys, odd window, three heads per key": mc.scaled_parallel((6, 2, 40, 8), (1, 8), 37, scales=(1.0, 0.0)),
    "shared keys, long window": mc.scaled_parallel((8, 1, 32, 8), (1, 8), 448, scales=(1.0, 0.0)),
    "latents, window of four pages": mc.rotated_latent(4, 48, 32, 72, 72, 8, 64),
    "latents, odd window": mc.rotated_latent(20, 40, 24, 100, 130, 8, 50),
    "latents, long window": mc.rotated_latent(3, 64, 64, 300, 512, 64, 449),
}


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", EDGES)
def test_one_key_stands_out_inside_the_window_and_is_gone_outside(mk, tmp_path, name, compute):
    """A query projects the other half of the embedding's channels with the key's matrix, and the asking token's embedding is the
    sought one's with its halves exchanged: in the dimensions that do not turn the query meets exactly that key.  The sought token
    sits at the last place the window shows, one before it, at page borders and right in front of the query."""
    layer = EDGES[name]
    m = layer["mixer"]
    cfg = mc.mamivik([layer], width=80, vocab=60, taps=2)
    latent = layer["type"] == "latent_attention"
    window = (m if latent else m["left"])["mask"]["size"]

    def change(w):
        w["embed"][1] = np.roll(w["embed"][0], 40)
        w["l0.canon1"][:] = 0.0
        w["l0.norm1"] = np.array(1.0)
        if latent:
            rank, dim, H = m["kv_rank"], m["dim"], m["heads"]
            assert m["q_rank"] <= rank
            w["l0.mix.dkv"][rank:] *= 0.02                      # hardly anything turns
            w["l0.mix.dq"][:] = np.roll(w["l0.mix.dkv"][:m["q_rank"]], 40, axis=1)
            w["l0.mix.dq.norm"][:] = w["l0.mix.dkv.norm"][:m["q_rank"]]
            uq = w["l0.mix.uq"].reshape(H, dim + m["rot_dim"], -1)
            uk = w["l0.mix.uk"].reshape(H, dim, rank)
            uk[..., m["q_rank"]:] = 0.0
            uq[:, :dim] = 2.5 * uk[..., :m["q_rank"]]
            w["l0.mix.sink"][:] = -3.0
        else:
            a = m["left"]
            q, k = w["l0.mix.left.q"].reshape(a["heads"], a["dim"], 80), w["l0.mix.left.k"].reshape(a["kv_heads"], a["dim"], 80)
            k[:, :a["rot"]["dims"]] *= 0.02
            k[:, a["rot"]["dims"]:] *= 2.0
            q[:] = np.repeat(np.roll(k, 40, axis=2), a["heads"] // a["kv_heads"], axis=0)
            w["l0.mix.left.q.b"][:] = 0.0
            w["l0.mix.left.k.b"][:] = 0.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=5, change=change)
    model = mc.load(folder, compute)
    sought, asking, filler = 0, 1, np.random.default_rng(2).integers(2, 60, 700)
    cases = [(q - window + 1 + off, q) for q in (window - 1, window, window + 5, 2 * window, 3 * window + 7) if q < 700 for off in (-1, 0, 1) if 0 <= q - window + 1 + off < q]
    cases += [(15, 16), (16, 31), (31, 32), (0, 1), (0, 15), (63, 64)]
    for key, query in cases:
        seen = query - key < window
        toks = filler[:query + 1].copy()
        toks[key], toks[query] = sought, asking
        want = oracle.logits(toks.tolist())[query]
        without = toks.copy()
        without[key] = 2
        shows = mc.row_errors(oracle.logits(without.tolist())[query], want)
        assert shows > 0.2 if seen else shows == 0, (key, query, shows)
        for portions in ([query + 1], [query, 1], mc.cut(query + 1, [48, 2])):
            got = mc.run_portions(model, toks.tolist(), portions)[query]
            assert mc.row_errors(got, want) <= mc.LIMIT[compute], (key, query, portions[:3])
    model.close()


@pytest.mark.parametrize("lanes", [2, 9])
@pytest.mark.parametrize("window", [4096, 700])
def test_long_histories_decoded_in_shares(mk, tmp_path, lanes, window):
    """A thousand keys (or the 700 of a window that starts inside a page), decoded together: shares of the keys meet one sink."""
    cfg = mc.mamivik([mc.rotated_latent(4, 48, 40, 64, 200, 24, window), mc.scaled_parallel((4, 2, 64, 32), (2, 32), window), mc.rotated_latent(33, 16, 24, 40, 128, 64, window)],
                     width=64, vocab=50, taps=4)
    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=1, change=lambda w: w.update({"l0.mix.sink": w["l0.mix.sink"] + 5.0, "l2.mix.sink": w["l2.mix.sink"] + 4.0}))
    seqs = [tokens_of(1000 - 111 * i, 50, seed=90 + i) for i in range(lanes)]
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


# ------------------------------------------------------------------------------------------------ parts that could be left out

PAR = mc.scaled_parallel((4, 2, 32, 16), (3, 32), 20)
LAT = mc.rotated_latent(4, 24, 32, 40, 48, 16, 20)


def zeros(name):
    return lambda w: w.update({name: np.zeros_like(w[name])})


def without_removal(w):
    """Removal rates of zero."""
    w["l0.mix.right.a.b"] = np.full_like(w["l0.mix.right.a.b"], -1e4)


PARTS = {
    # name: (layer, change of the weights, change of the layer, gains of tensors on both sides)
    "query biases": (PAR, zeros("l0.mix.left.q.b"), None, {"left.q.b": 4.0}),
    "key biases": (PAR, zeros("l0.mix.left.k.b"), None, {"left.k.b": 4.0}),
    "a left constant": (PAR, None, lambda l: l["mixer"].update(left_scale=1.0), {}),
    "a right constant": (PAR, None, lambda l: l["mixer"].update(right_scale=1.0), {}),
    "a scale": (PAR, None, lambda l: l["mixer"]["left"].update(scale=0.6), {}),
    "a removal": (PAR, without_removal, None, {}),
    "a removal's bias": (PAR, zeros("l0.mix.right.a.b"), None, {"right.a.b": 6.0, "right.a": 0.3, "right.o": 2.0}),
    "a decay's bias": (PAR, zeros("l0.mix.right.w0"), None, {}),
    "a decay that reads its input": (PAR, zeros("l0.mix.right.w2"), None, {"right.w2": 20.0, "right.w1": 3.0, "right.o": 2.0}),
    "a gate of the delta rule": (PAR, zeros("l0.mix.right.g"), None, {"right.g": 2.0}),
    "a convolution": (PAR, zeros("l0.canon1"), None, {}),
    "a sink": (LAT, lambda w: w.update({"l0.mix.sink": np.full_like(w["l0.mix.sink"], -1e30)}), None, {"sink": 3.0, "o": 2.0}),
    "a gate per value": (LAT, zeros("l0.mix.g"), None, {}),
    "a turned query part": (LAT, lambda w: w["l0.mix.dkv"].__setitem__(slice(48, None), 0.0), None, {}),
    "a stretched rotation": (mc.rotated_latent(4, 8, 32, 40, 48, 32, 64, scaling=dict(factor=16.0, original=64, fast=8.0, slow=1.0)), None,
                             lambda l: l["mixer"]["rot"]["scaling"].update(factor=1.0), {"uq": 2.0}),
    "an amplitude": (LAT, None, lambda l: l["mixer"]["rot"].update(scaling=None), {"uq": 2.0}),
}


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", PARTS)
def test_a_part_shows_and_is_there(mk, tmp_path, name, compute):
    """The plain statement without the part is far from the one with it, and the model follows the latter."""
    layer, change_w, change_layer, louder = PARTS[name]
    cfg = mc.mamivik([layer], width=64, vocab=60, taps=4)
    folder, oracle, w = checkpoint(tmp_path, cfg, seed=4, change=lambda w: w.update({f"l0.mix.{k}": f * w[f"l0.mix.{k}"] for k, f in louder.items()}))
    lacking_cfg, lacking_w = copy.deepcopy(cfg), {k: v.copy() for k, v in w.items()}
    if change_w:
        change_w(lacking_w)
    if change_layer:
        change_layer(lacking_cfg["layers"][0])
    toks = tokens_of(90, 60)
    want, lacking = oracle.logits(toks), mixers.decoder(lacking_cfg, lacking_w).logits(toks)
    assert np.sqrt(np.mean(mc.row_errors(lacking, want) ** 2)) > 1.5 * mc.LIMIT["bfloat16"]
    model = mc.load(folder, compute)
    for portions in ([90], mc.cut(90, [7, 2, 1]), [40] + [1] * 50):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


# ------------------------------------------------------------------------------------------------ the convolution's history

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_the_oldest_tap_crosses_every_cut(mk, tmp_path, taps, compute):
    """A convolution that is nothing but its oldest tap: the mixer and what follows see the token taps - 1 places back, across cuts
    shorter than the history, and zeros before the start."""
    cfg = mc.mamivik([mc.scaled_parallel((2, 1, 16, 8), (2, 16), 30), mc.rotated_latent(2, 16, 16, 20, 24, 8, 30)], width=48, vocab=40, taps=taps)

    def change(w):
        for l in (0, 1):
            w[f"l{l}.canon1"][:] = 0.0
            w[f"l{l}.canon1"][:, 0] = 3.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=8, change=change)
    toks = tokens_of(60, 40)
    model = mc.load(folder, compute)
    for portions in ([60], mc.cut(60, [1]), mc.cut(60, [2]), mc.cut(60, [2, 1, 3, 5]), mc.cut(60, [4, 9])):
        mc.assert_rows(mc.run_portions(model, toks, portions), oracle.logits(toks), compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("heads", [(3, 40), (2, 128), (2, 30), (1, 136)])
def test_wide_ticks_are_like_narrow_ones(mk, tmp_path, heads, compute):
    """Ticks of more rows than the kernels' small forms take, made of several lanes whose borders fall anywhere: prompts, a few tokens
    and single ones side by side, which take different forms of the delta rule."""
    cfg = mc.mamivik([mc.scaled_parallel((4, 2, 32, 16), heads, 50, ff=64), mc.rotated_latent(4, 24, 32, 40, 64, 16, 70, ff=40)], width=72, vocab=90, taps=4)
    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=3)
    seqs = [tokens_of(n, 90, seed=n) for n in (611, 2, 437, 53)]
    want = [oracle.logits(s) for s in seqs]
    model = mc.load(folder, compute, capacity=1200)
    for first in (1, 2, 0.5):
        sessions = [model.new_session() for _ in seqs]
        at = [int(first if first >= 1 else first * len(s)) for s in seqs]
        a, _ = model.forward_batch([(s, q[:k], 0) for s, q, k in zip(sessions, seqs, at)], want_tokens=False, rows=[range(k) for k in at])
        rest = [i for i in range(4) if at[i] < len(seqs[i])]
        b, _ = model.forward_batch([(sessions[i], seqs[i][at[i]:], at[i]) for i in rest], want_tokens=False, rows=[range(len(seqs[i]) - at[i]) for i in rest])
        got = [a[sum(at[:i]):sum(at[:i + 1])] for i in range(4)]
        offset = 0
        for i in rest:
            n = len(seqs[i]) - at[i]
            got[i] = np.concatenate([got[i], b[offset:offset + n]])
            offset += n
        for i in range(4):
            mc.assert_rows(got[i], want[i], compute, f"sequence {i}, first {at[i]} tokens")
        for s in sessions:
            s.close()
    model.close()


# ------------------------------------------------------------------------------------------------ the delta rule's state

@pytest.mark.parametrize("heads", [(2, 64), (3, 128), (2, 100), (3, 48)])
@pytest.mark.parametrize("decay", [None, -12.0, 12.0])
def test_forms_of_the_delta_rule_agree(mk, tmp_path, heads, decay):
    """In bfloat16 models the forms differ by what a rounding of their finished rows may flip: prompts in chunks, portions that go row
    by row, single tokens, and prompts cut at and beside a chunk's edge - with random, no and the fastest decay."""
    cfg = mc.mamivik([mc.scaled_parallel((2, 1, 16, 8), heads, 4, scales=(0.0, 1.0))], width=96, vocab=50, taps=2)

    def change(w):
        if decay is not None:
            w["l0.mix.right.w0"][:] = decay

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=3, rank=16, change=change)
    model = mc.load(folder, "bfloat16")
    toks = tokens_of(330, 50, seed=1)
    base = oracle.embedding_output(toks)
    size = np.sqrt(np.mean((oracle.residuals(toks)[0] - base) ** 2))
    model.capture_residuals(True)
    out = []
    for portions in (mc.cut(330, [1]), [330], mc.cut(330, [40]), [64, 266], [63, 65, 202], mc.cut(330, [128, 2, 49])):
        s, at, got = model.new_session(), 0, []
        for k in portions:
            model.forward_batch([(s, toks[at:at + k], at)], want_logits=False, want_tokens=False, rows=[[]])
            got.append(model.residuals(k)[0])
            at += k
        s.close()
        out.append(np.concatenate(got))
    for other in out[1:]:
        assert np.sqrt(np.mean((other - out[0]) ** 2)) / size < 6e-4
        assert np.sqrt(np.mean((other - out[0]) ** 2, axis=1)).max() / size < 5e-3
    model.close()

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("heads", [(2, 32), (3, 64), (1, 150)])
def test_one_far_write_stays_in_the_state(mk, tmp_path, heads, compute):
    """Hardly any decay or removal: what the first token wrote, far larger than the rest, is read hundreds of tokens later.  (150
    channels: the form without the finishing step, on one-token ticks too.)"""
    cfg = mc.mamivik([mc.scaled_parallel((2, 1, 16, 8), heads, 4, scales=(0.0, 1.0))], width=64, vocab=50, taps=2)
    mark, const = 0, 1   # channels: one that tells the first token, and one that is the same for all

    def change(w):
        w["embed"][:, mark] = 0.0
        w["embed"][0, mark] = 8.0
        w["embed"][:, const] = 6.0
        w["l0.canon1"][:] = 0.0
        key = np.random.default_rng(1).standard_normal(heads[0] * heads[1])
        w["l0.mix.right.k"] *= 0.03
        w["l0.mix.right.k"][:, mark] = key                # only the first token writes along it
        w["l0.mix.right.r"] *= 0.1
        w["l0.mix.right.r"][:, const] = key               # and everyone asks for it
        w["l0.mix.right.w0"][:] = -9.0
        w["l0.mix.right.w2"] *= 0.0
        w["l0.mix.right.a"] *= 0.0
        w["l0.mix.right.a.b"][:] = -9.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=6, change=change)
    toks = [0] + (1 + np.random.default_rng(4).integers(0, 49, 399)).tolist()
    want, lost = oracle.logits(toks), oracle.logits([1] + toks[1:])
    assert mc.row_errors(lost[-40:], want[-40:]).min() > 2 * mc.LIMIT["bfloat16"]
    model = mc.load(folder, compute)
    for portions in ([400], mc.cut(400, [37, 1, 2, 100]), mc.cut(400, [16, 64, 65]), [64] + [1] * 336):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("heads", [(2, 32), (2, 64), (3, 128)])
@pytest.mark.parametrize("fast", [False, True])
def test_keys_that_come_again_are_replaced(mk, tmp_path, heads, fast, compute):
    """Few different tokens and removal rates near one: the same keys are removed and written over and over, with the slowest and
    the fastest decay the design has (what a chunk of rows multiplies up stays in range)."""
    cfg = mc.mamivik([mc.scaled_parallel((2, 1, 16, 8), heads, 4, scales=(0.0, 1.0))], width=64, vocab=6, taps=2)

    def change(w):
        w["l0.canon1"] *= 0.1
        w["l0.mix.right.w2"] *= 0.0
        w["l0.mix.right.w0"][:] = 12.0 if fast else -12.0
        w["l0.mix.right.a.b"][:] = 5.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=10, change=change)
    toks = tokens_of(300, 6, seed=1)
    want = oracle.logits(toks)
    model = mc.load(folder, compute)
    for portions in ([300], mc.cut(300, [33, 2, 63]), [150] + [1] * 150):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
def test_decays_that_differ_by_channel(mk, tmp_path, compute):
    """Half of the key channels forget as fast as they can, the others not at all, and which half it is changes from token to token."""
    cfg = mc.mamivik([mc.scaled_parallel((2, 1, 16, 8), (2, 64), 4, scales=(0.0, 1.0))], width=64, vocab=50, taps=2)

    def change(w):
        w["l0.mix.right.w1"] *= 4.0
        w["l0.mix.right.w2"] *= 12.0
        w["l0.mix.right.w0"][:64] = np.where(np.arange(64) % 2, 8.0, -8.0)

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=12, change=change)
    toks = tokens_of(330, 50, seed=2)
    want = oracle.logits(toks)
    model = mc.load(folder, compute)
    limit = mc.LIMIT[compute] * (1 if compute == "float32" else 2)   # gates this steep carry the rounding of their bfloat16 inputs
    for portions in ([330], mc.cut(330, [5, 64, 17, 1]), [100] + [1] * 230):
        assert mc.row_errors(mc.run_portions(model, toks, portions), want).max() <= limit
    model.close()


# ------------------------------------------------------------------------------------------------ kernels' limits

@pytest.mark.parametrize("layer,message", [
    (mc.scaled_parallel((1, 1, 300, 8), (1, 8), 4), "above 256"),
    (mc.scaled_parallel((1, 1, 8, 8), (1, 300), 4), "above 256"),
    (mc.scaled_parallel((80, 1, 4, 4), (1, 8), 4), "64 query heads"),
    (mc.rotated_latent(1, 8, 8, 8, 1020, 16, 4), "above 1024"),
])
def test_sizes_beyond_the_kernels_are_refused(mk, tmp_path, layer, message):
    capi = importlib.import_module("macllm_infer_b200._capi")
    cfg = mc.mamivik([layer], width=64, vocab=20)
    with pytest.raises(capi.MkError) as e:
        mc.load(mc.write(tmp_path / "m", cfg, mc.weights(cfg)), "bfloat16")
    assert message in str(e.value)
