"""Tevanex decoders on the GPU: what random weights would hide - chunk edges, sinks, capped scores, gates, far writes of the matrix
memory, its running maximum, clamped experts, wide and narrow routing, tensors run twice - each made to stand out, against the plain
statement (oracle/mixers.py).  tests/test_mixer_gpu.py runs whole models of the design beside the others."""
import importlib

import numpy as np
import pytest

import mixer_cases as mc
from oracle import mixers

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def checkpoint(tmp_path, cfg, seed=0, change=None):
    w = mc.weights(cfg, seed)
    if change:
        change(w)
        w = {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in w.items()}
    return mc.write(tmp_path / "m", cfg, w), mixers.decoder(cfg, w), w


def tokens_of(n, vocab, seed=3):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


# ------------------------------------------------------------------------------------------------ chunk edges

EDGES = {
    "sink, chunk of three pages": mc.sink_attention(4, 2, 64, 64, 32, 48),
    "sink, odd chunk, three heads per key": mc.sink_attention(6, 2, 24, 40, 8, 37),
    "capped, chunk of four pages": mc.capped_attention(4, 2, 64, 48, 32, 64, softcap=60.0),
    "capped, odd chunk": mc.capped_attention(8, 1, 40, 24, 12, 50, softcap=60.0),
    "sink, long chunk": mc.sink_attention(4, 1, 32, 32, 16, 448),
}


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", EDGES)
def test_one_key_stands_out_inside_its_chunk_and_is_gone_outside(mk, tmp_path, name, compute):
    """A query projects the other half of the embedding's channels with the key's matrix, and the asking token's embedding is the
    sought one's with its halves exchanged: in the dimensions that do not turn the query meets exactly that key.  The sought
    token sits at the first place of the query's chunk, just before it, at page borders and right before the query."""
    layer = EDGES[name]
    m = layer["mixer"]
    cfg = mc.tevanex([layer], width=80, vocab=60, embed=2.0, softcap=30.0)
    heads, group, dim, turned, chunk = m["heads"], m["heads"] // m["kv_heads"], m["dim"], m["rot"]["dims"], m["mask"]["size"]

    def change(w):
        q, k = w["l0.mix.q"].reshape(heads, dim, 80), w["l0.mix.k"].reshape(-1, dim, 80)
        q[:] = np.repeat(np.roll(k, 40, axis=2), group, axis=0)
        w["embed"][1] = np.roll(w["embed"][0], 40)
        w["l0.mix.q.b"] *= 0
        w["l0.mix.k.b"] *= 0
        for n, h in (("q", heads), ("k", heads // group)):
            w[f"l0.mix.{n}.norm"].reshape(h, dim)[:, :turned] = 0.05
            w[f"l0.mix.{n}.norm"].reshape(h, dim)[:, turned:] = 4.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=5, change=change)
    model = mc.load(folder, compute)
    sought, asking, filler = 0, 1, np.random.default_rng(2).integers(2, 60, 500)
    first = 2 * chunk if 3 * chunk < 500 else 0   # a chunk with others in front of it
    cases = [(first, first + chunk - 1), (first, first + 1), (first + 1, first + chunk // 2), (first + chunk - 2, first + chunk - 1)]
    if first:
        cases += [(first - 1, first), (first - 1, first + chunk - 1), (first - chunk, first), (first + chunk - 1, first + chunk), (0, first)]
    else:
        cases += [(15, 16), (16, 31), (63, 400), (447, 448), (0, 448), (448, 449)]
    for key, query in cases:
        seen = key // chunk == query // chunk
        toks = filler[:query + 1].copy()
        toks[key], toks[query] = sought, asking
        want = oracle.logits(toks.tolist())[query]
        without = toks.copy()
        without[key] = 2
        shows = mc.row_errors(oracle.logits(without.tolist())[query], want)
        assert shows > 0.2 if seen else shows == 0
        for portions in ([query + 1], [query, 1], mc.cut(query + 1, [48, 2])):
            got = mc.run_portions(model, toks.tolist(), portions)[query]
            assert mc.row_errors(got, want) <= mc.LIMIT[compute], (key, query, portions[:3])
    model.close()


@pytest.mark.parametrize("lanes", [2, 9])
@pytest.mark.parametrize("chunk", [4096, 700])
def test_long_histories_decoded_in_shares(mk, tmp_path, lanes, chunk):
    """A thousand keys in one chunk (or a few hundred after its edge), decoded together: shares of the keys meet one sink."""
    cfg = mc.tevanex([mc.sink_attention(4, 2, 64, 40, 64, chunk), mc.capped_attention(2, 1, 32, 64, 16, chunk)], width=64, vocab=50)
    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=1, change=lambda w: w.update({"l0.mix.sink": w["l0.mix.sink"] + 5.0}))
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

def without_sink(w):
    w["l0.mix.sink"] = np.full_like(w["l0.mix.sink"], -1e30)


def without_bias(name):
    def change(w):
        w[f"l0.mix.{name}.b"] = np.zeros_like(w[f"l0.mix.{name}.b"])
    return change


def without_gate(w):
    w["l0.mix.g"] = np.zeros_like(w["l0.mix.g"])


PARTS = {
    "a sink": (mc.sink_attention(4, 2, 32, 32, 16, 20), without_sink, {}, {}),
    "query biases": (mc.sink_attention(4, 2, 32, 32, 16, 20), without_bias("q"), {}, {"q.b": 6.0}),
    "key biases": (mc.capped_attention(4, 2, 32, 32, 16, 20), without_bias("k"), {}, {"k.b": 20.0, "q.b": 6.0}),
    "value biases": (mc.sink_attention(4, 2, 32, 32, 16, 20), without_bias("v"), {}, {"v.b": 4.0}),
    "output biases": (mc.capped_attention(4, 2, 32, 32, 16, 20), without_bias("o"), {}, {"o.b": 4.0}),
    "a gate per value": (mc.capped_attention(4, 2, 32, 32, 16, 20), without_gate, {}, {}),
    "capped scores": (mc.capped_attention(4, 2, 32, 32, 16, 20, softcap=0.8), None, {"softcap": 1e6}, {}),
    "a scale": (mc.sink_attention(4, 2, 32, 32, 16, 20), None, {"scale": 0.6}, {}),
    "a gate cap": (mc.mlstm(3, 32, 32, cap=0.7), None, {"gate_cap": 1e6}, {}),
    "an expert's limit": (mc.mlstm(1, 8, 8, mlp=mc.experts(4, 2, 32, 0.3)), None, {"expert": 1e6}, {}),
    "a shared expert's limit": (mc.mlstm(1, 8, 8, mlp=mc.experts(4, 2, 32, 5.0, (64, 0.2))), None, {"shared": 1e6}, {}),
    "a stretched rotation": (mc.capped_attention(4, 2, 32, 32, 32, 64, softcap=50.0, yarn=dict(factor=16.0, original=64, fast=8.0, slow=1.0)), None, {"factor": 1.0}, {}),
}


@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("name", PARTS)
def test_a_part_shows_and_is_there(mk, tmp_path, name, compute):
    """The plain statement without the part is far from the one with it, and the model follows the latter."""
    import copy
    layer, change, other, louder = PARTS[name]
    cfg = mc.tevanex([layer], width=64, vocab=60)
    folder, oracle, w = checkpoint(tmp_path, cfg, seed=4, change=lambda w: w.update({f"l0.mix.{k}": f * w[f"l0.mix.{k}"] for k, f in louder.items()}))
    lacking_cfg, lacking_w = copy.deepcopy(cfg), dict(w)
    if change:
        change(lacking_w)
    l = lacking_cfg["layers"][0]
    for key, value in other.items():
        if key in ("expert", "shared"):
            l["mlp"][key]["limit"] = value
        elif key == "factor":
            l["mixer"]["rot"]["scaling"]["factor"] = value
        else:
            l["mixer"][key] = value
    toks = tokens_of(90, 60)
    want, lacking = oracle.logits(toks), mixers.decoder(lacking_cfg, lacking_w).logits(toks)
    assert np.sqrt(np.mean(mc.row_errors(lacking, want) ** 2)) > 2 * mc.LIMIT["bfloat16"]
    model = mc.load(folder, compute)
    for portions in ([90], mc.cut(90, [7, 2, 1]), [40] + [1] * 50):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


# ------------------------------------------------------------------------------------------------ matrix memory

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("sizes", [(2, 32, 32), (3, 24, 150)])
def test_one_far_write_stays_in_the_matrix_memory(mk, tmp_path, sizes, compute):
    """Forget gates that stay open and input gates that stay shut but for the first token: its write is read hundreds of tokens
    later.  (150 values: the form without the finishing step, on one-token ticks too.)"""
    cfg = mc.tevanex([mc.mlstm(*sizes, cap=12.0)], width=64, vocab=50, embed=1.0)
    mark = 0   # the channel that tells the first token

    def change(w):
        w["embed"][:, mark] = -2.0
        w["embed"][0, mark] = 4.0
        w["embed"][:, 1] = 3.0
        w["l0.mix.q"][:, 1] = 2.0 * w["l0.mix.k"][:, mark]     # every query meets the first token's key
        w["l0.mix.i"] *= 0.05
        w["l0.mix.i"][:, mark] = 2.0
        w["l0.mix.i.b"][:] = -2.0
        w["l0.mix.f"] *= 0.05
        w["l0.mix.f.b"][:] = 11.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=6, change=change)
    toks = [0] + (1 + np.random.default_rng(4).integers(0, 49, 399)).tolist()
    want, lost = oracle.logits(toks), oracle.logits([1] + toks[1:])
    assert mc.row_errors(lost[-40:], want[-40:]).min() > 2 * mc.LIMIT["bfloat16"]
    model = mc.load(folder, compute)
    for portions in ([400], mc.cut(400, [37, 1, 2, 100]), [64] + [1] * 336):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


@pytest.mark.parametrize("compute", DTYPES)
def test_the_running_maximum_is_carried(mk, tmp_path, compute):
    """Input gates of e^40 and shut forget gates in turn: without a maximum that moves with the state the sums leave the range of a
    float, and a maximum that is lost at a cut shows at once.  Where the state is nearly empty the floor of the denominator counts."""
    cfg = mc.tevanex([mc.mlstm(3, 16, 20, cap=45.0)], width=48, vocab=40, embed=1.0)

    def change(w):
        w["l0.mix.i"] *= 0.02
        w["l0.mix.f"] *= 0.02
        w["l0.mix.i"][:, 0] = 3.0
        w["l0.mix.f"][:, 1] = 3.0
        w["embed"][:, 0] = np.linspace(-9, 11, 40)
        w["embed"][:, 1] = np.random.default_rng(0).permutation(np.linspace(-3, 8, 40))

    folder, oracle, w = checkpoint(tmp_path, cfg, seed=2, change=change)
    toks = tokens_of(200, 40, seed=8)
    want = oracle.logits(toks)
    assert np.isfinite(want).all()
    x = oracle.embedding_output(toks)
    i, f = mixers.mlstm_gates(x @ w["l0.mix.i"].T.astype(np.float64) + w["l0.mix.i.b"], x @ w["l0.mix.f"].T.astype(np.float64) + w["l0.mix.f.b"], 45.0)
    assert i.max() > 25 and i.min() < -20 and f.min() < -5
    model = mc.load(folder, compute)
    whole = mc.run_portions(model, toks, [200])
    limit = mc.LIMIT[compute] * (1 if compute == "float32" else 4)   # gates of this size carry the rounding of their bfloat16 inputs
    assert mc.row_errors(whole, want).max() <= limit
    for portions in (mc.cut(200, [3, 17, 64, 1]), mc.cut(200, [2]), [100] + [1] * 100):
        got = mc.run_portions(model, toks, portions)
        assert mc.row_errors(got, want).max() <= limit
        assert mc.row_errors(got, whole).max() <= mc.LIMIT["float32"] * (1 if compute == "float32" else 100)
    model.close()


# ------------------------------------------------------------------------------------------------ experts

@pytest.mark.parametrize("compute", DTYPES)
@pytest.mark.parametrize("mlp", [mc.experts(3, 2, 40, 0.7), mc.experts(64, 4, 24, 1.0, (33, 0.5)), mc.experts(7, 4, 96, 1.0, (20, 0.9)), mc.experts(20, 1, 16)])
def test_wide_ticks_route_like_narrow_ones(mk, tmp_path, mlp, compute):
    """Ticks of a thousand and more routed rows (grouped over the whole GPU, wide tiles), of a few, and of one."""
    cfg = mc.tevanex([mc.capped_attention(2, 1, 32, 32, 16, 64, mlp=mlp), mc.sink_attention(2, 1, 16, 16, 8, 40, mlp=mlp)], width=72, vocab=90)
    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=3)
    toks = tokens_of(1100, 90)
    want = oracle.logits(toks)
    model = mc.load(folder, compute, capacity=1200)
    for portions in ([1100], [300, 2, 1, 400, 30, 367], [1090] + [1] * 10):
        mc.assert_rows(mc.run_portions(model, toks, portions), want, compute, f"portions {portions[:4]}")
    model.close()


def test_every_token_on_one_expert(mk, tmp_path):
    """All rows of a tick meet one expert, and the other experts none."""
    cfg = mc.tevanex([mc.capped_attention(2, 1, 32, 32, 16, 64, mlp=mc.experts(9, 1, 48, 0.8, (30, 0.8)))], width=64, vocab=40)

    def change(w):
        w["l0.mlp.router"] *= 0.1
        w["l0.mlp.router"][6, :mc.ROUTING] = 0.0
        w["l0.mlp.router"][6, 0] = 3.0
        w["embed"][:, 0] = 1.0

    folder, oracle, _ = checkpoint(tmp_path, cfg, seed=3, change=change)
    toks = tokens_of(400, 40)
    model = mc.load(folder, "bfloat16")
    for portions in ([400], mc.cut(400, [64, 1, 65])):
        mc.assert_rows(mc.run_portions(model, toks, portions), oracle.logits(toks), "bfloat16", f"portions {portions[:3]}")
    model.close()


# ------------------------------------------------------------------------------------------------ tensors run twice

@pytest.mark.parametrize("compute", DTYPES)
def test_layers_run_again_keep_a_cache_and_a_state_of_their_own(mk, tmp_path, compute):
    """Against the same layers with copies of the tensors, through a chain of references and an order of its own."""
    base = [mc.mlstm(2, 24, 20, mlp=mc.experts(4, 2, 24)), mc.capped_attention(4, 2, 32, 32, 16, 30)]
    layers = base + [mc.again(base, 1), mc.again(base, 0)]
    layers.append({**layers[3], "weights_of": 3})      # which runs layer 0
    cfg = mc.tevanex(layers, width=64, vocab=60)
    w = mc.weights(cfg, 9)
    copied = dict(w)
    plain = []
    for i, l in enumerate(layers):
        plain.append({k: v for k, v in l.items() if k != "weights_of"})
        root = {2: 1, 3: 0, 4: 0}.get(i)
        if root is not None:
            copied.update({f"l{i}." + k[3:]: v for k, v in w.items() if k.startswith(f"l{root}.")})
    shared = mc.load(mc.write(tmp_path / "shared", cfg, w), compute)
    copies = mc.load(mc.write(tmp_path / "copies", {**cfg, "layers": plain}, copied), compute)
    toks = tokens_of(100, 60)
    want = mixers.decoder(cfg, w).logits(toks)
    for portions in ([100], mc.cut(100, [31, 2, 1])):
        a, b = mc.run_portions(shared, toks, portions), mc.run_portions(copies, toks, portions)
        mc.assert_rows(a, want, compute)
        assert np.array_equal(a, b)
    shared.close()
    copies.close()


def test_weight_bytes_count_shared_tensors_once(mk, tmp_path):
    base = [mc.mlstm(2, 24, 20, mlp=mc.experts(4, 2, 24))]
    one = mc.load(mc.write(tmp_path / "one", mc.tevanex(base), mc.weights(mc.tevanex(base))), "bfloat16")
    cfg = mc.tevanex(base + [mc.again(base, 0)])
    two = mc.load(mc.write(tmp_path / "two", cfg, mc.weights(cfg)), "bfloat16")
    assert one.spec().weight_bytes == two.spec().weight_bytes and one.spec().weight_bytes_per_token < two.spec().weight_bytes_per_token
    assert (one.spec().n_layers, two.spec().n_layers) == (1, 2)
    one.close()
    two.close()


# ------------------------------------------------------------------------------------------------ kernels' limits

@pytest.mark.parametrize("layer,message", [
    (mc.mlstm(1, 300, 8), "above 256"),
    (mc.sink_attention(1, 1, 300, 8, 16, 8), "above 256"),
    (mc.sink_attention(80, 1, 4, 4, 4, 8), "64 query heads"),
])
def test_sizes_beyond_the_kernels_are_refused(mk, tmp_path, layer, message):
    capi = importlib.import_module("macllm_infer_b200._capi")
    cfg = mc.tevanex([layer], width=64, vocab=20)
    with pytest.raises(capi.MkError) as e:
        mc.load(mc.write(tmp_path / "m", cfg, mc.weights(cfg)), "bfloat16")
    assert message in str(e.value)
