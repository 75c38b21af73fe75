"""Small random checkpoints of mixer-built decoders, and schedules that cut sequences into forwards, for the tests."""
import importlib
import json

import numpy as np

from oracle import mixers

SCALING = dict(factor=8.0, low=1.0, high=4.0, original=64)


def wkv(heads, dim, ff=0):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel(left, right, ff=0):
    """left = (heads, kv_heads, dim, vdim, rot dims, scaled?), right = (heads, kv_heads, dim, vdim, taps)."""
    h, g, d, e, rd, scaled = left
    rot = {"dims": rd, "base": 500.0, "scaling": dict(SCALING) if scaled else None} if rd else None
    rh, rg, rk, rv, taps = right
    return {"type": "parallel",
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": e, "scale": 0.9 / d ** 0.5, "rot": rot},
                      "right": {"heads": rh, "kv_heads": rg, "dim": rk, "vdim": rv, "conv": taps}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mingru(width, ff=0):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, vdim, q_rank, kv_rank, ff=0):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": 0.9 / dim ** 0.5}}


def kunonex(layers, width=96, vocab=131, loop=None, eps=3e-5, logit_scale=0.7):
    """loop = (start, stop, times)."""
    return {"architecture": "Kunonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None, "layers": layers}


def config(layers, width=96, vocab=131, side=12, eps=3e-5):
    return {"architecture": "Sizilorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "token_side": {"dim": side} if side else None, "layers": layers}


def experts(n, top, ff, limit=1.0, shared=None):
    """shared = (ff, limit) of the expert every token runs."""
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": {"ff": shared[0], "limit": shared[1]} if shared else None}


def mlstm(heads, dim, vdim, cap=4.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


def sink_attention(heads, kv_heads, dim, vdim, rot, chunk, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 0.9 / dim ** 0.5,
                                                       "mask": {"size": chunk}, "rot": {"base": 500.0, "dims": rot}}}


def capped_attention(heads, kv_heads, dim, vdim, rot, chunk, softcap=2.5, mlp=None, yarn=YARN):
    m = sink_attention(heads, kv_heads, dim, vdim, rot, chunk, mlp)
    m["type"] = "attention_2"
    m["mixer"]["softcap"] = softcap
    m["mixer"]["rot"]["scaling"] = dict(yarn)
    return m


def again(layers, i):
    """An entry that runs layer i's tensors again."""
    return {**layers[i], "weights_of": i}


def tevanex(layers, width=96, vocab=131, eps=3e-5, embed=1.7, mult=0.6, logit_scale=0.8, softcap=9.0):
    return {"architecture": "Tevanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "residual_mult": mult, "logit_scale": logit_scale, "logit_softcap": softcap, "layers": layers}


ROUTING = 8   # channels that only embeddings write and routers read, so that a choice is a token's and never close; one more is constant


def tevanex_weights(cfg, seed):
    rng = np.random.default_rng(seed)
    C, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def around_one(name, n):
        w[name] = 1.0 + 0.3 * rng.standard_normal(n)

    def bias(name, n, dev=0.3):
        w[name] = dev * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((V, C))
    w["embed"][:, ROUTING] = 1.0
    routers = []
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "mlstm":
            mat(p + "mix.q", H * d, C)
            mat(p + "mix.k", H * d, C)
            mat(p + "mix.v", H * e, C)
            # the constant channel gives queries and keys a common part: denominators are sums without much cancellation
            w[p + "mix.q"][:, ROUTING] = w[p + "mix.k"][:, ROUTING] = rng.standard_normal(H * d)
            mat(p + "mix.g", H * e, C)
            for s, b in (("i", -1.0), ("f", 3.0)):
                mat(p + "mix." + s, H, C)
                w[p + "mix." + s + ".b"] = b + rng.standard_normal(H)
            around_one(p + "mix.norm", H * e)
        else:
            G = m["kv_heads"]
            for s, n in (("q", H * d), ("k", G * d), ("v", G * e)):
                mat(p + "mix." + s, n, C)
                bias(p + "mix." + s + ".b", n)
            w[p + "mix.q.norm"] = 1.5 + 0.3 * rng.standard_normal(H * d)
            w[p + "mix.k.norm"] = 1.5 + 0.3 * rng.standard_normal(G * d)
            bias(p + "mix.o.b", C)
            if layer["type"] == "attention":
                w[p + "mix.sink"] = 1.5 + rng.standard_normal(H)
            else:
                mat(p + "mix.g", H * e, C)
        mat(p + "mix.o", C, H * e)
        around_one(p + "norm1", C)
        w[p + "norm1"][:ROUTING + 1] = 0.0
        if layer["mlp"]:
            x = layer["mlp"]
            around_one(p + "norm2", C)
            w[p + "norm2"][:ROUTING + 1] = 0.0
            for name, ff in [(f"e{j}", x["expert"]["ff"]) for j in range(x["router"]["experts"])] + ([("shared", x["shared"]["ff"])] if x["shared"] else []):
                mat(p + f"mlp.{name}.gate", ff, C)
                mat(p + f"mlp.{name}.up", ff, C)
                mat(p + f"mlp.{name}.down", C, ff)
            if x["shared"]:
                mat(p + "mlp.shared.sg", 1, C)
            r = np.zeros((x["router"]["experts"], C))
            r[:, :ROUTING] = mixers.bf16(rng.standard_normal((len(r), ROUTING)).astype(np.float32) / np.sqrt(ROUTING) / cfg["embedding"]["scale"])
            w[p + "mlp.router"] = r
            routers.append((r, x["router"]["top"]))
    # a token's last chosen and first left-out logits are well apart in every layer
    for t in range(V):
        for _ in range(100000):
            z = [np.sort(r @ (w["embed"][t] * cfg["embedding"]["scale"]))[::-1] for r, _ in routers]
            if all(k == len(s) or s[k - 1] - s[k] > 0.06 for s, (_, k) in zip(z, routers)):
                break
            w["embed"][t, :ROUTING] = 1.5 * rng.standard_normal(ROUTING)
        else:
            raise AssertionError("no embedding with clear choices was found")
    around_one("final.norm", C)
    mat("head", V, C, 2.0)
    return w


def kunonex_weights(cfg, seed):
    rng = np.random.default_rng(seed)
    C, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def around_one(name, n):
        w[name] = 1.0 + 0.3 * rng.standard_normal(n)

    def bias(name, n, dev=0.3):
        w[name] = dev * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((V, C))
    around_one("embed.norm", C)
    if cfg["loop"]:
        mat("loop.in", C, 2 * C)
        bias("loop.step", (cfg["loop"]["times"], C))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        around_one(p + "norm1", C)
        w[p + "shift"] = rng.uniform(0, 1, C)
        if layer["type"] == "mingru":
            n = m["width"]
            for s in "zxg":
                mat(p + "mix." + s, n, C)
            w[p + "mix.z.b"] = rng.uniform(-5.0, 1.0, n)
            bias(p + "mix.x.b", n)
            mat(p + "mix.o", C, n)
        else:
            mat(p + "mix.dq", m["q_rank"], C)
            around_one(p + "mix.dq.norm", m["q_rank"])
            mat(p + "mix.uq", m["heads"] * m["dim"], m["q_rank"], 2.0)
            mat(p + "mix.dkv", m["kv_rank"], C)
            around_one(p + "mix.dkv.norm", m["kv_rank"])
            mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5)
            mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(p + "mix.g", m["heads"], C)
            mat(p + "mix.o", C, m["heads"] * m["vdim"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            mat(p + "mlp.up", ff, C)
            bias(p + "mlp.up.b", ff)
            mat(p + "mlp.down", C, ff)
            bias(p + "mlp.down.b", C)
            w[p + "mlp.act"] = np.array([0.6, 0.4, -0.3, 0.2]) + 0.1 * rng.standard_normal(4)
    around_one("final.norm", C)
    mat("head", V, C)
    return w


def scaled_parallel(left, right, window, scales=(0.8, 0.5), ff=0, base=500.0, scale=None):
    """left = (heads, kv_heads, dim, rot dims), right = (heads, dim)."""
    h, g, d, rd = left
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "scale": scale or 0.9 / d ** 0.5, "mask": {"size": window},
                               "rot": {"base": base, "dims": rd}},
                      "right": {"heads": right[0], "dim": right[1]}, "left_scale": scales[0], "right_scale": scales[1]}}


def rotated_latent(heads, dim, vdim, q_rank, kv_rank, rot_dim, window, ff=0, scaling=YARN, base=500.0, scale=None):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot_dim,
                      "scale": scale or 0.9 / (dim + rot_dim) ** 0.5, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim, "scaling": dict(scaling) if scaling else None}}}


def mamivik(layers, width=96, vocab=131, taps=3, eps=3e-5):
    return {"architecture": "Mamivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


def mamivik_weights(cfg, seed, rank):
    rng = np.random.default_rng(seed)
    C, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def around_one(name, *shape):
        w[name] = 1.0 + 0.3 * rng.standard_normal(shape)

    w["embed"] = rng.standard_normal((V, C))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        around_one(p + "norm1")
        w[p + "canon1"] = rng.standard_normal((C, taps)) * 0.6 / np.sqrt(taps)
        if layer["type"] == "parallel":
            a, L, R = m["left"], p + "mix.left.", p + "mix.right."
            n = m["right"]["heads"] * m["right"]["dim"]
            for x, heads in (("q", a["heads"]), ("k", a["kv_heads"])):
                mat(L + x, heads * a["dim"], C, 1.3)
                w[L + x + ".b"] = 0.4 * rng.standard_normal(heads * a["dim"])
            mat(L + "o", C, a["heads"] * a["dim"])
            for x in "kvga":
                mat(R + x, n, C)
            # queries that have something in common with the keys: what the heads give is a sum without much cancellation, from the
            # first token on
            w[R + "r"] = 0.8 * w[R + "k"] + 0.6 * rng.standard_normal((n, C)) / np.sqrt(C)
            w[R + "a.b"] = rng.standard_normal(n)
            mat(R + "w1", rank, C)
            mat(R + "w2", n, rank)
            w[R + "w0"] = rng.uniform(-6.0, 2.0, n)
            around_one(R + "norm", n)
            mat(R + "o", C, n)
        else:
            H, q_rank, kv_rank = m["heads"], m["q_rank"], m["kv_rank"]
            mat(p + "mix.dq", q_rank, C)
            around_one(p + "mix.dq.norm", q_rank)
            mat(p + "mix.uq", H * (m["dim"] + m["rot_dim"]), q_rank, 1.5)
            mat(p + "mix.dkv", kv_rank + m["rot_dim"], C)
            around_one(p + "mix.dkv.norm", kv_rank)
            mat(p + "mix.uk", H * m["dim"], kv_rank, 1.2)
            mat(p + "mix.uv", H * m["vdim"], kv_rank)
            w[p + "mix.sink"] = 1.0 + rng.standard_normal(H)
            mat(p + "mix.g", H * m["vdim"], C)
            mat(p + "mix.o", C, H * m["vdim"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            around_one(p + "norm2")
            mat(p + "mlp.gate", ff, C)
            mat(p + "mlp.up", ff, C)
            mat(p + "mlp.down", C, ff)
    around_one("final.norm")
    mat("head", V, C)
    return w


def weights(cfg, seed=0, rank=5):
    """name -> float32 array holding bfloat16 values."""
    if cfg["architecture"] == "Mamivik":
        return {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in mamivik_weights(cfg, seed, rank).items()}
    if cfg["architecture"] == "Kunonex":
        return {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in kunonex_weights(cfg, seed).items()}
    if cfg["architecture"] == "Tevanex":
        return {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in tevanex_weights(cfg, seed).items()}
    rng = np.random.default_rng(seed)
    C, V, side = cfg["width"], cfg["vocab"], (cfg.get("token_side") or {}).get("dim", 0)
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def around_one(name, n):
        w[name] = 1.0 + 0.3 * rng.standard_normal(n)

    def norm(name):
        around_one(name, C)
        w[name + ".b"] = 0.1 * rng.standard_normal(C)
        w[name + ".alpha"] = np.array(rng.uniform(0.5, 0.9))

    w["embed"] = rng.standard_normal((V, C))
    if side:
        w["side.embed"] = rng.standard_normal((V, side * len(cfg["layers"])))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                w[p + "mix.mu." + s] = rng.uniform(0, 1, C)
            for s in "rkvg":
                mat(p + "mix." + s, n, C)
            mat(p + "mix.w1", rank, C)
            mat(p + "mix.w2", n, rank)
            w[p + "mix.w0"] = rng.uniform(-6.0, 0.5, n)
            w[p + "mix.u"] = rng.standard_normal((m["heads"], m["dim"]))
            around_one(p + "mix.norm", n)
            mat(p + "mix.o", C, n)
        else:
            a, d = m["left"], m["right"]
            L, R = p + "mix.left.", p + "mix.right."
            mat(L + "q", a["heads"] * a["dim"], C)
            mat(L + "k", a["kv_heads"] * a["dim"], C)
            mat(L + "v", a["kv_heads"] * a["vdim"], C)
            mat(L + "g", a["heads"], C)
            w[L + "q.norm"] = 1.5 + 0.3 * rng.standard_normal(a["dim"])
            w[L + "k.norm"] = 1.5 + 0.3 * rng.standard_normal(a["dim"])
            mat(L + "o", C, a["heads"] * a["vdim"])
            around_one(L + "out", C)
            for s, n in (("q", d["kv_heads"] * d["dim"]), ("k", d["kv_heads"] * d["dim"]), ("v", d["heads"] * d["vdim"])):
                mat(R + s, n, C, 2.0)
                w[R + s + ".conv"] = rng.standard_normal((n, d["conv"])) / np.sqrt(d["conv"])
            mat(R + "a", d["heads"], C)
            mat(R + "b", d["heads"], C)
            w[R + "A_log"] = rng.uniform(-1.0, 1.0, d["heads"])
            w[R + "dt_bias"] = rng.uniform(-5.0, 0.0, d["heads"])
            mat(R + "g", d["heads"] * d["vdim"], C)
            around_one(R + "norm", d["vdim"])
            mat(R + "o", C, d["heads"] * d["vdim"])
            around_one(R + "out", C)
        if layer["mlp"]:
            norm(p + "norm2")
            ff = layer["mlp"]["ff"]
            mat(p + "mlp.gate", ff, C)
            mat(p + "mlp.up", ff, C)
            mat(p + "mlp.down", C, ff)
        if side:
            mat(p + "side.gate", side, C)
            mat(p + "side.proj", C, side)
            w[p + "side.norm"] = 0.5 + 0.2 * rng.standard_normal(C)
    norm("final.norm")
    mat("head", V, C)
    return {k: mixers.bf16(np.asarray(v, np.float32)) for k, v in w.items()}


def write(folder, cfg, w):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    mixers.write_safetensors(folder / "model.safetensors", w)
    return folder


def load(folder, compute, capacity=1024, lanes=4, slots=4, **kw):
    eng = importlib.import_module("macllm_infer_b200.engine")
    return eng.Model.load(folder, compute=compute, kv_dtype="f32" if compute == "float32" else "f16", kv_capacity_tokens=capacity,
                          max_batch_tokens=capacity, max_batch_lanes=lanes, state_slots=slots, **kw)


# Root mean square of the difference over that of the expected rows.
LIMIT = {"float32": 3e-5, "bfloat16": 4e-2}


def row_errors(got, want):
    return np.sqrt(np.mean((got - want) ** 2, axis=-1) / np.mean(want ** 2))


def assert_rows(got, want, compute, what=""):
    e = row_errors(got, want)
    assert e.max() <= LIMIT[compute], f"{what}: row {int(e.argmax())} of {len(e)} is off by {e.max():.2e}"


def cut(n, sizes):
    """Portions of the given sizes, over and over, until n tokens are used."""
    out, at, i = [], 0, 0
    while at < n:
        k = min(sizes[i % len(sizes)], n - at)
        out.append(k)
        at += k
        i += 1
    return out


def run_portions(model, tokens, portions):
    """Logits of every token, the sequence fed in portions."""
    s = model.new_session()
    rows, at = [], 0
    for k in portions:
        logits, _ = model.forward_batch([(s, tokens[at:at + k], at)], want_tokens=False, rows=[range(k)])
        rows.append(logits)
        at += k
    s.close()
    return np.concatenate(rows)
