"""Throughput of mixer-built decoders (random weights, layers of real-model sizes) beside the closest GGUF family of the same
width, heads, feed-forward and layer count (looped layers counted once per pass): dense BF16 matrices, or, beside mixtures of experts,
the sparse family with its own quantised ones.  Used by `bench.py --mixer`.

Every figure is device time (CUDA events around the tick, median over the timed ticks); the weights of a tick are several
times the L2.  The per-class table comes from separate ticks with an event pair around every launch; `roofline` there is the
slower of bytes / measured copy bandwidth and flops / measured bf16 rate, over the time taken.
"""
from __future__ import annotations

import json
import tempfile
from dataclasses import dataclass
from pathlib import Path

import numpy as np

from . import _capi as capi
from . import engine
from . import seed_gguf


@dataclass
class Shape:
    name: str
    width: int
    pairs: int           # (time-mixing layer, parallel layer) pairs
    wkv_heads: int
    wkv_dim: int
    rank: int
    heads: int
    kv_heads: int
    dim: int
    delta_heads: int
    delta_kv: int
    delta_dim: int
    ff: int
    side: int
    vocab: int = 32000


SHAPES = [
    Shape("w2048", 2048, 4, 32, 64, 64, 16, 4, 128, 16, 8, 128, 8192, 256),
    Shape("w4096", 4096, 2, 64, 64, 64, 32, 8, 128, 32, 16, 128, 12288, 256),
]


@dataclass
class BesideShape:
    """Pairs of latent-attention and minGRU layers with the feed-forward beside the mixer; `loop` = (start, stop, times)."""
    name: str
    width: int
    pairs: int
    loop: tuple
    heads: int
    dim: int
    q_rank: int
    kv_rank: int
    gru: int
    ff: int
    kv_heads: int        # of the closest model
    vocab: int = 32000

    @property
    def runs(self) -> int:
        a, b, n = self.loop
        return 2 * self.pairs + (b - a) * (n - 1)


BESIDE_SHAPES = [
    BesideShape("w2048", 2048, 3, (2, 4, 2), 16, 128, 1024, 512, 2048, 8192, 4),
    BesideShape("w4096", 4096, 1, (0, 2, 2), 32, 128, 1536, 512, 4096, 12288, 8),
]


@dataclass
class ExpertShape:
    """Groups of four layers - capped attention, two of mLSTM, sink attention - over a mixture of experts."""
    name: str
    width: int
    groups: int
    heads: int           # of attention
    kv_heads: int
    dim: int
    chunk: int
    mem_heads: int       # of mLSTM
    mem_dim: int
    mem_vdim: int
    experts: int
    top: int
    ff: int
    vocab: int = 32000

    @property
    def runs(self) -> int:
        return 4 * self.groups


EXPERT_SHAPES = [
    ExpertShape("w2048", 2048, 1, 16, 4, 128, 8192, 8, 128, 256, 64, 8, 768),
    ExpertShape("w4096", 4096, 1, 32, 8, 128, 8192, 16, 128, 256, 16, 2, 2048),
]


@dataclass
class ConvShape:
    """Groups of four layers behind a short convolution: attention beside the delta rule with channel gates, twice, latent attention with
    a rotated part, and the first kind again."""
    name: str
    width: int
    groups: int
    heads: int
    kv_heads: int
    dim: int
    delta_heads: int
    delta_dim: int
    rank: int
    q_rank: int
    kv_rank: int
    rot_dim: int
    window: int
    ff: int
    vocab: int = 32000

    @property
    def runs(self) -> int:
        return 4 * self.groups


CONV_SHAPES = [
    ConvShape("w2048", 2048, 2, 16, 4, 128, 16, 128, 64, 1024, 512, 64, 8192, 8192),
    ConvShape("w4096", 4096, 1, 32, 8, 128, 32, 128, 64, 1536, 512, 64, 8192, 12288),
]


def conv_layers(s) -> list:
    mlp = {"kind": "dense", "ff": s.ff}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.dim, "scale": s.dim ** -0.5, "mask": {"size": s.window},
                 "rot": {"base": 500000.0, "dims": s.dim // 4}},
        "right": {"heads": s.delta_heads, "dim": s.delta_dim}, "left_scale": 0.7, "right_scale": 0.7}}
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": s.heads, "dim": s.dim, "vdim": s.dim, "q_rank": s.q_rank, "kv_rank": s.kv_rank, "rot_dim": s.rot_dim, "scale": (s.dim + s.rot_dim) ** -0.5,
        "mask": {"size": s.window}, "rot": {"base": 10000.0, "dims": s.rot_dim, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    return [par, par, lat, par] * s.groups


def expert_layers(s) -> list:
    mlp = {"kind": "moe", "router": {"experts": s.experts, "top": s.top}, "expert": {"ff": s.ff, "limit": 7.0}, "shared": {"ff": s.ff, "limit": 7.0}}
    attn = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.dim, "scale": s.dim ** -0.5, "mask": {"size": s.chunk}}
    sink = {"type": "attention", "mlp": mlp, "mixer": {**attn, "rot": {"base": 10000.0, "dims": s.dim}}}
    capped = {"type": "attention_2", "mlp": mlp, "mixer": {**attn, "softcap": 30.0, "rot": {
        "base": 500000.0, "dims": s.dim, "scaling": {"factor": 16.0, "original": 4096, "fast": 24.0, "slow": 1.5}}}}
    mem = {"type": "mlstm", "mlp": mlp, "mixer": {"heads": s.mem_heads, "dim": s.mem_dim, "vdim": s.mem_vdim, "gate_cap": 12.0}}
    return [capped, mem, mem, sink] * s.groups


def config_of(s) -> dict:
    if isinstance(s, ConvShape):
        return {"architecture": "Mamivik", "vocab": s.vocab, "width": s.width, "norm": {"eps": 1e-6}, "canon": {"taps": 4}, "layers": conv_layers(s)}
    if isinstance(s, ExpertShape):
        return {"architecture": "Tevanex", "vocab": s.vocab, "width": s.width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "residual_mult": 0.5,
                "logit_scale": 1.0, "logit_softcap": 30.0, "layers": expert_layers(s)}
    if isinstance(s, BesideShape):
        mlp = {"kind": "dense", "ff": s.ff}
        lat = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": s.heads, "dim": s.dim, "vdim": s.dim, "q_rank": s.q_rank, "kv_rank": s.kv_rank,
                                                                 "scale": s.dim ** -0.5}}
        gru = {"type": "mingru", "mlp": mlp, "mixer": {"width": s.gru}}
        return {"architecture": "Kunonex", "vocab": s.vocab, "width": s.width, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
                "loop": dict(zip(("start", "stop", "times"), s.loop)), "layers": [lat, gru] * s.pairs}
    mlp = {"kind": "dense", "ff": s.ff}
    wkv = {"type": "wkv", "mixer": {"heads": s.wkv_heads, "dim": s.wkv_dim}, "mlp": mlp}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.dim, "scale": s.dim ** -0.5,
                 "rot": {"base": 500000.0, "dims": s.dim, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}},
        "right": {"heads": s.delta_heads, "kv_heads": s.delta_kv, "dim": s.delta_dim, "vdim": s.delta_dim, "conv": 4}}}
    return {"architecture": "Sizilorn", "vocab": s.vocab, "width": s.width, "norm": {"eps": 1e-6}, "token_side": {"dim": s.side},
            "layers": [wkv, par] * s.pairs}


def tensor_shapes(s) -> dict[str, tuple]:
    """name -> (shape, mean, deviation)."""
    C, V, out = s.width, s.vocab, {}
    beside = isinstance(s, BesideShape)

    def mat(name, rows, cols):
        out[name] = ((rows, cols), 0.0, cols ** -0.5)

    def vec(name, *shape, mean=1.0, dev=0.1):
        out[name] = (shape, mean, dev)

    def norm(name):
        vec(name, C)
        if not beside:
            vec(name + ".b", C, mean=0.0)
            vec(name + ".alpha", mean=0.7, dev=0.0)

    out["embed"] = ((V, C), 0.0, 1.0)
    if isinstance(s, ConvShape):
        for i, layer in enumerate(conv_layers(s)):
            p, m = f"l{i}.", layer["mixer"]
            vec(p + "norm1")
            vec(p + "norm2")
            out[p + "canon1"] = ((C, 4), 0.0, 0.3)
            if layer["type"] == "parallel":
                L, R, n = p + "mix.left.", p + "mix.right.", s.delta_heads * s.delta_dim
                for x, rows in (("q", s.heads * s.dim), ("k", s.kv_heads * s.dim)):
                    mat(L + x, rows, C)
                    vec(L + x + ".b", rows, mean=0.0)
                mat(L + "o", C, s.heads * s.dim)
                for x in "rkvga":
                    mat(R + x, n, C)
                vec(R + "a.b", n, mean=0.0)
                mat(R + "w1", s.rank, C)
                mat(R + "w2", n, s.rank)
                vec(R + "w0", n, mean=-3.0, dev=1.0)
                vec(R + "norm", n)
                mat(R + "o", C, n)
            else:
                n = s.heads * s.dim
                mat(p + "mix.dq", s.q_rank, C)
                vec(p + "mix.dq.norm", s.q_rank)
                mat(p + "mix.uq", n + s.heads * s.rot_dim, s.q_rank)
                mat(p + "mix.dkv", s.kv_rank + s.rot_dim, C)
                vec(p + "mix.dkv.norm", s.kv_rank)
                mat(p + "mix.uk", n, s.kv_rank)
                mat(p + "mix.uv", n, s.kv_rank)
                vec(p + "mix.sink", s.heads)
                mat(p + "mix.g", n, C)
                mat(p + "mix.o", C, n)
            mat(p + "mlp.gate", s.ff, C)
            mat(p + "mlp.up", s.ff, C)
            mat(p + "mlp.down", C, s.ff)
        vec("final.norm")
        mat("head", V, C)
        return out
    if isinstance(s, ExpertShape):
        for i, layer in enumerate(expert_layers(s)):
            p, m = f"l{i}.", layer["mixer"]
            vec(p + "norm1", C)
            vec(p + "norm2", C)
            qw, vw = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            G = m.get("kv_heads", m["heads"])
            mat(p + "mix.q", qw, C)
            mat(p + "mix.k", G * m["dim"], C)
            mat(p + "mix.v", G * m["vdim"], C)
            mat(p + "mix.o", C, vw)
            if layer["type"] != "attention":
                mat(p + "mix.g", vw, C)
            if layer["type"] == "mlstm":
                vec(p + "mix.norm", vw)
                for x, mean in (("i", -1.0), ("f", 4.0)):
                    mat(p + "mix." + x, m["heads"], C)
                    vec(p + f"mix.{x}.b", m["heads"], mean=mean)
            else:
                for x, n in (("q", qw), ("k", G * m["dim"]), ("v", G * m["vdim"]), ("o", C)):
                    vec(p + f"mix.{x}.b", n, mean=0.0)
                vec(p + "mix.q.norm", qw)
                vec(p + "mix.k.norm", G * m["dim"])
            if layer["type"] == "attention":
                vec(p + "mix.sink", m["heads"])
            for name in [f"e{e}" for e in range(s.experts)] + ["shared"]:
                mat(p + f"mlp.{name}.gate", s.ff, C)
                mat(p + f"mlp.{name}.up", s.ff, C)
                mat(p + f"mlp.{name}.down", C, s.ff)
            mat(p + "mlp.router", s.experts, C)
            mat(p + "mlp.shared.sg", 1, C)
        vec("final.norm", C)
        mat("head", V, C)
        return out
    if beside:
        norm("embed.norm")
        mat("loop.in", C, 2 * C)
        vec("loop.step", s.loop[2], C, mean=0.0)
        for i in range(2 * s.pairs):
            p = f"l{i}."
            norm(p + "norm1")
            vec(p + "shift", C, mean=0.5)
            if i % 2 == 0:
                n = s.heads * s.dim
                mat(p + "mix.dq", s.q_rank, C)
                vec(p + "mix.dq.norm", s.q_rank)
                mat(p + "mix.uq", n, s.q_rank)
                mat(p + "mix.dkv", s.kv_rank, C)
                vec(p + "mix.dkv.norm", s.kv_rank)
                mat(p + "mix.uk", n, s.kv_rank)
                mat(p + "mix.uv", n, s.kv_rank)
                mat(p + "mix.g", s.heads, C)
                mat(p + "mix.o", C, n)
            else:
                for x in "zxg":
                    mat(p + "mix." + x, s.gru, C)
                vec(p + "mix.z.b", s.gru, mean=-2.0, dev=1.0)
                vec(p + "mix.x.b", s.gru, mean=0.0)
                mat(p + "mix.o", C, s.gru)
            mat(p + "mlp.up", s.ff, C)
            vec(p + "mlp.up.b", s.ff, mean=0.0)
            mat(p + "mlp.down", C, s.ff)
            vec(p + "mlp.down.b", C, mean=0.0)
            vec(p + "mlp.act", 4, mean=0.5)
        norm("final.norm")
        mat("head", V, C)
        return out
    out["side.embed"] = ((V, 2 * s.pairs * s.side), 0.0, 1.0)
    for i in range(2 * s.pairs):
        p = f"l{i}."
        norm(p + "norm1")
        if i % 2 == 0:
            n = s.wkv_heads * s.wkv_dim
            for x in "rkvgw":
                vec(p + "mix.mu." + x, C, mean=0.5)
            for x in "rkvg":
                mat(p + "mix." + x, n, C)
            mat(p + "mix.w1", s.rank, C)
            mat(p + "mix.w2", n, s.rank)
            vec(p + "mix.w0", n, mean=-3.0, dev=1.0)
            vec(p + "mix.u", s.wkv_heads, s.wkv_dim, mean=0.0, dev=1.0)
            vec(p + "mix.norm", n)
            mat(p + "mix.o", C, n)
        else:
            L, R = p + "mix.left.", p + "mix.right."
            mat(L + "q", s.heads * s.dim, C)
            mat(L + "k", s.kv_heads * s.dim, C)
            mat(L + "v", s.kv_heads * s.dim, C)
            mat(L + "g", s.heads, C)
            vec(L + "q.norm", s.dim)
            vec(L + "k.norm", s.dim)
            mat(L + "o", C, s.heads * s.dim)
            vec(L + "out", C)
            for x, n in (("q", s.delta_kv), ("k", s.delta_kv), ("v", s.delta_heads)):
                mat(R + x, n * s.delta_dim, C)
                out[R + x + ".conv"] = ((n * s.delta_dim, 4), 0.0, 0.5)
            for x in "ab":
                mat(R + x, s.delta_heads, C)
            vec(R + "A_log", s.delta_heads, mean=0.0)
            vec(R + "dt_bias", s.delta_heads, mean=-3.0)
            mat(R + "g", s.delta_heads * s.delta_dim, C)
            vec(R + "norm", s.delta_dim)
            mat(R + "o", C, s.delta_heads * s.delta_dim)
            vec(R + "out", C)
        norm(p + "norm2")
        mat(p + "mlp.gate", s.ff, C)
        mat(p + "mlp.up", s.ff, C)
        mat(p + "mlp.down", C, s.ff)
        mat(p + "side.gate", s.side, C)
        mat(p + "side.proj", C, s.side)
        vec(p + "side.norm", C)
    norm("final.norm")
    mat("head", V, C)
    return out


def write_checkpoint(folder: Path, s) -> Path:
    """A random checkpoint; big matrices repeat one block of random numbers."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config_of(s)))
    base = np.random.default_rng(0).standard_normal((1 << 20) + 7).astype(np.float32)
    plan, head, at = tensor_shapes(s), {}, 0
    for name, (shape, _, _) in plan.items():
        n = 2 * int(np.prod(shape))
        head[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + n]}
        at += n
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for shape, mean, dev in plan.values():
            n = int(np.prod(shape))
            bits = ((base[:min(n, len(base))] * np.float32(dev) + np.float32(mean)).view(np.uint32) >> 16).astype(np.uint16)
            f.write(np.resize(bits, n).tobytes())
    return folder


def closest_spec(s) -> seed_gguf.SeedSpec:
    if isinstance(s, ExpertShape):
        return seed_gguf.SeedSpec("qwen3moe", s.runs, s.width, s.heads, s.kv_heads, s.dim, 4 * s.ff, s.vocab, context=16384, theta=1e6, eps=1e-6, experts=s.experts,
                                  experts_used=s.top, expert_ffn=s.ff, name=f"closest-{s.name}")
    layers = s.runs if isinstance(s, (BesideShape, ConvShape)) else 2 * s.pairs
    return seed_gguf.SeedSpec("qwen3", layers, s.width, s.heads, s.kv_heads, s.dim, s.ff, s.vocab, context=16384, theta=1e6, eps=1e-6,
                              matrix_type=capi.TYPE_BF16, high_type=capi.TYPE_BF16, name=f"closest-{s.name}")


def timed(model, lanes_of, warmup: int, steps: int) -> float:
    """Median device ms of `steps` ticks after `warmup`; lanes_of(i) gives tick i's lanes."""
    ms = []
    for i in range(warmup + steps):
        model.forward_batch(lanes_of(i), want_logits=False)
        if i >= warmup:
            ms.append(model.last_forward_ms())
    return float(np.median(ms))


def classes(model, peaks: dict) -> list[dict]:
    out = []
    for k in model.profile_query():
        sec = k["ms"] / 1e3
        ideal = max(k["bytes"] / (peaks["hbm_gbs"] * 1e9), k["flops"] / (peaks["tflops"] * 1e12))
        out.append(dict(kernel=k["name"], launches=int(k["launches"]), us_per_launch=round(1e3 * k["ms"] / k["launches"], 2),
                        gbs=round(k["bytes"] / sec / 1e9, 1), tflops=round(k["flops"] / sec / 1e12, 2), roofline=round(ideal / sec, 3),
                        ms=round(k["ms"], 3)))
    return sorted(out, key=lambda c: -c["ms"])


def measure(model, vocab: int, prompt: int, lanes: int, context: int, warmup: int, steps: int, peaks: dict) -> dict:
    rng = np.random.default_rng(1)
    out = {}

    def prefill(_):
        session.clear()
        return [(session, toks, 0)]

    session = model.new_session()
    toks = rng.integers(0, vocab, prompt).astype(np.uint32)
    ms = timed(model, prefill, warmup, steps)
    out["prefill"] = dict(tokens=prompt, ms=round(ms, 3), tokens_per_s=round(prompt / ms * 1e3))
    model.profile_enable(True)
    for i in range(2):
        model.forward_batch(prefill(i), want_logits=False)
    out["prefill"]["classes"] = classes(model, peaks)
    model.profile_enable(False)
    session.close()

    sessions = [model.new_session() for _ in range(lanes)]
    for i in range(0, lanes, 2):
        model.forward_batch([(s, rng.integers(0, vocab, context).astype(np.uint32), 0) for s in sessions[i:i + 2]], want_logits=False)
    one = rng.integers(0, vocab, lanes).astype(np.uint32)

    def decode(_):
        return [(s, one[i:i + 1], len(s)) for i, s in enumerate(sessions)]

    ms = timed(model, decode, warmup, steps)
    out["decode"] = dict(lanes=lanes, context=context, ms=round(ms, 3), tokens_per_s=round(lanes / ms * 1e3))
    model.profile_enable(True)
    for i in range(3):
        model.forward_batch(decode(i), want_logits=False)
    out["decode"]["classes"] = classes(model, peaks)
    model.profile_enable(False)
    for s in sessions:
        s.close()
    return out


DESIGNS = {"sizilorn": ("Sizilorn", SHAPES), "kunonex": ("Kunonex", BESIDE_SHAPES), "tevanex": ("Tevanex", EXPERT_SHAPES), "mamivik": ("Mamivik", CONV_SHAPES)}


def run(peaks: dict, warmup: int, steps: int, design="sizilorn", prompt=2048, lanes=64, context=1024) -> list[dict]:
    title, shapes = DESIGNS[design]
    results = []
    capacity = lanes * (context + 256)
    with tempfile.TemporaryDirectory() as tmp:
        for s in shapes:
            kw = dict(kv_capacity_tokens=capacity, max_batch_tokens=max(prompt, 2 * context), max_batch_lanes=lanes)
            for kind in (design, "closest"):
                if kind == design:
                    path = write_checkpoint(Path(tmp) / s.name, s)
                    model = engine.Model.load(path, state_slots=lanes + 1, **kw)
                    weights = model.spec().weight_bytes_per_token
                else:
                    path = seed_gguf.write_seed_gguf(Path(tmp) / f"{s.name}.gguf", closest_spec(s), seed=0)
                    model = engine.Model.load(path, **kw)
                    weights = seed_gguf.weight_bytes(closest_spec(s))["per_token"]
                r = measure(model, s.vocab, prompt, lanes, context, warmup, steps, peaks)
                sp = model.spec()
                results.append(dict(shape=s.name, model=title if kind == design else ("qwen3moe family, Q4_K / Q6_K matrices" if isinstance(s, ExpertShape) else "qwen3 family, dense BF16 matrices"), layers=int(sp.n_layers),
                                    width=int(sp.hidden_size), weight_gb=round(weights / 1e9, 3), **r))
                model.close()
    return results
