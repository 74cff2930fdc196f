"""Small Livitar configurations and random weights for the tests.  Sizes are odd on purpose: head counts
that are not powers of two, one, several and as many key/value heads as heads, value sizes above and
below the key sizes, rotations of a part of a head, all of it and none, decays of 1 and of almost
nothing, one to five residual streams, few and many distance buckets with the last one reached early,
late or never, queries that warm up every position and hardly ever, experts of which one, some or all
are used, shared experts and none, layers without a feed-forward."""

from __future__ import annotations

import torch


def retention(heads, dim, vdim, decay, rot=None, base=10000.0):
    out = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        out["rot"] = {"dims": rot, "base": base}
    return "retention", out


def attention(heads, kv_heads, dim, vdim, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                         "scale": dim ** -0.5 if scale is None else scale}


def attention_2(heads, kv_heads, dim, vdim, bias_max, q_temp=None, scale=None, buckets=16):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "bias_buckets": buckets,
           "scale": dim ** -0.5 if scale is None else scale}
    if q_temp:
        out["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return "attention_2", out


def moe(experts, top, ff, shared=None, scale=1.0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(width, vocab, layers, *, streams, eps=1e-5):
    return {"architecture": "Livitar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


def without_bucket_counts(cfg: dict) -> dict:
    """The configuration as a model folder may hold it: the number of distance buckets is the shape of a
    tensor and need not be written down."""
    return dict(cfg, layers=[dict(layer, mixer={k: v for k, v in layer["mixer"].items() if k != "bias_buckets"})
                             for layer in cfg["layers"]])


# every kind of mixer; streams read and mixed differently; grouped and single key/value heads
MIXED = config(72, 131, [
    (retention(3, 16, 8, (0.9, 0.99, 0.5), rot=8, base=500.0), moe(8, 2, 24, shared=40, scale=1.5)),
    (attention(6, 2, 16, 24), moe(5, 1, 16, shared=16)),
    (attention_2(4, 1, 12, 20, 40, q_temp=(0.7, 8), scale=0.45), None),
    (retention(2, 20, 36, (1.0, 0.97), rot=20), moe(6, 6, 20)),
    (attention_2(2, 2, 8, 8, 9, scale=0.6, buckets=6), moe(4, 3, 12, shared=8, scale=2.5)),
], streams=3)
# nothing a multiple of four; one stream; the state forgets almost at once in one head; no rotation
ODD = config(50, 61, [
    (attention_2(5, 5, 6, 7, 17.5, q_temp=(0.3, 1), scale=0.9, buckets=2), moe(7, 7, 9, shared=11)),
    (retention(5, 6, 10, (0.05, 0.7, 0.95, 0.999, 0.9)), None),
    (attention(3, 1, 10, 6, scale=0.4), moe(4, 2, 14, scale=0.5)),
], streams=1, eps=1e-4)
# five streams, retention first and last, a bias that reaches its last bucket after few positions and
# one that never does
STREAMS = config(64, 97, [
    (retention(4, 8, 8, (0.8, 0.9, 0.96, 0.99), rot=4, base=77.0), moe(4, 2, 20, shared=12, scale=2.2)),
    (attention_2(4, 4, 16, 8, 5, q_temp=(0.5, 16), scale=0.4, buckets=8), moe(3, 1, 12)),
    (attention_2(2, 1, 8, 16, 5000, q_temp=(1.0, 300), scale=0.6, buckets=32), None),
    (attention(4, 2, 8, 8), None),
    (retention(1, 33, 17, (0.98,), rot=32), moe(2, 1, 18, shared=6)),
], streams=5)
# a single bucket for every distance; two streams
ONE_BUCKET = config(48, 83, [
    (attention_2(2, 1, 24, 12, 3, scale=1.0, buckets=1), moe(6, 2, 10, shared=20, scale=3.0)),
    (attention(3, 3, 16, 4), moe(2, 2, 18)),
], streams=2)
# sizes the bfloat16 tensor-core kernels take; prompts over several chunks, tiles and pages of 16
WIDE = config(128, 211, [
    (retention(4, 64, 48, (0.9, 0.99, 0.995, 0.97), rot=32), moe(8, 2, 64, shared=96, scale=2.0)),
    (attention(8, 2, 64, 32), moe(8, 3, 32)),
    (attention_2(6, 3, 32, 128, 150, q_temp=(0.4, 64), scale=0.3, buckets=24), None),
    (retention(2, 128, 128, (0.98, 0.999), rot=128, base=2e5), moe(4, 1, 48, shared=32)),
    (attention_2(4, 1, 48, 48, 3000, scale=0.25, buckets=32), moe(4, 2, 32, shared=64)),
], streams=4)

CONFIGS = {"mixed": MIXED, "odd": ODD, "streams": STREAMS, "one_bucket": ONE_BUCKET}
ALL_CONFIGS = dict(CONFIGS, wide=WIDE)


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    h, s = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], h), "head": (cfg["vocab"], h)}

    def norm(name):
        shapes.update({name: (h,), name + ".b": (h,), name + ".alpha": ()})

    def mixing(name):
        shapes.update({name + ".in": (s,), name + ".mix": (s, s), name + ".out": (s,)})

    def gated(name, ff):
        shapes.update({name + ".gate": (ff, h), name + ".up": (ff, h), name + ".down": (h, ff)})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        q, v_out = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        norm(p + ".norm1")
        mixing(p + ".hc1")
        kv = m["heads"] if layer["type"] == "retention" else m["kv_heads"]
        shapes.update({f"{p}.mix.q": (q, h), f"{p}.mix.k": (kv * m["dim"], h), f"{p}.mix.v": (kv * m["vdim"], h),
                       f"{p}.mix.g": (v_out, h), f"{p}.mix.o": (h, v_out)})
        if layer["type"] == "attention":
            shapes.update({f"{p}.mix.{n}": (m["heads"],) for n in ("temp", "r1", "r2")})
        elif layer["type"] == "attention_2":
            shapes[f"{p}.mix.rel"] = (m["bias_buckets"], m["heads"])
        mlp = layer["mlp"]
        if mlp is None:
            continue
        norm(p + ".norm2")
        mixing(p + ".hc2")
        shapes[p + ".mlp.router"] = (mlp["router"]["experts"], h)
        for e in range(mlp["router"]["experts"]):
            gated(f"{p}.mlp.e{e}", mlp["expert"]["ff"])
        if mlp.get("shared"):
            gated(p + ".mlp.shared", mlp["shared"]["ff"])
    return shapes


def make_weights(cfg: dict, seed: int = 0) -> dict:
    """Random weights, stored as bfloat16 values.  Matrices are N(0, 1/sqrt(fan-in)).  Query and key
    projections are scaled up so that attention is peaked (with flat attention a lost key moves the
    output by one part in dozens and hides in the tolerance); the biases by distance are of the scores'
    size and differ from bucket to bucket; the streams' coefficients differ from stream to stream and
    the mixing is not symmetric; alphas bend the tanh without saturating it; routers are spread so that
    the choice of experts is not a close call."""
    g = torch.Generator().manual_seed(seed)
    uniform = lambda shape, lo, hi: lo + (hi - lo) * torch.rand(shape, generator=g)  # noqa: E731
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = uniform(shape, 0.6, 1.8)
        elif last == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        elif last == "alpha":
            t = uniform(shape, 0.4, 0.9)
        elif last in ("in", "out"):
            t = uniform(shape, 0.2, 1.1)
        elif ".hc" in name and last == "mix":
            t = 0.8 * torch.eye(shape[0]) + 0.2 * torch.randn(shape, generator=g)
        elif last == "temp":
            t = uniform(shape, 0.5, 2.0)
        elif last == "r1":
            t = uniform(shape, 0.1, 2.5)
        elif last == "r2":
            t = uniform(shape, 0.05, 0.6)
        elif last == "rel":
            t = 1.5 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if name.endswith(("mix.q", "mix.k")):
                t = t * 1.5
            if name.endswith("mlp.router"):
                t = t * 4.0
        out[name] = t.to(torch.bfloat16)
    return out
