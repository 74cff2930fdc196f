"""Small Kolisun configurations and random weights for the tests.  Sizes are odd on purpose: head counts that are
not powers of two, one, several and as many key/value heads as heads, value sizes above and below the key
sizes, rotations of a part of a head, all of it and none, with every branch of both frequency scalings, windows of
one position, of a few and longer than the requests, groups and norm parts that do and do not follow the heads,
one to six taps, layers without a feed-forward, factors that are one and that are not."""

from __future__ import annotations

import torch


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def llama3(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def _rot(dims, base, scaling):
    out = {"dims": dims, "base": base}
    return out if scaling is None else {**out, "scaling": scaling}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale=None, base=10000.0, scaling=None):
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
           "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if rot_dim:
        out["rot"] = _rot(rot_dim, base, scaling)
    return "latent_attention", out


def attention(heads, kv_heads, dim, vdim, window, rot=None, base=10000.0, scaling=None, scale=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
           "mask": {"size": window}}
    if rot:
        out["rot"] = _rot(rot, base, scaling)
    return out


def recurrence(heads, vdim, state, groups=1, norm_groups=1, conv=4):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return "parallel", {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Kolisun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


# both kinds of layers in turn, both scalings, a window of a few pages, parts of the norm across heads
MIXED = config(72, 131, [
    (parallel(attention(6, 2, 12, 20, 9, rot=8, base=500.0, scaling=llama3(4.0, 1.0, 4.0, 64)),
              recurrence(6, 8, 12, groups=2, norm_groups=4, conv=4), 0.7, 1.3), dense(100)),
    (latent(3, 12, 8, 20, 24, 28, base=300.0, scaling=yarn(4.0, 32, 8.0, 1.0)), None),
    (latent(5, 8, 16, 8, 20, 12, scale=0.4), dense(56)),
    (parallel(attention(4, 4, 16, 8, 13), recurrence(4, 20, 8, groups=4, norm_groups=1, conv=2), 1.0, 1.0), None),
])
# nothing a multiple of four; a window of one position; one tap; no rotation in the latent
ODD = config(50, 61, [
    (latent(3, 7, 0, 9, 15, 11, scale=0.5), dense(30)),
    (parallel(attention(3, 1, 10, 7, 1, rot=10, base=40.0, scaling=llama3(8.0, 0.5, 2.0, 30)),
              recurrence(3, 7, 5, groups=1, norm_groups=7, conv=1), 1.4, 0.6), None),
    (latent(1, 5, 6, 3, 10, 9, base=100.0, scaling=yarn(10.0, 200, 60.0, 5.0)), dense(14)),
    (parallel(attention(5, 5, 6, 11, 10, rot=2), recurrence(2, 13, 33, groups=2, norm_groups=2, conv=6), 0.5, 2.0), dense(22)),
], eps=1e-4)
# the recurrence's layers alone (a window longer than every request; the sixth tap looks past short portions)
PARALLEL_ONLY = config(64, 97, [
    (parallel(attention(4, 2, 16, 16, 500, rot=16, base=2000.0), recurrence(8, 16, 24, groups=2, norm_groups=2, conv=3), 0.9, 1.1),
     dense(48)),
    (parallel(attention(2, 1, 32, 24, 7, rot=20, scaling=llama3(2.0, 1.5, 1.5, 100)),
              recurrence(5, 12, 16, norm_groups=5, conv=6), 1.2, 0.8), dense(40)),
])
# latent layers alone (no state slots)
LATENT_ONLY = config(48, 83, [
    (latent(4, 16, 16, 16, 32, 40, base=10000.0, scaling=yarn(16.0, 100, 20.0, 2.0)), dense(64)),
    (latent(2, 24, 8, 40, 16, 20, scale=0.25), None),
])
# sizes the bfloat16 tensor-core kernels take; prompts over several chunks, tiles and pages of 16
WIDE = config(128, 211, [
    (latent(6, 32, 32, 48, 96, 64, base=30000.0, scaling=yarn(6.0, 128, 16.0, 1.5)), dense(192)),
    (parallel(attention(8, 2, 48, 32, 70, rot=32, base=9000.0, scaling=llama3(6.0, 1.0, 3.0, 256)),
              recurrence(6, 64, 128, groups=2, norm_groups=3, conv=4), 0.8, 1.2), dense(160)),
    (latent(4, 48, 16, 32, 80, 56), None),
    (parallel(attention(4, 4, 32, 64, 200, rot=32), recurrence(4, 32, 48, groups=1, norm_groups=2, conv=3), 1.1, 0.7), dense(96)),
])

CONFIGS = {"mixed": MIXED, "odd": ODD, "parallel_only": PARALLEL_ONLY, "latent_only": LATENT_ONLY}
ALL_CONFIGS = dict(CONFIGS, wide=WIDE)


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    h = cfg["width"]
    shapes = {"embed": (cfg["vocab"], h), "head": (cfg["vocab"], h), "final.norm": (h,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        shapes[f"l{i}.norm1"] = (h,)
        if layer["type"] == "latent_attention":
            H, D, R, V, K, Q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            shapes.update({f"{p}.dq": (Q, h), f"{p}.dq.norm": (Q,), f"{p}.uq": (H * (D + R), Q), f"{p}.dkv": (K + R, h),
                           f"{p}.dkv.norm": (K,), f"{p}.uk": (H * D, K), f"{p}.uv": (H * V, K), f"{p}.sink": (H,),
                           f"{p}.o": (h, H * V)})
        else:
            a, r = m["left"], m["right"]
            q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            for n, size in (("q", q), ("k", k), ("v", v)):
                shapes.update({f"{p}.left.{n}": (size, h), f"{p}.left.{n}.b": (size,)})
            shapes.update({f"{p}.left.q.norm": (q,), f"{p}.left.k.norm": (k,), f"{p}.left.o": (h, a["heads"] * a["vdim"])})
            inner = r["heads"] * r["vdim"]
            channels = inner + 2 * r["groups"] * r["state"]
            shapes.update({f"{p}.right.in": (inner + channels + r["heads"], h), f"{p}.right.conv": (channels, r["conv"]),
                           f"{p}.right.conv.b": (channels,), f"{p}.right.norm": (inner,), f"{p}.right.o": (h, inner)})
            shapes.update({f"{p}.right.{n}": (r["heads"],) for n in ("dt_bias", "A_log", "D")})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            shapes.update({f"l{i}.norm2": (h,), f"l{i}.mlp.gate": (ff, h), f"l{i}.mlp.up": (ff, h), f"l{i}.mlp.down": (h, ff)})
    return shapes


def make_weights(cfg: dict, seed: int = 0) -> dict:
    """Random weights, stored as bfloat16 values.  Matrices are N(0, 1/sqrt(fan-in)).  Query and key norms and
    projections are scaled up so that attention is peaked (with flat attention a lost key moves the output by one
    part in dozens and hides in the tolerance); sinks are of the scores' size; the recurrence forgets
    slowly in some heads and fast in others; the convolutions weigh every tap."""
    g = torch.Generator().manual_seed(seed)
    uniform = lambda shape, lo, hi: lo + (hi - lo) * torch.rand(shape, generator=g)  # noqa: E731
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if name.endswith((".q.norm", ".k.norm")):
            t = uniform(shape, 1.0, 2.5)
        elif last in ("norm1", "norm2", "norm"):
            t = uniform(shape, 0.6, 1.6)
        elif last == "b":
            t = 0.4 * torch.randn(shape, generator=g)
        elif last == "sink":
            t = 1.5 * torch.randn(shape, generator=g)
        elif last == "A_log":
            t = uniform(shape, -3.0, 1.0)
        elif last == "dt_bias":
            t = uniform(shape, -3.0, 0.5)
        elif last == "D":
            t = uniform(shape, 0.3, 1.5)
        elif last == "conv":
            t = 0.4 * torch.randn(shape, generator=g) + 0.3
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if last in ("uq", "uk"):
                t = t * 1.6
        out[name] = t.to(torch.bfloat16)
    return out
