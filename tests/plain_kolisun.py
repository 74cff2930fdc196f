"""A plain, slow Kolisun in PyTorch (64-bit unless asked otherwise): whole sequences, no cache, one
function per mechanism.

The oracle of the Kolisun tests.  It shares no code with the engine: it takes the configuration as the
dictionary ``config.json`` holds and the tensors by their stored names.

The residual stream starts as the token's embedding; a sublayer reads the stream as it is, and what it
returns is normalised before it is added.  Mixers: ``latent_attention`` (queries through a latent, keys
and values from a cached latent, a sink per head) and ``parallel`` (windowed grouped-query attention
beside a state-space recurrence, the two added with a factor each).  The feed-forward is gated by silu.
"""

from __future__ import annotations

import math

import torch


def rms(x, eps, w=None):
    y = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def base_frequencies(dims, base):
    return float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)


def by_wavelength(f, scaling):
    """Llama 3.1: short wavelengths keep their frequency, long ones have it divided, a blend between."""
    out = []
    for x in f.tolist():
        length = 2 * math.pi / x
        if length < scaling["original"] / scaling["high"]:
            out.append(x)
        elif length > scaling["original"] / scaling["low"]:
            out.append(x / scaling["factor"])
        else:
            s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1 - s) * x / scaling["factor"] + s * x)
    return torch.tensor(out, dtype=torch.float64)


def yarn(f, dims, base, scaling):
    """YaRN: (frequencies, what cos and sin are multiplied by)."""
    def turns_at(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turns_at(scaling["fast"])), 0)
    hi = min(math.ceil(turns_at(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f.tolist()):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / scaling["factor"] * ramp + x * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1


def turn(x, freqs, interleaved, amplitude=1.0):
    """x: [T, heads, dim]; the first ``2 * len(freqs)`` entries are turned by position times frequency."""
    half = freqs.shape[0]
    if half == 0:
        return x
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freqs
    c, s = (ang.cos() * amplitude).to(x.dtype)[:, None], (ang.sin() * amplitude).to(x.dtype)[:, None]
    y = x.clone()
    first, second = (slice(0, 2 * half, 2), slice(1, 2 * half, 2)) if interleaved else (slice(0, half), slice(half, 2 * half))
    u, v = x[..., first], x[..., second]
    y[..., first] = u * c - v * s
    y[..., second] = v * c + u * s
    return y


def softmax_attention(q, k, v, scale, window=None, sinks=None):
    """q, k: [T, heads, dim], v: [T, heads, vdim]; ``sinks``: one more term of the denominator per head."""
    T = q.shape[0]
    score = torch.einsum("ihd,jhd->hij", q, k) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) if window is None else (j <= i) & (i - j < window)
    score = score.masked_fill(~seen, -math.inf)
    top = score.amax(-1, keepdim=True)
    if sinks is not None:
        top = torch.maximum(top, sinks[:, None, None])
    p = torch.exp(score - top)
    below = p.sum(-1, keepdim=True)
    if sinks is not None:
        below = below + torch.exp(sinks[:, None, None] - top)
    return torch.einsum("hij,jhd->ihd", p / below, v)


def windowed_attention(h, w, name, m, eps):
    """Biased projections, norms over all query rows and all key rows at once, then heads and rotation."""
    T, H, G, D, DV = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[f"{name}.{x}"].T + w[f"{name}.{x}.b"] for x in "qkv")
    q, k = rms(q, eps, w[f"{name}.q.norm"]), rms(k, eps, w[f"{name}.k.norm"])
    rot = m.get("rot")
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, DV)
    if rot:
        f = base_frequencies(rot["dims"], rot["base"])
        if rot.get("scaling"):
            f = by_wavelength(f, rot["scaling"])
        q, k = turn(q, f, True), turn(k, f, True)
    group = torch.arange(H) // (H // G)
    window = m["mask"]["size"] if m.get("mask") else None
    o = softmax_attention(q, k[:, group], v[:, group], m["scale"], window)
    return o.reshape(T, H * DV) @ w[f"{name}.o"].T


def causal_conv(x, weight, bias):
    """x: [T, channels], weight: [channels, taps], the last tap weighs the token itself."""
    taps = weight.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return bias + sum(padded[t: t + x.shape[0]] * weight[:, t] for t in range(taps))


def ssd_recurrence(x, b, c, dt, decay, d):
    """x: [T, heads, vdim], b, c: [T, heads, state], dt, decay: [T, heads], d: [heads]."""
    S = x.new_zeros(x.shape[1], b.shape[2], x.shape[2])
    out = []
    for t in range(x.shape[0]):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, c[t]) + d[:, None] * x[t])
    return torch.stack(out)


def gated_group_norm(y, z, weight, groups, eps):
    """The gate first, then the norm over each of ``groups`` equal parts."""
    y = y * silu(z)
    T, size = y.shape
    return rms(y.view(T, groups, size // groups), eps).reshape(T, size) * weight


def state_space(h, w, name, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = (h @ w[f"{name}.in"].T).split([inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, w[f"{name}.conv"], w[f"{name}.conv.b"]))
    x, b, c = xbc.split([inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[f"{name}.dt_bias"])
    group = torch.arange(H) // (H // G)
    y = ssd_recurrence(x.view(T, H, P), b.view(T, G, N)[:, group], c.view(T, G, N)[:, group], dt,
                       torch.exp(-torch.exp(w[f"{name}.A_log"]) * dt), w[f"{name}.D"])
    y = gated_group_norm(y.reshape(T, inner), z, w[f"{name}.norm"], m["norm_groups"], eps)
    return y @ w[f"{name}.o"].T


def parallel(h, w, name, m, eps):
    return (m["left_scale"] * windowed_attention(h, w, f"{name}.left", m["left"], eps)
            + m["right_scale"] * state_space(h, w, f"{name}.right", m["right"], eps))


def latent_attention(h, w, name, m, eps):
    T, H, D, R, DV, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ w[f"{name}.dq"].T, eps, w[f"{name}.dq.norm"])
    q = (cq @ w[f"{name}.uq"].T).view(T, H, D + R)
    down = h @ w[f"{name}.dkv"].T
    c, key_part = rms(down[:, :K], eps, w[f"{name}.dkv.norm"]), down[:, None, K:]
    q_plain, q_turned = q[..., :D], q[..., D:]
    rot = m.get("rot")
    if rot and R:
        f, amplitude = base_frequencies(rot["dims"], rot["base"]), 1.0
        if rot.get("scaling"):
            f, amplitude = yarn(f, rot["dims"], rot["base"], rot["scaling"])
        q_turned, key_part = turn(q_turned, f, False, amplitude), turn(key_part, f, False, amplitude)
    k = torch.cat([(c @ w[f"{name}.uk"].T).view(T, H, D), key_part.expand(T, H, R)], dim=-1)
    v = (c @ w[f"{name}.uv"].T).view(T, H, DV)
    o = softmax_attention(torch.cat([q_plain, q_turned], dim=-1), k, v, m["scale"], sinks=w[f"{name}.sink"])
    return o.reshape(T, H * DV) @ w[f"{name}.o"].T


def dense(h, w, name):
    return (silu(h @ w[f"{name}.gate"].T) * (h @ w[f"{name}.up"].T)) @ w[f"{name}.down"].T


MIXERS = {"parallel": parallel, "latent_attention": latent_attention}


def run(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x, after = w["embed"][torch.tensor(tokens)], []
    for i, layer in enumerate(cfg["layers"]):
        x = x + rms(MIXERS[layer["type"]](x, w, f"l{i}.mix", layer["mixer"], eps), eps, w[f"l{i}.norm1"])
        if layer.get("mlp") is not None:
            x = x + rms(dense(x, w, f"l{i}.mlp"), eps, w[f"l{i}.norm2"])
        after.append(x)
    return rms(x, eps, w["final.norm"]) @ w["head"].T, torch.stack(after)


def logits_for(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64):
    return run(cfg, weights, tokens, dtype)[0]
