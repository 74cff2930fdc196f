"""A plain, slow Livitar in PyTorch (64-bit unless asked otherwise): whole sequences, no cache, one
function per mechanism.

The oracle of the Livitar tests.  It shares no code with the engine: it takes the configuration as
the dictionary ``config.json`` holds and the tensors by their stored names.

The model keeps ``streams`` residual streams, all equal to the token's embedding at the start.  A
sublayer reads a weighted sum of them through a norm ``tanh(alpha x) w + b``; afterwards every stream
becomes a weighted sum of the old ones plus its own multiple of the sublayer's output.  Mixers:
``retention`` (a matrix state per head with a fixed decay), ``attention`` (a temperature per head and a
penalty that grows with the logarithm of the distance) and ``attention_2`` (unit-RMS queries and keys,
queries warmed up by position, a learned bias per bucket of distances).  The feed-forward is a mixture
of gated experts beside a shared one.
"""

from __future__ import annotations

import math

import torch


def dynamic_tanh(x, w, name):
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def read_streams(xs, coef):
    """xs: [S, T, width] -> what a sublayer reads, [T, width]."""
    return sum(coef[s] * xs[s] for s in range(xs.shape[0]))


def write_streams(xs, y, mix, out):
    """Every new stream from the old ones (``mix[from, to]``) and the sublayer's output."""
    S = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(S)) + out[t] * y for t in range(S)])


def rotate_half(x, dims, base):
    """x: [T, heads, dim]: the pairs (i, i + dims / 2) are turned by position * base^(-2i / dims)."""
    if not dims:
        return x
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    cos, sin = ang.cos()[:, None, :].to(x.dtype), ang.sin()[:, None, :].to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def retention_core(q, k, v, decay, state=None):
    """q, k: [T, H, d], v: [T, H, dv], decay: [H] -> ([T, H, dv], the state [H, d, dv] afterwards), token
    by token."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def mixer_retention(w, p, h, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {}
    q = rotate_half((h @ w[p + ".q"].T).view(T, H, d), rot.get("dims", 0), rot.get("base", 1.0))
    k = rotate_half((h @ w[p + ".k"].T).view(T, H, d), rot.get("dims", 0), rot.get("base", 1.0)) * d ** -0.5
    v = (h @ w[p + ".v"].T).view(T, H, dv)
    o, _ = retention_core(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    o = unit_rms(o, eps).reshape(T, H * dv)
    return (o * torch.nn.functional.silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def log_distance_bias(dist, r1, r2):
    """What is added to a score at distance ``dist`` (a tensor of any shape), for one head."""
    return -r1 * torch.log(1.0 + r2 * dist)


def bucket(n: int, buckets: int, bias_max: float) -> int:
    half = buckets / 2
    if n < half:
        return n
    return int(min(buckets - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (buckets - half))))


def bucket_bias(dist, rel, bias_max, h):
    """The learned bias of every distance, for head ``h``."""
    of = torch.tensor([bucket(n, rel.shape[0], bias_max) for n in range(int(dist.max()) + 1)])
    return rel[of[dist.clamp(min=0)], h]


def query_warmth(positions, coef, every):
    """The factor of the queries at each position."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in positions], dtype=torch.float64)


def attention_core(q, k, v, scale, bias):
    """q: [T, H, d], k: [T, G, d], v: [T, G, dv]; ``scale``: a number or one per head; ``bias(h)``: [T, T]
    added to the scores (or None) -> [T, H, dv]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * (scale[h] if torch.is_tensor(scale) else scale)
        if bias is not None:
            s = s + bias(h)
        out[:, h] = torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1) @ v[:, h // rep]
    return out


def distances(T):
    return (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)


def _project(w, p, h, m):
    T, H, G = h.shape[0], m["heads"], m.get("kv_heads") or m["heads"]
    return ((h @ w[p + ".q"].T).view(T, H, m["dim"]), (h @ w[p + ".k"].T).view(T, G, m["dim"]),
            (h @ w[p + ".v"].T).view(T, G, m["vdim"]))


def _gated_output(w, p, h, o):
    return (o.reshape(h.shape[0], -1) * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def mixer_attention(w, p, h, m):
    q, k, v = _project(w, p, h, m)
    dist = distances(h.shape[0]).to(h.dtype)
    o = attention_core(q, k, v, m["scale"] * w[p + ".temp"],
                       lambda i: log_distance_bias(dist, w[p + ".r1"][i], w[p + ".r2"][i]))
    return _gated_output(w, p, h, o)


def mixer_attention_2(w, p, h, m, eps):
    q, k, v = _project(w, p, h, m)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    if m.get("q_temp"):
        q = q * query_warmth(range(h.shape[0]), m["q_temp"]["coef"], m["q_temp"]["every"]).to(h.dtype)[:, None, None]
    dist = distances(h.shape[0])
    o = attention_core(q, k, v, m["scale"], lambda i: bucket_bias(dist, w[p + ".rel"], m["bias_max"], i))
    return _gated_output(w, p, h, o)


def gated(w, p, h):
    return (torch.nn.functional.silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(w, p, h, router, margins=None):
    """(ids [T, top], weights [T, top]).  ``margins``: a list that receives, per token, how far the last
    chosen expert's logit is above the best one that was not chosen."""
    z = h @ w[p + ".router"].T
    s = torch.softmax(z, dim=-1)
    ids = s.topk(router["top"], dim=-1).indices
    if margins is not None and router["top"] < router["experts"]:
        ranked = z.sort(-1, descending=True).values
        margins.extend((ranked[:, router["top"] - 1] - ranked[:, router["top"]]).tolist())
    picked = s.gather(1, ids)
    return ids, picked / (picked.sum(-1, keepdim=True) + 1e-20) * router.get("scale", 1.0)


def feed_forward_moe(w, p, h, mlp, margins=None):
    ids, weights = route(w, p, h, mlp["router"], margins)
    out = gated(w, p + ".shared", h) if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        share = (weights * (ids == e)).sum(-1)
        rows = share.nonzero().flatten()
        if len(rows):
            out[rows] = out[rows] + share[rows, None] * gated(w, f"{p}.e{e}", h[rows])
    return out


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False, margins=None):
    """Logits [T, vocab] of a whole sequence (and the sum of the streams after every layer)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    xs = torch.stack([w["embed"][tokens]] * cfg["streams"])
    seen = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = dynamic_tanh(read_streams(xs, w[p + ".hc1.in"]), w, p + ".norm1")
        if layer["type"] == "retention":
            y = mixer_retention(w, p + ".mix", h, m, eps)
        elif layer["type"] == "attention":
            y = mixer_attention(w, p + ".mix", h, m)
        else:
            y = mixer_attention_2(w, p + ".mix", h, m, eps)
        xs = write_streams(xs, y, w[p + ".hc1.mix"], w[p + ".hc1.out"])
        if layer.get("mlp") is not None:
            h = dynamic_tanh(read_streams(xs, w[p + ".hc2.in"]), w, p + ".norm2")
            y = feed_forward_moe(w, p + ".mlp", h, layer["mlp"], margins)
            xs = write_streams(xs, y, w[p + ".hc2.mix"], w[p + ".hc2.out"])
        seen.append(xs.sum(0))
    logits = dynamic_tanh(xs.sum(0), w, "final.norm") @ w["head"].T
    return (logits, torch.stack(seen)) if return_layers else logits
