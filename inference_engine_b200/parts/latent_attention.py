"""Attention over a shared low-rank latent: every token caches one latent vector and one rotated
key part, from which all heads' keys and values follow.

Per token, with ``h`` the mixer's input: ``q = W_q h`` is laid out head by head as ``dim``
unrotated then ``rot_dim`` rotated entries.  ``W_dkv h`` has ``kv_rank + rot_dim`` rows: the first
``kv_rank``, divided by their root mean square (eps inside the root) and multiplied by a weight,
are the latent ``c``; the rest is one key part shared by all heads.  The rotated query and key
parts are turned by the position's angles (pairs ``2i, 2i+1`` or ``i, i + rot.dims/2``, as the encoding says; the
first ``rot.dims`` entries of the part, the rest pass).  Head ``n``'s key is ``[W_uk[n] c, rotated part]``, its value
``W_uv[n] c``; scores are scaled by ``scale``, masked causally and soft-maxed; each head's output
is multiplied by ``sigmoid(W_g h)[n]``, and ``W_o`` maps the concatenated heads back.

Variants by the tensors named.  ``dq``, ``dq_norm`` and ``uq`` in place of ``q``: the queries go through a latent of
their own, ``q = W_uq (c_q)`` with ``c_q = W_dq h`` divided by its root mean square and multiplied by a weight.
No ``gate``: the heads' outputs are not gated.  ``sink``: the softmax's denominator holds one more term ``exp(sink[n])``
per head, which has no key and no value and is not scaled.

Only ``c`` and the rotated key part are cached (one row of ``kv_rank + rot_dim`` numbers per
token and layer, shared by the heads).  The products with ``W_uk`` and ``W_uv`` are moved to the
query side: ``q_unrotated[n] . (W_uk[n] c) = (W_uk[n]^T q_unrotated[n]) . c``, and
``sum_j p_j W_uv[n] c_j = W_uv[n] sum_j p_j c_j``.  So the attention runs with one shared
key/value head whose key rows are the cached rows and whose value rows are their first
``kv_rank`` entries, in prompts and in decoding alike, and nothing is expanded per cached token.
"""

from __future__ import annotations

from .base import BuildEnv, CacheBinding, Mixer, PagedKVRequest, WeightDecl
from .registry import register_part


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    def __init__(self, *, names: dict, hidden_size: int, heads: int, dim: int, rot_dim: int, vdim: int,
                 kv_rank: int, scale: float, eps: float, position, dtype, q_rank: int | None = None) -> None:
        self.hidden_size, self.heads = hidden_size, heads
        self.dim, self.rot_dim, self.vdim, self.kv_rank = dim, rot_dim, vdim, kv_rank
        self.scale, self.eps, self.position, self.dtype = float(scale), float(eps), position, dtype
        self.names = {k: v for k, v in names.items() if v}
        self.q_rank = None if q_rank is None else int(q_rank)
        low_rank = ("dq", "dq_norm", "uq")
        wanted = ("q",) if self.q_rank is None else low_rank
        if any(k not in self.names for k in wanted) or any(k in self.names for k in ("q", *low_rank) if k not in wanted):
            raise ValueError("queries come from one matrix, or from a latent of a given rank (dq, dq_norm, uq)")
        self.interleaved = True
        if position is not None:
            self.interleaved = getattr(position, "layout", "halves") == "interleaved"
            if position.rotary_dim > rot_dim:
                raise ValueError(f"rotary dims ({position.rotary_dim}) exceed the rotated part ({rot_dim})")
        self.q_size = heads * (dim + rot_dim)
        self.row = kv_rank + rot_dim  # a cached row
        self.w_in = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = self.latent_norm = self.q_norm = self.sinks = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        position = env.positions[params["position"]] if params.get("position") else None
        return cls(names=params["names"], hidden_size=params.get("hidden_size", env.hidden_size),
                   heads=params["heads"], dim=params["dim"], rot_dim=params["rot_dim"],
                   vdim=params["vdim"], kv_rank=params["kv_rank"], scale=params["scale"],
                   eps=params["eps"], position=position, dtype=env.torch_dtype, q_rank=params.get("q_rank"))

    def weights(self) -> dict[str, WeightDecl]:
        n, h = self.names, self.hidden_size
        out = {
            n["dkv"]: WeightDecl((self.row, h)),
            n["latent_norm"]: WeightDecl((self.kv_rank,), "vector", "ones_plus_normal"),
            n["uk"]: WeightDecl((self.heads * self.dim, self.kv_rank)),
            n["uv"]: WeightDecl((self.heads * self.vdim, self.kv_rank)),
            n["o"]: WeightDecl((h, self.heads * self.vdim)),
        }
        if self.q_rank is None:
            out[n["q"]] = WeightDecl((self.q_size, h))
        else:
            out[n["dq"]] = WeightDecl((self.q_rank, h))
            out[n["dq_norm"]] = WeightDecl((self.q_rank,), "vector", "ones_plus_normal")
            out[n["uq"]] = WeightDecl((self.q_size, self.q_rank))
        if "gate" in n:
            out[n["gate"]] = WeightDecl((self.heads, h))
        if "sink" in n:
            out[n["sink"]] = WeightDecl((self.heads,), "vector")
        return out

    def bind(self, tensors, env: BuildEnv) -> None:
        import torch

        n = self.names
        # one product for the queries (or their latent), the latent with the shared key part, and the gate
        rows = [tensors[n[k]].to(self.dtype) for k in ("q" if self.q_rank is None else "dq", "dkv", "gate") if k in n]
        self.w_in = torch.cat(rows).contiguous()
        if self.q_rank is not None:
            self.w_uq = tensors[n["uq"]].to(self.dtype).contiguous()
            self.q_norm = tensors[n["dq_norm"]].float().contiguous()
        self.latent_norm = tensors[n["latent_norm"]].float().contiguous()
        uk = tensors[n["uk"]].to(self.dtype).view(self.heads, self.dim, self.kv_rank)
        self.w_uk_t = uk.transpose(1, 2).contiguous()  # [heads, kv_rank, dim]: query side of the key product
        self.w_uv = tensors[n["uv"]].to(self.dtype).view(self.heads, self.vdim, self.kv_rank).contiguous()
        self.w_o = tensors[n["o"]].to(self.dtype).contiguous()
        if "sink" in n:
            self.sinks = tensors[n["sink"]].float().contiguous()

    def cache_request(self) -> PagedKVRequest:
        return PagedKVRequest(1, self.row, None, value_dim=0)

    def forward(self, x, ctx, binding: CacheBinding):
        import torch

        n, H, ops, ws = x.shape[0], self.heads, ctx.ops, ctx.ws
        group = ctx.groups[binding.group]
        cache = group.k[binding.slot]
        table = self.position.rotary_table() if self.position is not None else None
        rot_dims = self.position.rotary_dim if self.position is not None else 0
        sizes = dict(heads=H, dim=self.dim, rot_dim=self.rot_dim, rank=self.kv_rank, page_size=group.page_size,
                     interleaved=self.interleaved)
        proj = ops.linear(x, self.w_in, ws=ws, tag="latent.in", out_dtype=torch.float32, allow_split=True)
        at = self.q_size if self.q_rank is None else self.q_rank  # where the latent's columns start
        gate = cq = None
        extra = {}
        if "gate" in self.names:
            gate = ws.buffer("latent.gate", n, H, torch.float32)
            extra.update(gate_pre=proj[..., at + self.row: at + self.row + H], gate=gate)
        if self.q_rank is not None:
            cq = ws.buffer("latent.cq", n, self.q_rank, self.dtype)
            extra.update(cq=proj[..., : self.q_rank], cq_norm_w=self.q_norm, cq_out=cq)
        ops.latent_prep(ctx.positions, table, rot_dims, **sizes, eps=self.eps, dkv=proj[..., at: at + self.row],
                        norm_w=self.latent_norm, cache=cache,
                        slot_mapping=group.slot_mapping if binding.writes else None, **extra)
        q = proj[..., : self.q_size]
        if cq is not None:
            q = ops.linear(cq, self.w_uq, ws=ws, tag="latent.uq", out_dtype=torch.float32, allow_split=True)
        q_abs = ws.buffer("latent.q", n, H * self.row, self.dtype)
        ops.latent_queries(q, self.w_uk_t, q_abs, ctx.positions, table, rot_dims, **sizes, ws=ws)
        mixed = ws.buffer("latent.mixed", n, H * self.kv_rank, self.dtype)
        ops.paged_attention(q_abs, cache, cache, group.block_tables, ctx, H, 1, self.row,
                            group.page_size, self.scale, 0, mixed, ragged=group.ragged,
                            value_dim=self.kv_rank, sinks=self.sinks)
        out = ws.buffer("latent.out", n, H * self.vdim, self.dtype)
        ops.headwise_linear(mixed.view(n, H, self.kv_rank), self.w_uv, out.view(n, H, self.vdim), row_scale=gate)
        return ops.linear(out, self.w_o, ws=ws, tag="mixer.delta", out_dtype=torch.float32, allow_split=True)
