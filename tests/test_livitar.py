"""The Livitar design in the engine against the plain whole-sequence implementation
(`tests/plain_livitar.py`): whole prompts, token-by-token decoding, portions down to two tokens, mixed
batches with pages and slots used again, configurations of odd sizes; every mechanism alone against its
plain function, with inputs made so that a key far away, a bias that is one position off, a lost state, a
stream that is read or written wrongly or a missing shared expert shows; on the CPU through the plain
stand-ins of the kernels, on the GPU through the kernels in both precisions; long decoding; greedy
generation through the engine's own entry point and scheduler."""

from __future__ import annotations

import math
from types import SimpleNamespace

import pytest
import torch

from tests import helpers as H
from tests import livitar_configs as V
from tests import plain_livitar as P

LENGTHS = [50, 21, 37, 64, 9, 1]
# (under these names the run's summary lists this file's comparisons: their bounds are measured)
LABEL = {"float32": "float32, Livitar", "bfloat16": "bfloat16, Livitar"}
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
D = torch.float64


def _requests(cfg, lengths=LENGTHS, seed=700):
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed + i)).tolist()
            for i, n in enumerate(lengths)}


def _want(cfg, weights, requests):
    return {rid: P.forward(cfg, weights, toks, D).float() for rid, toks in requests.items()}


def _float32_bound(cfg, weights, requests, want) -> dict:
    """Three times what rounding alone does to the plain implementation when it runs in 32-bit
    instead of 64-bit, and never below the engine's fixed bound for tiny models."""
    worst = max(float((P.forward(cfg, weights, toks, torch.float32) - want[rid]).abs().max())
                for rid, toks in requests.items())
    return dict(atol=max(3 * worst, H.TOL["float32"]["atol"]), rtol=H.TOL["float32"]["rtol"])


def _position_errors(got, want):
    """Per position, over all requests: the root mean square of the difference over that of the logits."""
    err = [(got[rid].double() - want[rid].double()).pow(2).mean(-1).sqrt() / want[rid].double().pow(2).mean(-1).sqrt()
           for rid in want]
    return torch.cat(err)


def _bfloat16_bound(tmp_path, cfg, weights, requests, want) -> dict:
    """From the same requests on the plain stand-ins of the kernels run in bfloat16 (activations rounded
    between the parts, as the kernels round them): three times the median error of a position (never below
    0.04), and the share of positions that rounding alone carries beyond that.  Such positions there are:
    where a token's experts are a close call, rounding chooses another one, and everything after sees it."""
    from tests.ref_ops import RefOps

    room = sum(H.round64(len(t)) for t in requests.values())
    got = H.collect(_session(tmp_path / "bound", cfg, weights, "bfloat16", "cpu", RefOps(), room, 16),
                    H.trace_whole(requests))
    err = _position_errors(got, want)
    bound = max(3 * float(err.median()), 0.04)
    assert bound < 0.3, "the test weights magnify rounding so much that a fault would hide in it"
    return dict(pos_rel_rms=bound, share=float((err > bound).float().mean()))


def _bound(tmp_path, dtype, cfg, weights, requests, want):
    return (_float32_bound(cfg, weights, requests, want) if dtype == "float32"
            else _bfloat16_bound(tmp_path, cfg, weights, requests, want))


def _check(got, want, dtype, what, tol) -> None:
    """32-bit: every position within the bound.  bfloat16: at most twice the share of positions beyond it that
    rounding alone brings, and 4 % (a fault of a cache, a state or a batch is not limited to a few)."""
    if dtype == "float32":
        for rid in want:
            H.assert_close(got[rid], want[rid], LABEL[dtype], f"{what} {rid}", tol)
        return
    assert all(got[rid].shape == want[rid].shape and bool(torch.isfinite(got[rid]).all()) for rid in want), what
    err = _position_errors(got, want)
    share, allowed = float((err > tol["pos_rel_rms"]).float().mean()), 2 * tol["share"] + 0.04
    H._record(LABEL[dtype], max_median_pos_rel_rms=float(err.median()), max_share_beyond=share)
    assert float(err.median()) < tol["pos_rel_rms"] / 1.5, (what, float(err.median()), tol)
    assert share <= allowed, (what, share, tol)


def _session(tmp_path, cfg, weights, dtype, device, ops, max_tokens, page_size):
    from inference_engine_b200.engine.replay import ReplaySession

    raw = V.without_bucket_counts(cfg)  # (the folder leaves them to the tensors' shapes)
    folder = H.write_model_dir(tmp_path / f"m{abs(hash(str(cfg))) % 10**8}", raw, weights)
    return ReplaySession(folder, dtype, max_tokens, device=device, ops=ops, page_size=page_size)


def _run_all_modes(tmp_path, name, dtype, device, ops, page_size=4, lengths=LENGTHS):
    cfg = V.ALL_CONFIGS[name]
    weights = V.make_weights(cfg, seed=11)
    requests = _requests(cfg, lengths)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, dtype, cfg, weights, requests, want)
    mixed, peak = H.trace_mixed(requests, seed=5, tail=7, max_portion=15)
    whole_room = sum(H.round64(len(t)) for t in requests.values())
    results = {}
    for mode, (trace, room) in {"whole": (H.trace_whole(requests), whole_room),
                                "tail": (H.trace_decode_tail(requests, 14), whole_room),
                                "portions": (H.trace_portions(requests, (5, 2, 13, 3, 2, 8)), whole_room),
                                "mixed": (mixed, peak)}.items():
        session = _session(tmp_path, cfg, weights, dtype, device, ops, room, page_size)
        got = H.collect(session, trace)
        _check(got, want, dtype, f"livitar {name} {mode}", tol)
        # everything went back to the pools
        assert session.cache.num_free_pages == [p.num_pages for p in session.cache.pools]
        assert session.cache.slots.num_free == session.cache.slots.num_slots
        results[mode] = got
    return results


def test_the_test_weights_make_no_close_call_in_the_routers():
    """The experts the plain implementation chooses are chosen by a margin that 32-bit rounding does not
    reach, so a difference in the logits is a fault and not another expert."""
    for name, cfg in V.CONFIGS.items():
        weights = V.make_weights(cfg, seed=11)
        margins = []
        for toks in _requests(cfg, [30, 13, 21, 9, 1]).values():
            P.forward(cfg, weights, toks, D, margins=margins)
        assert margins and min(margins) > 1e-4, (name, min(margins))


@pytest.mark.parametrize("name", list(V.CONFIGS))
def test_every_way_of_cutting_on_the_plain_kernels(tmp_path, name):
    from tests.ref_ops import RefOps

    _run_all_modes(tmp_path, name, "float32", "cpu", RefOps(), lengths=[30, 13, 21, 9, 1])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(V.CONFIGS))
def test_every_way_of_cutting_on_the_gpu(tmp_path, name, dtype):
    from inference_engine_b200.kernels import get_ops

    results = _run_all_modes(tmp_path, name, dtype, "cuda", get_ops("cuda"), lengths=[150, 21, 67, 64, 9, 1, 33])
    if dtype == "float32":  # a row's arithmetic does not depend on the cutting or the batch at all
        for mode in ("tail", "portions", "mixed"):
            for rid, rows in results["whole"].items():
                assert torch.equal(rows, results[mode][rid]), f"{name} {mode} {rid}: 32-bit logits differ by cutting"
    get_ops("cuda").check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model_with_long_prompts(tmp_path, dtype):
    """Prompts of hundreds of tokens over several chunks of the retention, many tiles and pages of 16,
    sizes that reach the tensor-core kernels in bfloat16."""
    from inference_engine_b200.kernels import get_ops

    cfg = V.WIDE
    weights = V.make_weights(cfg, seed=21)
    requests = _requests(cfg, [420, 130, 257, 64], seed=900)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, dtype, cfg, weights, requests, want)
    mixed, peak = H.trace_mixed(requests, seed=8, tail=20, max_portion=90)
    room = sum(H.round64(len(t)) for t in requests.values())
    names = ("sink_attention_mma", "retention_chunks", "retention_step")
    before = {n: get_ops("cuda").launch_counts.get(n, 0) for n in names}
    results = {}
    for mode, (trace, space) in {"whole": (H.trace_whole(requests), room),
                                 "tail": (H.trace_decode_tail(requests, 40), room),
                                 "portions": (H.trace_portions(requests, (70, 2, 129, 3, 64, 33)), room),
                                 "mixed": (mixed, peak)}.items():
        session = _session(tmp_path / mode, cfg, weights, dtype, "cuda", get_ops("cuda"), space, 16)
        results[mode] = H.collect(session, trace)
        _check(results[mode], want, dtype, f"wide {mode}", tol)
        assert session.cache.num_free_pages == [p.num_pages for p in session.cache.pools]
    ran = {n: get_ops("cuda").launch_counts.get(n, 0) - before[n] for n in names}
    if dtype == "float32":
        assert not any(ran.values())
        for mode in ("tail", "portions", "mixed"):
            for rid in requests:
                assert torch.equal(results["whole"][rid], results[mode][rid]), (mode, rid)
    else:
        assert all(ran.values()), ran  # (the tensor-core and fused kernels did serve these sizes)
    get_ops("cuda").check_errors()


# --- what the model is made of ---------------------------------------------------------------------


def test_layout_of_the_model_and_its_caches():
    from inference_engine_b200.config import build_model_spec, config_from_dict
    from inference_engine_b200.engine.model import Model

    spec = build_model_spec(config_from_dict(V.MIXED))
    model = Model(spec, "float32", 64)
    assert [type(b).__name__ for b in model.blocks] == ["HyperResidualBlock"] * 5
    assert [type(b.mixer).__name__ for b in model.blocks] == [
        "Retention", "SinkAttention", "SinkAttention", "Retention", "SinkAttention"]
    assert [type(b.feed_forward).__name__ for b in model.blocks] == [
        "RoutedExperts", "RoutedExperts", "NoneType", "RoutedExperts", "RoutedExperts"]
    assert [type(p.feed_forward.shared).__name__ if p.feed_forward else None for p in model.blocks] == [
        "SwiGLU", "SwiGLU", None, "NoneType", "SwiGLU"]
    assert all(type(n).__name__ == "DynamicTanh" for b in model.blocks for n in b.norms.values())
    assert model.embedding.copies == 3 and all(b.streams == 3 for b in model.blocks)
    groups = sorted((g.num_kv_heads, g.head_dim, g.value_dim, g.window, g.num_layers) for g in model.paged_groups)
    assert groups == [(1, 12, 20, None, 1), (2, 8, 8, None, 1), (2, 16, 24, None, 1)]
    assert sorted((g.shape, g.num_layers) for g in model.state_groups) == [((3 * 16 * 8,), 1), ((2 * 20 * 36,), 1)]
    first, log, rel, second, last = (b.mixer for b in model.blocks)
    assert first.position.rotary_dim == 8 and first.position.theta == 500.0 and second.position.rotary_dim == 20
    assert not log.unit_qk and log.warmth == (0.0, 0) and set(log.names) >= {"temp", "r1", "r2", "gate"}
    assert rel.unit_qk and rel.warmth == (0.7, 8) and rel.rel_buckets == 16 and rel.bias_max == 40
    assert last.rel_buckets == 6 and last.warmth == (0.0, 0)
    assert model.blocks[0].feed_forward.weight_scale == 1.5 and model.blocks[0].feed_forward.scoring == "softmax"
    for name, raw in V.ALL_CONFIGS.items():
        declared = Model(build_model_spec(config_from_dict(raw)), "float32", 64).declared_weights()
        assert {n: d.shape for n, d in declared.items()} == V.tensor_shapes(raw), name


def test_bucket_counts_come_from_the_tensors_shapes():
    from inference_engine_b200.config import ConfigError, build_model_spec, config_from_dict

    cfg = config_from_dict(V.without_bucket_counts(V.MIXED))
    with pytest.raises(ConfigError, match="buckets"):
        build_model_spec(cfg)
    spec = build_model_spec(cfg.with_tensor_shapes(V.tensor_shapes(V.MIXED)))
    assert [layer.mixer.params.get("rel_buckets") for layer in spec.layers] == [None, None, 16, None, 6]


@pytest.mark.parametrize("name", list(V.ALL_CONFIGS))
def test_footprint_formula_counts_what_the_model_declares(name):
    from inference_engine_b200.architectures.livitar import livitar_footprint
    from inference_engine_b200.config import build_model_spec, config_from_dict
    from inference_engine_b200.engine.model import Model

    cfg = config_from_dict(V.ALL_CONFIGS[name])
    assert livitar_footprint(cfg) == Model(build_model_spec(cfg), "float32", 64).footprint()


def test_configuration_errors():
    from inference_engine_b200.config import ConfigError, build_model_spec, config_from_dict

    layers = V.MIXED["layers"]

    def changed(i, **mixer):
        return dict(V.MIXED, layers=[dict(layers[i], mixer=dict(layers[i]["mixer"], **mixer))])

    def feeding(mlp):
        return dict(V.MIXED, layers=[dict(layers[0], mlp=mlp)])

    for raw, match in [
            (dict(V.MIXED, layers=[dict(layers[0], type="other")]), "type"),
            (dict(V.MIXED, layers=[]), "layers"),
            (dict(V.MIXED, streams=0), "streams"), (dict(V.MIXED, streams=17), "streams"),
            ({k: v for k, v in V.MIXED.items() if k != "streams"}, "streams"),
            ({k: v for k, v in V.MIXED.items() if k != "norm"}, "eps"),
            (changed(0, decay=[0.5]), "decay"), (changed(0, decay=None), "decay"),
            (changed(0, rot={"dims": 7, "base": 10.0}), "rot"), (changed(0, rot={"dims": 18, "base": 10.0}), "rot"),
            (changed(1, kv_heads=4), "kv_heads"), (changed(1, scale=None), "scale"), (changed(1, vdim=0), "vdim"),
            (changed(2, bias_max=None), "bias_max"), (changed(2, q_temp={"coef": 1.0, "every": 0}), "every"),
            (changed(2, q_temp={"coef": 1.0, "every": 2.5}), "every"),
            (feeding({"kind": "dense", "ff": 8}), "kind"), (feeding(V.moe(4, 5, 8)), "top"),
            (feeding(V.moe(4, 2, 0)), "unit")]:
        with pytest.raises(ConfigError, match=match):
            config_from_dict(raw)
    with pytest.raises(ConfigError, match="bias_max"):  # (the widening buckets need distances to widen over)
        build_model_spec(config_from_dict(changed(2, bias_max=8)))


def test_streams_need_layers_and_norms_that_know_them():
    from inference_engine_b200.parts.norm import AddedTerms, DynamicTanh, StreamMix
    from inference_engine_b200.parts.block import HyperResidualBlock

    norm = DynamicTanh("w", "b", "a", 4, torch.float32)
    ctx = SimpleNamespace(ws=None, ops=None)
    with pytest.raises(ValueError, match="multiplier"):
        norm.add_norm(torch.zeros(1, 4), None, ctx, delta_scale=0.5)
    with pytest.raises(ValueError, match="AddedTerms"):
        norm.add_norm(torch.zeros(1, 4), None, ctx, delta_post=AddedTerms())
    block = HyperResidualBlock(SimpleNamespace(), None, {"mixer": norm}, {"mixer": {}}, 2)
    block.read["mixer"] = None
    with pytest.raises(ValueError, match="streams"):
        block.forward(torch.zeros(1, 8), None, ctx, None, delta_post=StreamMix(3))
    with pytest.raises(ValueError, match="16"):
        HyperResidualBlock(SimpleNamespace(), None, {"mixer": norm}, {"mixer": {}}, 17)


def test_random_weights_keep_the_streams_apart_and_finite():
    """The random-weights mode draws a mixing near the unit matrix and positive numbers for the logarithmic
    bias, whose argument a random sign would make negative."""
    from inference_engine_b200.engine.loading import random_model
    from inference_engine_b200.weights.random_weights import random_tensor

    model, _ = random_model(V.STREAMS, seed=1, dtype="float32", device="cpu", max_positions=64)
    mix = model.blocks[0].write["mixer"].mix
    assert (mix - torch.eye(5)).abs().max() < 0.2
    decls = model.declared_weights()
    assert (random_tensor("l3.mix.r2", decls["l3.mix.r2"], 0, 0.02, torch.bfloat16) > 0.5).all()


# --- every mechanism alone, against its plain function -------------------------------------------


def _ops(device):
    if device == "cpu":
        from tests.ref_ops import RefOps

        return RefOps()
    from inference_engine_b200.kernels import get_ops

    return get_ops("cuda")


def _ctx(lens, starts, device, slots=None, ws=None):
    """The parts of a step's context the kernels read, for requests with `lens` new tokens that
    start at positions `starts`."""
    b = len(lens)
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    seq = [i for i, n in enumerate(lens) for _ in range(n)]
    pos = [s + t for s, n in zip(starts, lens) for t in range(n)]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    return SimpleNamespace(num_tokens=cu[-1], num_seqs=b, seq_of_token=i32(seq), positions=i32(pos), cu_q=i32(cu),
                           q_starts=cu[:-1], q_lens=list(lens), start_positions=list(starts), max_q_len=max(lens),
                           ctx_lens=i32([s + n for s, n in zip(starts, lens)]), bounds=None, padded=False,
                           slots=i32(slots if slots is not None else list(range(b))), ws=ws)


def _paged(x, page_size, pages_total, order, device):
    """Rows [T, G, d] into a cache [pages, G, page_size, d] at the pages `order` names."""
    T, G, d = x.shape
    cache = torch.full((pages_total + 1, G, page_size, d), 9.0, device=device)  # (unused rows hold nonsense)
    for t in range(T):
        cache[order[t // page_size], :, t % page_size] = x[t].to(device)
    return cache


@pytest.mark.parametrize("buckets,bias_max", [(2, 17.5), (6, 9), (8, 5), (16, 40), (32, 5000), (1, 3), (32, 128), (64, 1000)])
def test_buckets_of_distances(buckets, bias_max):
    """The table the kernels read against the formula at every distance, the first and last distance of the
    widening buckets included; from its end on the last bucket holds everything."""
    from inference_engine_b200.parts.sink_attention import buckets_by_distance

    table = buckets_by_distance(buckets, bias_max)
    assert table[: buckets // 2] == list(range(buckets // 2)) or buckets == 1
    assert table[-1] == buckets - 1 and len(table) <= max(math.ceil(bias_max), 1) + 1
    for n in range(2 * len(table) + 50):
        assert table[min(n, len(table) - 1)] == P.bucket(n, buckets, bias_max), n
    assert sorted(table) == table


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("streams,width", [(1, 50), (2, 72), (3, 72), (4, 1100), (5, 50), (16, 24), (7, 2048)])
@pytest.mark.parametrize("norm", ["tanh", "rms"])
def test_streams_are_mixed_read_and_normalised(device, streams, width, norm):
    """Every stream from all the old ones and the sublayer's output (whole or in parts), the next
    sublayer's reading of the new streams and its norm; the first reading (nothing to add), chosen rows
    (the streams then stay as they are), the plain sum at the model's end, no norm at all."""
    ops, g = _ops(device), torch.Generator().manual_seed(streams + width)
    n, eps = 7, 1e-5
    h = torch.randn(n, streams * width, generator=g)
    delta = torch.randn(3, n, width, generator=g) * 2
    mix, out_c = torch.randn(streams, streams, generator=g) / streams ** 0.5, torch.randn(streams, generator=g)
    read = torch.randn(streams, generator=g)
    w, b, alpha = torch.randn(width, generator=g), torch.randn(width, generator=g), torch.tensor([0.7])
    W = {"n": w.to(D), "n.b": b.to(D), "n.alpha": alpha[0].to(D)}
    dev = lambda t: None if t is None else t.to(device)  # noqa: E731
    xs = h.to(D).view(n, streams, width).transpose(0, 1)

    def normed(u):
        return P.dynamic_tanh(u, W, "n") if norm == "tanh" else P.unit_rms(u, eps) * w.to(D)

    def run(y, mixing, rows=None, rd=read, with_out=True, dtype=torch.float32):
        hd = h.clone().to(device)
        out = torch.zeros(n if rows is None else len(rows), width, device=device, dtype=dtype) if with_out else None
        r = None if rows is None else torch.tensor(rows, dtype=torch.int32, device=device)
        ops.stream_mix_norm(hd, streams, dev(y), dev(mix) if mixing else None, dev(out_c) if mixing else None, dev(rd),
                            dev(w), dev(b) if norm == "tanh" else None, dev(alpha) if norm == "tanh" else None, eps, out, r)
        return hd.cpu(), None if out is None else out.float().cpu()

    tol = dict(atol=2e-5, rtol=2e-5)
    for y in (delta, delta[0]):
        total = y.to(D).sum(0) if y.dim() == 3 else y.to(D)
        new = P.write_streams(xs, total, mix.to(D), out_c.to(D))
        want_h = new.transpose(0, 1).reshape(n, -1).float()
        u = P.read_streams(new, read.to(D))
        got_h, got = run(y, True)
        torch.testing.assert_close(got_h, want_h, **tol)
        torch.testing.assert_close(got, normed(u).float(), **tol)
        got_h, got = run(y, True, rows=[5, 0, 5], dtype=torch.bfloat16)
        torch.testing.assert_close(got, normed(u).float()[[5, 0, 5]], atol=5e-2, rtol=2e-2)
        assert torch.equal(got_h, h)
        _, got = run(y, True, rd=None)
        torch.testing.assert_close(got, normed(new.sum(0)).float(), **tol)
        got_h, _ = run(y, True, with_out=False)
        torch.testing.assert_close(got_h, want_h, **tol)
        # without coefficients: the output is added to every stream
        got_h, _ = run(y, False)
        torch.testing.assert_close(got_h, (xs + total).transpose(0, 1).reshape(n, -1).float(), **tol)
        if streams > 1:  # (a transposed mixing would show)
            other = P.write_streams(xs, total, mix.T.to(D), out_c.to(D))
            assert (other - new).abs().max() > 0.1
    got_h, got = run(None, True)
    torch.testing.assert_close(got, normed(P.read_streams(xs, read.to(D))).float(), **tol)
    assert torch.equal(got_h, h)


@pytest.mark.parametrize("device", DEVICES)
def test_embedding_fills_every_stream(device):
    ops, g = _ops(device), torch.Generator().manual_seed(1)
    table = torch.randn(11, 24, generator=g)
    ids = torch.tensor([3, 0, 10, 3], dtype=torch.int32)
    out = torch.zeros(4, 3 * 24, device=device)
    ops.embedding(table.to(device), ids.to(device), out, 1.0, 3)
    assert torch.equal(out.cpu().view(4, 3, 24), table[ids.long()][:, None].expand(4, 3, 24))


def _retention_case(g, lens, starts, H, d, dv, rot, decay, base=30.0):
    """The fused projection of a step, the state every request brings, and what must come out: outputs and
    states of the plain functions, request by request, in 64-bit."""
    n, eps = sum(lens), 1e-5
    proj = torch.randn(n, 2 * H * (d + dv), generator=g)
    state = torch.randn(len(lens) + 1, H * dv * d, generator=g)  # (one slot nobody owns)
    slots = torch.randperm(len(lens) + 1, generator=g).tolist()[: len(lens)]
    want, after, at = torch.zeros(n, H * dv, dtype=D), state.to(D).clone(), 0
    for length, start, slot in zip(lens, starts, slots):
        rows = proj[at: at + length].to(D)
        pad = torch.zeros(start, H, d, dtype=D)  # (the rotation counts from the request's position 0)
        q, k = (P.rotate_half(torch.cat([pad, rows[:, i * H * d: (i + 1) * H * d].reshape(length, H, d)]), rot, base)[start:]
                for i in range(2))
        v = rows[:, 2 * H * d: 2 * H * d + H * dv].reshape(length, H, dv)
        before = state[slot].to(D).view(H, dv, d).transpose(1, 2)
        # (the kernels scale the read-out instead of the keys: the state holds unscaled keys)
        o, S = P.retention_core(q, k, v, decay.to(D), before)
        o = P.unit_rms(o * d ** -0.5, eps).reshape(length, -1)
        want[at: at + length] = o * torch.nn.functional.silu(rows[:, 2 * H * d + H * dv:])
        after[slot] = S.transpose(1, 2).reshape(-1)
        at += length
    table = None
    if rot:
        ang = torch.arange(700, dtype=D)[:, None] * base ** (-torch.arange(0, rot, 2, dtype=D) / rot)
        table = torch.stack((ang.cos(), ang.sin()), dim=1).float()
    return proj, state, slots, want.float(), after.float(), table, eps


RETENTION_STEPS = [([1, 1, 3], [5, 0, 9]), ([8, 2], [0, 600]), ([150, 1, 64, 63, 65], [0, 100, 7, 3, 64]), ([300], [11]),
                   ([2, 9], [64, 0]), ([65], [0])]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv,rot", [(3, 64, 48, 64), (2, 128, 128, 64), (4, 20, 28, 10), (1, 33, 17, 0), (5, 16, 112, 16),
                                        (2, 100, 120, 100), (1, 1, 1, 0), (2, 144, 40, 16), (1, 6, 130, 6)])
def test_retention_in_every_kind_of_step(device, dtype, H, d, dv, rot):
    """Requests of one to hundreds of tokens in one step, from states that others left in scattered slots:
    outputs, the slots afterwards, and the slot that nobody owns.  Decays from one that forgets at once to
    one that never does.  On the GPU in bfloat16 the fused kernels (a few tokens per request; chunks),
    for sizes beyond theirs and in 32-bit rotation, recurrence and read-out by themselves."""
    from inference_engine_b200.engine.workspace import Workspace

    ops, g = _ops(device), torch.Generator().manual_seed(d + dv)
    decay = torch.tensor([0.0, 0.9, 0.999, 1.0, 0.3])[:H] if H > 1 else torch.tensor([0.97])
    gates = torch.stack([decay, torch.ones(H), torch.ones(H)], -1)[None].contiguous()
    powers = (decay.to(D)[:, None] ** torch.arange(65, dtype=D)).float()
    out_dtype = getattr(torch, dtype)
    dev = lambda t: None if t is None else t.to(device)  # noqa: E731
    for lens, starts in RETENTION_STEPS if d > 1 else RETENTION_STEPS[:3]:
        proj, state, slots, want, after, table, eps = _retention_case(g, lens, starts, H, d, dv, rot, decay)
        ctx = _ctx(lens, starts, device, slots)
        got_state = state.clone().to(device)
        out = torch.full((sum(lens), H * dv), 7.0, device=device, dtype=out_dtype)
        ops.retention(proj.clone().to(device), ctx, dev(table), rot, dev(gates), dev(powers), got_state, ctx.slots, out, H, d,
                      dv, eps, Workspace(device))
        tol = dict(atol=2e-4, rtol=2e-4) if dtype == "float32" else dict(atol=4e-3, rtol=1e-2)
        torch.testing.assert_close(out.float().cpu(), want, **tol)
        scale = float(after.abs().max())
        assert float((got_state.cpu() - after).abs().max()) < 5e-5 * scale  # (16 bits of mantissa at least)
        idle = next(i for i in range(len(lens) + 1) if i not in slots)
        assert torch.equal(got_state.cpu()[idle], state[idle])
    ops.check_errors()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_retention_remembers_its_first_token(device, dtype):
    """A mark that only the first token carries, read hundreds of tokens and several portions later through a
    head that hardly forgets: a state lost between portions, chunks or steps shows."""
    from inference_engine_b200.engine.workspace import Workspace

    ops, g = _ops(device), torch.Generator().manual_seed(2)
    H, d, dv, T = 2, 32, 16, 290
    decay = torch.tensor([1.0, 0.9995])
    q, k = torch.randn(T, H, d, generator=g) * 0.02, torch.randn(T, H, d, generator=g) * 0.02
    k[:, :, 0], q[:, :, 0] = 0.0, 1.0
    k[0, :, 0] = 4.0  # (nobody else writes along entry 0, and everyone reads there)
    v, gate = torch.randn(T, H, dv, generator=g), torch.full((T, H, dv), 3.0)
    o, _ = P.retention_core(q.to(D), k.to(D), v.to(D), decay.to(D))
    want = (P.unit_rms(o * d ** -0.5, 1e-5) * torch.nn.functional.silu(gate.to(D))).reshape(T, -1).float()
    lost, _ = P.retention_core(q[1:].to(D), k[1:].to(D), v[1:].to(D), decay.to(D))
    lost = (P.unit_rms(lost * d ** -0.5, 1e-5) * torch.nn.functional.silu(gate[1:].to(D))).reshape(T - 1, -1).float()
    assert (lost - want[1:]).abs().amax(-1).min() > 0.3
    proj = torch.cat([t.reshape(T, -1) for t in (q, k, v, gate)], dim=1)
    gates = torch.stack([decay, torch.ones(H), torch.ones(H)], -1)[None].contiguous().to(device)
    powers = (decay.to(D)[:, None] ** torch.arange(65, dtype=D)).float().to(device)
    for portions in ([290], [1] * 12 + [70, 2, 130, 64, 8, 3, 1], [64, 64, 64, 64, 34], [200] + [1] * 90):
        state, got, at = torch.zeros(2, H * d * dv, device=device), [], 0
        for n in portions:
            ctx = _ctx([n], [at], device, [1])
            out = torch.zeros(n, H * dv, device=device, dtype=getattr(torch, dtype))
            ops.retention(proj[at: at + n].clone().to(device), ctx, None, 0, gates, powers, state, ctx.slots, out, H, d, dv, 1e-5,
                          Workspace(device))
            got.append(out.float().cpu())
            at += n
        tol = dict(atol=1e-3, rtol=1e-3) if dtype == "float32" else dict(atol=2e-2, rtol=1e-2)
        torch.testing.assert_close(torch.cat(got), want, **tol)


def _bias_inputs(kind, H, T, g):
    """(arguments for the kernels, a function of the head for the plain one) for one kind of bias."""
    dist = P.distances(T)
    if kind == "log":
        r1, r2 = 0.2 + 2.5 * torch.rand(H, generator=g), 0.05 + 0.5 * torch.rand(H, generator=g)
        return dict(log_bias=(r1, r2)), lambda h: P.log_distance_bias(dist.to(D), r1[h].to(D), r2[h].to(D))
    if kind == "none":
        return {}, None
    buckets, bias_max = kind
    rel = torch.randn(buckets, H, generator=g) * 2
    from inference_engine_b200.parts.sink_attention import buckets_by_distance

    table = rel[torch.tensor(buckets_by_distance(buckets, bias_max))].t().contiguous()
    return dict(bias_table=table), lambda h: P.bucket_bias(dist, rel.to(D), bias_max, h)


def _to(kw, device):
    return {k: tuple(t.to(device) for t in v) if isinstance(v, tuple) else v.to(device) for k, v in kw.items()}


KINDS = ["log", "none", (16, 40), (2, 17.5), (32, 5000), (8, 5), (1, 3)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind", KINDS, ids=str)
def test_attention_with_a_bias_by_distance(device, kind):
    """Every earlier position is seen, with the bias of its distance; value rows of another size than key rows;
    a gate per value entry that lies beside other columns; portions and single tokens over scattered
    pages of 4; one key per query, near or far, stands out.  A bias that is off by one position or one
    head, or a gate taken per head, is checked to show."""
    ops, g = _ops(device), torch.Generator().manual_seed(3)
    T, H, G, d, dv, ps = 45, 4, 2, 12, 20, 4
    k, q = torch.randn(T, G, d, generator=g) * 0.3, torch.randn(T, H, d, generator=g) * 0.3
    for t in range(T):
        target = [0, t // 2, max(t - 1, 0)][t % 3]
        k[target, :, t % d] += 1.0
        q[t, :, t % d] += 3.0
    v, gate = torch.randn(T, G, dv, generator=g), torch.randn(T, H, dv, generator=g) * 2
    scale = 0.6
    kw, bias = _bias_inputs(kind, H, T, g)
    want = P.attention_core(q.to(D), k.to(D), v.to(D), scale, bias) * torch.sigmoid(gate.to(D))
    if kind not in ("none", (1, 3)):
        shifted = P.attention_core(q.to(D), k.to(D), v.to(D), scale,
                                   lambda h: torch.cat([bias(h)[1:], bias(h)[-1:]]))  # (every distance one more)
        assert (shifted * torch.sigmoid(gate.to(D)) - want)[8:-1].abs().max() > 0.02
        swapped = P.attention_core(q.to(D), k.to(D), v.to(D), scale, lambda h: bias((h + 1) % H))
        assert (swapped * torch.sigmoid(gate.to(D)) - want).abs().max() > 0.05
    order = [7, 2, 11, 0, 5, 9, 3, 10, 1, 8, 6, 4]
    kc, vc = _paged(k, ps, 12, order, device), _paged(v, ps, 12, order, device)
    tables = torch.tensor([order], dtype=torch.int32, device=device)
    got, at = [], 0
    for n in [13, 1, 1, 2, 20, 1, 7]:
        out = torch.zeros(n, H * dv, device=device)
        wide = torch.cat([torch.zeros(n, 3), gate[at: at + n].reshape(n, -1)], dim=1).to(device)
        ops.sink_attention(q[at: at + n].reshape(n, -1).to(device).contiguous(), kc, vc, tables, _ctx([n], [at], device), H, G,
                           d, dv, ps, scale, None, None, wide[:, 3:], out, **_to(kw, device))
        got.append(out.cpu().view(n, H, dv))
        at += n
    torch.testing.assert_close(torch.cat(got), want.float(), atol=1e-4, rtol=1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("d,dv,heads,kv", [(64, 48, 5, 5), (80, 112, 6, 3), (128, 128, 4, 1), (16, 48, 5, 5), (48, 16, 8, 2),
                                           (256, 64, 2, 1)])
@pytest.mark.parametrize("kind", ["log", (16, 40), (32, 5000), (24, 150), (1, 3)], ids=str)
def test_biased_attention_on_the_tensor_cores(d, dv, heads, kv, kind):
    """The bfloat16 kernel against the plain function: portions that start and end inside tiles of 64, a second
    request of one token in every step, scattered pages, gates per value entry, keys that stand out near
    and far; steps of few tokens cut the keys among blocks that serve several heads with biases of their
    own; tiles that lie wholly beyond the table's end, across it and before it."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(d + heads)
    T, H, G, ps = 333, heads, kv, 16
    bf = lambda x: x.to(torch.bfloat16).float()  # noqa: E731
    k, q = torch.randn(T, G, d, generator=g) * 0.3, torch.randn(T, H, d, generator=g) * 0.3
    v = bf(torch.randn(T, G, dv, generator=g))
    for t in range(0, T, 3):
        target = [0, t // 2, max(t - 40, 0), t][(t // 3) % 4]
        k[target, :, t % d] += 2.0
        q[t, :, t % d] += 5.0
    q, k = bf(q), bf(k)
    gate = torch.randn(T, H, dv, generator=g) * 2
    scale = 0.5
    kw, bias = _bias_inputs(kind, H, T, g)
    want = (P.attention_core(q.to(D), k.to(D), v.to(D), scale, bias) * torch.sigmoid(gate.to(D))).float()
    pages = -(-T // ps)
    order = torch.randperm(pages + 3, generator=g).tolist()[:pages]
    kc, vc = (_paged(x, ps, pages + 3, order, "cuda").to(torch.bfloat16) for x in (k, v))
    tables = torch.tensor([order, [pages + 3] * pages], dtype=torch.int32, device="cuda")
    kc[pages + 3], vc[pages + 3] = 0.5, 0.25  # the second request: one token on the scratch page
    before = ops.launch_counts.get("sink_attention_mma", 0), ops.launch_counts.get("sink_attention_merge", 0)
    got, at = [], 0
    portions = [70, 33, 1, 2, 5, 130, 1, 8, 83]
    for n in portions:
        qq = torch.cat([q[at: at + n].reshape(n, -1), torch.ones(1, H * d)]).to("cuda", torch.bfloat16)
        gg = torch.cat([gate[at: at + n].reshape(n, -1), torch.zeros(1, H * dv)]).cuda()
        out = torch.zeros(n + 1, H * dv, device="cuda", dtype=torch.bfloat16)
        ops.sink_attention(qq, kc, vc, tables, _ctx([n, 1], [at, 0], "cuda"), H, G, d, dv, ps, scale, None, None, gg, out,
                           **_to(kw, "cuda"))
        got.append(out[:n].float().cpu().view(n, H, dv))
        torch.testing.assert_close(out[n].float().cpu(), torch.full((H * dv,), 0.125), atol=2e-3, rtol=0)
        at += n
    ops.check_errors()
    assert at == T and ops.launch_counts.get("sink_attention_mma", 0) == before[0] + len(portions)
    assert ops.launch_counts.get("sink_attention_merge", 0) > before[1]  # (the steps of few tokens were cut)
    torch.testing.assert_close(torch.cat(got), want, atol=0.015, rtol=0.01)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["log", (32, 5000), (32, 128)], ids=str)
def test_far_keys_in_long_decoding(kind):
    """Single tokens at contexts of thousands of positions, where the keys are cut among many blocks: each
    query's key that stands out lies thousands of positions back or among the first, and carries the
    result in spite of its bias, in both precisions' kernels."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(9)
    T, H, G, d, ps = 4500, 4, 2, 64, 16
    bf = lambda x: x.to(torch.bfloat16).float()  # noqa: E731
    k, v = bf(torch.randn(T, G, d, generator=g) * 0.3), bf(torch.randn(T, G, d, generator=g))
    far = {T - 1: 3, T - 2: 1100, 4099: 4035, 4031: 64, 2500: 0, 70: 63}
    q = torch.randn(T, H, d, generator=g) * 0.3
    for i, (t, target) in enumerate(far.items()):  # (a dimension of its own for every probe)
        q[:, :, 5 + i], k[:, :, 5 + i] = 0.0, 0.0
        k[target, :, 5 + i] = 3.0
        q[t, :, 5 + i] = 24.0
    q, k = bf(q), bf(k)
    scale = 0.5
    if kind == "log":
        r1, r2 = torch.tensor([0.3, 1.0, 1.5, 0.7]), torch.tensor([0.1, 0.02, 0.3, 0.5])
        kw, bias_of = dict(log_bias=(r1, r2)), lambda n, h: P.log_distance_bias(n.to(D), r1[h].to(D), r2[h].to(D))
    else:
        kw, _ = _bias_inputs(kind, H, 2, g)
        table = kw["bias_table"].to(D)
        bias_of = lambda n, h: table[h][n.clamp(max=table.shape[1] - 1)]  # noqa: E731
    pages = -(-T // ps)
    order = torch.randperm(pages, generator=g).tolist()
    tables = torch.tensor([order], dtype=torch.int32, device="cuda")
    for dtype, tol in ((torch.bfloat16, 0.02), (torch.float32, 2e-4)):
        kc, vc = _paged(k, ps, pages, order, "cuda").to(dtype), _paged(v, ps, pages, order, "cuda").to(dtype)
        for t, target in far.items():
            want = torch.zeros(H, d, dtype=D)
            for h in range(H):
                s = (k[: t + 1, h // 2].to(D) @ q[t, h].to(D)) * scale + bias_of(t - torch.arange(t + 1), h)
                p = torch.softmax(s, dim=-1)
                assert p[target] > 0.5  # (the far key carries the result)
                want[h] = p @ v[: t + 1, h // 2].to(D)
            out = torch.zeros(1, H * d, device="cuda", dtype=dtype)
            ops.sink_attention(q[t].reshape(1, -1).to("cuda", dtype), kc, vc, tables, _ctx([1], [t], "cuda"), H, G, d, d,
                               ps, scale, None, None, None, out, **_to(kw, "cuda"))
            torch.testing.assert_close(out.float().cpu().view(H, d), want.float(), atol=tol, rtol=tol)
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["log", (16, 40)], ids=str)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_bias_beside_a_window_a_cap_and_a_sink(kind, dtype):
    """The kernels' parameters go together: a bias by distance with a window, kept first positions, capped
    scores, a learned sink and a gate per head."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(4)
    T, H, G, d, ps, window, keep, cap, scale = 150, 4, 2, 32, 16, 70, 5, 6.0, 0.6
    cast = (lambda x: x.to(torch.bfloat16).float()) if dtype == "bfloat16" else (lambda x: x)
    q, k, v = (cast(torch.randn(T, n, d, generator=g)) for n in (H, G, G))
    gate, sinks = torch.randn(T, H, generator=g), torch.randn(H, generator=g)
    kw, bias = _bias_inputs(kind, H, T, g)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    mask = (j <= i) & ((i - j < window) | (j < keep))
    want = torch.zeros(T, H, d, dtype=D)
    for h in range(H):
        s = cap * torch.tanh((q[:, h].to(D) @ k[:, h // 2].to(D).T) * scale / cap) + bias(h)
        s = torch.cat([s.masked_fill(~mask, float("-inf")), sinks[h].to(D).expand(T, 1)], dim=1)
        want[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, h // 2].to(D)
    want = want * torch.sigmoid(gate.to(D))[..., None]
    order = list(range(10))[::-1]
    kc, vc = (_paged(x, ps, 10, order, "cuda").to(getattr(torch, dtype)) for x in (k, v))
    tables, got, at = torch.tensor([order], dtype=torch.int32, device="cuda"), [], 0
    for n in [100, 1, 2, 40, 1, 1, 5]:
        out = torch.zeros(n, H * d, device="cuda", dtype=getattr(torch, dtype))
        ops.sink_attention(q[at: at + n].reshape(n, -1).to("cuda", getattr(torch, dtype)), kc, vc, tables,
                           _ctx([n], [at], "cuda"), H, G, d, d, ps, scale, window, sinks.cuda(), gate[at: at + n].cuda(), out,
                           softcap=cap, keep_first=keep, **_to(kw, "cuda"))
        got.append(out.float().cpu().view(n, H, d))
        at += n
    tol = dict(atol=1e-4, rtol=1e-4) if dtype == "float32" else dict(atol=0.015, rtol=0.01)
    torch.testing.assert_close(torch.cat(got), want.float(), **tol)
    ops.check_errors()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("unit,temp,warmth", [(True, False, (0.7, 4)), (False, True, None), (True, True, (1.3, 1)),
                                              (True, False, None), (False, False, (0.5, 7))])
def test_unit_queries_and_keys_temperatures_and_warmth(device, unit, temp, warmth):
    """Queries and keys of very different sizes divided by their root mean square, a temperature per query
    head, a factor that steps up every few positions (positions around the steps): keys take neither
    temperature nor warmth, values nothing at all, the columns behind them (gates) are left alone."""
    ops, g = _ops(device), torch.Generator().manual_seed(8)
    n, H, G, d, dv, ps, eps = 10, 3, 2, 10, 6, 4, 1e-3
    size = (H + G) * d + G * dv
    proj = torch.randn(n, size + 5, generator=g) * (10.0 ** torch.linspace(-2, 2, n))[:, None]
    pos = torch.tensor([0, 1, 2, 3, 17, 18, 19, 5, 6, 7])
    q, k = proj[:, : H * d].to(D).view(n, H, d), proj[:, H * d: (H + G) * d].to(D).view(n, G, d)
    v = proj[:, (H + G) * d: size].view(n, G, dv)
    if unit:
        q, k = P.unit_rms(q, eps), P.unit_rms(k, eps)
    temps = 0.5 + torch.rand(H, generator=g)
    if temp:
        q = q * temps.to(D)[:, None]
    if warmth:
        factor = P.query_warmth(pos.tolist(), *warmth)
        assert factor.unique().numel() > 2
        q = q * factor[:, None, None]
    q_out = torch.zeros(n, H * d, device=device)
    kc, vc = torch.zeros(9, G, ps, d, device=device), torch.zeros(9, G, ps, dv, device=device)
    slots = torch.tensor([p + 8 for p in pos.tolist()], dtype=torch.int32, device=device)
    kw = dict(warm_coef=warmth[0], warm_every=warmth[1]) if warmth else {}
    ops.qk_norm_rope_write(proj.to(device), pos.to(torch.int32).to(device), None, 0, None, None, eps, q_out, kc, vc, slots, H, G,
                           d, dv, ps, unit_norm=unit, q_head_scale=temps.to(device) if temp else None, **kw)
    torch.testing.assert_close(q_out.cpu(), q.reshape(n, -1).float(), atol=1e-5, rtol=1e-5)
    for i, s in enumerate(slots.tolist()):
        torch.testing.assert_close(kc[s // ps, :, s % ps].cpu(), k[i].float(), atol=1e-5, rtol=1e-5)
        assert torch.equal(vc[s // ps, :, s % ps].cpu(), v[i])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n", [1, 5, 40])
@pytest.mark.parametrize("experts,top,ff,shared", [(8, 2, 24, 40), (5, 1, 16, 8), (6, 6, 20, 16), (7, 3, 9, 11), (4, 2, 12, None)])
def test_experts_beside_a_shared_one(device, n, experts, top, ff, shared):
    """The weighted sum of the chosen experts and the shared expert's output as one list of slices: the router's
    scale multiplies the former alone, the weights are softmax scores over their sum, and a token's
    experts do not depend on its batch."""
    from inference_engine_b200.config.spec import PartSpec
    from inference_engine_b200.engine.workspace import Workspace
    from inference_engine_b200.parts.base import BuildEnv
    from inference_engine_b200.parts.registry import build_part

    g, hidden = torch.Generator().manual_seed(experts), 48
    params = {"router": "m.router", "expert_prefix": "m.e", "experts": experts, "top": top, "intermediate_size": ff,
              "weight_scale": 2.5, "limit": None, "alpha": 1.0, "up_offset": 0.0}
    if shared:
        params["shared"] = PartSpec("swiglu", {"gate_proj": "m.shared.gate", "up_proj": "m.shared.up",
                                               "down_proj": "m.shared.down", "intermediate_size": shared})
    env = BuildEnv(hidden, "float32", 16, {}, device)
    part = build_part("feed_forward", PartSpec("routed_experts", params), env)
    children = part.parts()
    decls = {**part.weights(), **(children[0].weights() if children else {})}
    W = {name: torch.randn(decl.shape, generator=g) / decl.shape[-1] ** 0.5 for name, decl in decls.items()}
    W["m.router"] *= 4.0
    for p in [part, *children]:
        p.bind({name: W[name].to(device) for name in p.weights()}, env)
    x = torch.randn(n, hidden, generator=g)
    mlp = {"router": {"experts": experts, "top": top, "scale": 2.5}, "expert": {"ff": ff}, "shared": shared and {"ff": shared}}
    W64 = {name: t.to(D) for name, t in W.items()}
    want = P.feed_forward_moe(W64, "m", x.to(D), mlp)
    got = part.forward(x.to(device), SimpleNamespace(ops=_ops(device), ws=Workspace(device)))
    assert got.dim() == 3 and got.shape[0] >= top + (1 if shared else 0)
    torch.testing.assert_close(got.sum(0).cpu(), want.float(), atol=2e-5, rtol=2e-5)
    if shared:
        alone = P.feed_forward_moe(W64, "m", x.to(D), dict(mlp, shared=None))
        assert (alone - want).abs().max() > 0.05  # (a shared expert that is left out shows)
        torch.testing.assert_close(got[:top].sum(0).cpu(), alone.float(), atol=2e-5, rtol=2e-5)


# --- long decoding and generation through the engine ------------------------------------------------


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    """400 tokens decoded one by one after a short prompt: states that run on, distances that pass every
    bucket, queries that warm up, pages that fill to the pool's last."""
    from inference_engine_b200.kernels import get_ops

    cfg = V.MIXED
    weights = V.make_weights(cfg, seed=3)
    toks = _requests(cfg, [410], seed=5)["r0"]
    want = P.forward(cfg, weights, toks, D).float()
    session = _session(tmp_path, cfg, weights, dtype, "cuda", get_ops("cuda"), 448, 16)
    got = H.collect(session, H.trace_decode_tail({"a": toks}, 400))["a"]
    _check({"a": got}, {"a": want}, dtype, "long decoding", _bound(tmp_path, dtype, cfg, weights, {"a": toks}, {"a": want}))


def _greedy_plain(cfg, weights, prompt, count):
    ids = list(prompt)
    for _ in range(count):
        ids.append(int(P.forward(cfg, weights, ids, D)[-1].argmax()))
    return ids[len(prompt):]


def _generate(cfg, weights, device, **kw):
    from inference_engine_b200 import SamplingParams
    from inference_engine_b200.engine.llm_engine import LLMEngine
    from inference_engine_b200.engine.loading import model_from_tensors

    model, _ = model_from_tensors(V.without_bucket_counts(cfg), weights, "float32", device, 128)
    engine = LLMEngine(model, None, (), num_blocks=48, block_size=8, max_num_seqs=3,
                       max_num_batched_tokens=16, debug_checks=True, **kw)
    prompts = {f"p{i}": _requests(cfg, [n], seed=90 + i)["r0"] for i, n in enumerate([5, 40, 23, 1, 31])}
    for rid, prompt in prompts.items():
        engine.add_request(rid, prompt, SamplingParams(max_tokens=10, temperature=0.0))
    got: dict[str, list[int]] = {rid: [] for rid in prompts}
    while engine.has_unfinished():
        for out in engine.step():
            got[out.request_id].append(out.token_id)
    engine.cache.check_invariants()
    assert engine.cache.slots.num_free == engine.cache.slots.num_slots
    return engine, prompts, got


def test_greedy_generation_on_the_plain_kernels():
    """The engine's own entry point and scheduler on the CPU stand-ins of the kernels."""
    from tests.ref_ops import RefOps

    cfg = V.STREAMS
    weights = V.make_weights(cfg, seed=4)
    _, prompts, got = _generate(cfg, weights, "cpu", ops=RefOps())
    for rid, prompt in prompts.items():
        assert got[rid] == _greedy_plain(cfg, weights, prompt, 10), rid


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "odd", "one_bucket"])
def test_greedy_generation_through_the_engine(name):
    """`LLMEngine` with the scheduler cutting prompts into portions and batching requests (three at
    a time, so slots and pages serve one request after another), decode steps captured and launched
    ahead: the tokens are the plain implementation's greedy choices."""
    cfg = V.CONFIGS[name]
    weights = V.make_weights(cfg, seed=4)
    engine, prompts, got = _generate(cfg, weights, "cuda")
    assert engine.graphs is not None  # decode steps are captured
    for rid, prompt in prompts.items():
        assert got[rid] == _greedy_plain(cfg, weights, prompt, 10), rid


CAPTURED = V.config(64, 89, [
    (V.retention(2, 32, 16, (0.95, 0.99), rot=16), V.moe(4, 2, 24, shared=32, scale=1.5)),
    (V.attention(4, 2, 16, 32), V.moe(6, 2, 16)),
    (V.attention_2(4, 1, 32, 16, 60, q_temp=(0.5, 16), scale=1.0, buckets=16), None),
    (V.retention(1, 64, 64, (0.98,)), V.moe(4, 1, 16, shared=16)),
], streams=2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_short_steps_with_portions(tmp_path, dtype):
    """Portions and mixed batches replayed through captured launch sequences (launched for bounds,
    padded with tokens that belong to no request and requests without tokens): in bfloat16 the
    retention's chunks and the tensor-core attention are sized by the token bound.  Against the plain
    implementation; in 32-bit equal bit for bit to the eagerly launched steps."""
    from inference_engine_b200.engine.graphs import DecodeGraphs, MixedGraphs
    from inference_engine_b200.kernels import get_ops

    cfg = CAPTURED
    weights = V.make_weights(cfg, seed=6)
    requests = _requests(cfg, [170, 45, 33, 90, 20, 60], seed=300)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, dtype, cfg, weights, requests, want)
    mixed, peak = H.trace_mixed(requests, seed=2, tail=6, max_portion=80)
    portions = H.trace_portions(requests, (7, 2, 100, 3, 2, 33, 5, 2, 16, 70))
    results = {}
    for captured in (True, False):
        for mode, (trace, room) in {"portions": (portions, 256), "mixed": (mixed, peak)}.items():
            session = _session(tmp_path / f"{mode}{captured}", cfg, weights, dtype, "cuda", get_ops("cuda"), room, 8)
            if captured:
                graphs = MixedGraphs(DecodeGraphs(session.runner, 256, max(64, -(-room // 8))))
                eager = session.runner.step
                session.runner.step = lambda entries, g=graphs, e=eager: g.run(entries) if g.can_run(entries) else e(entries)
            got = H.collect(session, trace)
            _check(got, want, dtype, f"captured={captured} {mode}", tol)
            if captured:
                assert graphs.replays > len(requests)
            results[(captured, mode)] = got
    if dtype == "float32":
        for mode in ("portions", "mixed"):
            for rid in requests:
                assert torch.equal(results[(True, mode)][rid], results[(False, mode)][rid]), (mode, rid)
    get_ops("cuda").check_errors()


@pytest.mark.gpu
def test_captured_decoding_in_bfloat16(tmp_path):
    """Decode steps through captured launch sequences with padding rows (buckets larger than the batch), after
    prompts run eagerly: the retention's step kernel and the cut attention against the plain implementation."""
    from inference_engine_b200.engine.graphs import DecodeGraphs
    from inference_engine_b200.kernels import get_ops

    cfg = CAPTURED
    weights = V.make_weights(cfg, seed=6)
    requests = _requests(cfg, [80, 33, 64], seed=500)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, "bfloat16", cfg, weights, requests, want)
    session = _session(tmp_path, cfg, weights, "bfloat16", "cuda", get_ops("cuda"), 256, 8)
    graphs = DecodeGraphs(session.runner, 4, 64)
    eager = session.runner.step
    session.runner.step = lambda entries: (graphs.run(entries) if all(len(e.tokens) == 1 for e in entries)
                                           else eager(entries))
    tail, steps = 20, []
    heads = {rid: len(toks) - tail for rid, toks in requests.items()}
    steps.append({"step": 0, "entries": [{"id": rid, "tokens": toks[: heads[rid]], "want": list(range(heads[rid]))}
                                         for rid, toks in requests.items()], "end": []})
    for i in range(tail):
        steps.append({"step": i + 1, "entries": [{"id": rid, "tokens": [toks[heads[rid] + i]], "want": [0]}
                                                 for rid, toks in requests.items()], "end": []})
    got = H.collect(session, steps)
    _check(got, want, "bfloat16", "captured decoding", tol)
    get_ops("cuda").check_errors()


def test_tables_by_position_are_as_long_as_a_request_can_get():
    """The model has no position limit of its own: its rotation tables are made for the engine's longest request
    (or what its pages hold), and for 131,072 positions where nothing says more."""
    from inference_engine_b200.config.engine_config import EngineConfig
    from inference_engine_b200.engine.loading import random_model

    assert EngineConfig(num_blocks=6, block_size=8).most_positions == 48
    assert EngineConfig(num_blocks=6, block_size=8, max_model_len=20).most_positions == 20
    assert EngineConfig().most_positions is None
    for asked, rows in ((48, 48), (None, 1 << 17)):
        model, _ = random_model(V.MIXED, dtype="float32", device="cpu", max_positions=asked)
        assert model.blocks[0].mixer.position.rotary_table().shape == (rows, 2, 4)
