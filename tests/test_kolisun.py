"""The Kolisun design in the engine against the plain whole-sequence implementation
(`tests/plain_kolisun.py`): whole prompts, token-by-token decoding, portions down to two tokens, mixed
batches with pages and slots used again, configurations of odd sizes; every mechanism alone against its
plain function, with inputs made so that a key far away, a window's edge that is one token off, a sink that is
left out or a lost state shows; on the CPU through the plain stand-ins of the kernels, on the GPU through the
kernels in both precisions; long decoding; greedy generation through the engine's own entry point and
scheduler."""

from __future__ import annotations

import math
from types import SimpleNamespace

import pytest
import torch

from tests import helpers as H
from tests import kolisun_configs as V
from tests import plain_kolisun as P

LENGTHS = [50, 21, 37, 64, 9, 1]
# (under these names the run's summary lists this file's comparisons: their bounds are measured)
LABEL = {"float32": "float32, Kolisun", "bfloat16": "bfloat16, Kolisun"}
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
D = torch.float64


def _requests(cfg, lengths=LENGTHS, seed=700):
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed + i)).tolist()
            for i, n in enumerate(lengths)}


def _want(cfg, weights, requests):
    return {rid: P.logits_for(cfg, weights, toks, D).float() for rid, toks in requests.items()}


def _float32_bound(cfg, weights, requests, want) -> dict:
    """Three times what rounding alone does to the plain implementation when it runs in 32-bit
    instead of 64-bit, and never below the engine's fixed bound for tiny models."""
    worst = max(float((P.logits_for(cfg, weights, toks, torch.float32) - want[rid]).abs().max())
                for rid, toks in requests.items())
    return dict(atol=max(3 * worst, H.TOL["float32"]["atol"]), rtol=H.TOL["float32"]["rtol"])


def _position_errors(got, want):
    """Per position, over all requests: the root mean square of the difference over that of the logits."""
    err = [(got[rid].double() - want[rid].double()).pow(2).mean(-1).sqrt() / want[rid].double().pow(2).mean(-1).sqrt()
           for rid in want]
    return torch.cat(err)


def _bfloat16_bound(tmp_path, cfg, weights, requests, want) -> dict:
    """From the same requests on the plain stand-ins of the kernels run in bfloat16 (activations rounded
    between the parts, as the kernels round them): no position may be off by more than twice the worst one
    there, and hardly more positions than there by more than three times the median.  (A sublayer's output
    that nearly cancels is magnified by its norm, its rounding with it, so a few positions stand out.)"""
    from tests.ref_ops import RefOps

    room = sum(H.round64(len(t)) for t in requests.values())
    got = H.collect(_session(tmp_path / "bound", cfg, weights, "bfloat16", "cpu", RefOps(), room, 16),
                    H.trace_whole(requests))
    err = _position_errors(got, want)
    bound = max(3 * float(err.median()), 0.03)
    assert bound < 0.1 and float(err.max()) < 0.2, "the test weights magnify rounding so much that a fault would hide in it"
    return dict(usual=bound, share=float((err > bound).float().mean()), most=max(2 * float(err.max()), bound))


def _bound(tmp_path, dtype, cfg, weights, requests, want):
    return (_float32_bound(cfg, weights, requests, want) if dtype == "float32"
            else _bfloat16_bound(tmp_path, cfg, weights, requests, want))


def _check(got, want, dtype, what, tol) -> None:
    if dtype == "float32":
        for rid in want:
            H.assert_close(got[rid], want[rid], LABEL[dtype], f"{what} {rid}", tol)
        return
    assert all(got[rid].shape == want[rid].shape and bool(torch.isfinite(got[rid]).all()) for rid in want), what
    err = _position_errors(got, want)
    share, allowed = float((err > tol["usual"]).float().mean()), 2 * tol["share"] + 0.02
    H._record(LABEL[dtype], max_pos_rel_rms=float(err.max()), max_median_pos_rel_rms=float(err.median()), max_share_beyond=share)
    assert float(err.max()) <= tol["most"], (what, float(err.max()), tol)
    assert share <= allowed, (what, share, tol)


def _session(tmp_path, cfg, weights, dtype, device, ops, max_tokens, page_size):
    from inference_engine_b200.engine.replay import ReplaySession

    folder = H.write_model_dir(tmp_path / f"m{abs(hash(str(cfg))) % 10**8}", cfg, weights)
    return ReplaySession(folder, dtype, max_tokens, device=device, ops=ops, page_size=page_size)


def _given_back(session):
    assert session.cache.num_free_pages == [p.num_pages for p in session.cache.pools]
    assert session.cache.slots.num_free == session.cache.slots.num_slots


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
        _check(got, want, dtype, f"kolisun {name} {mode}", tol)
        _given_back(session)
        results[mode] = got
    return results


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
    """Prompts of hundreds of tokens over several chunks of the recurrence, many tiles and pages of 16,
    sizes that reach the tensor-core and fused kernels in bfloat16."""
    from inference_engine_b200.kernels import get_ops

    cfg = V.WIDE
    weights = V.make_weights(cfg, seed=21)
    requests = _requests(cfg, [420, 130, 257, 64], seed=900)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, dtype, cfg, weights, requests, want)
    mixed, peak = H.trace_mixed(requests, seed=8, tail=20, max_portion=90)
    room = sum(H.round64(len(t)) for t in requests.values())
    names = ("sink_attention_mma", "latent_attention_mma", "headwise_mma", "state_space_step", "state_space_chunks")
    before = {n: get_ops("cuda").launch_counts.get(n, 0) for n in names}
    results = {}
    for mode, (trace, space) in {"whole": (H.trace_whole(requests), room),
                                 "tail": (H.trace_decode_tail(requests, 40), room),
                                 "portions": (H.trace_portions(requests, (70, 2, 129, 3, 64, 33)), room),
                                 "mixed": (mixed, peak)}.items():
        session = _session(tmp_path / mode, cfg, weights, dtype, "cuda", get_ops("cuda"), space, 16)
        results[mode] = H.collect(session, trace)
        _check(results[mode], want, dtype, f"wide {mode}", tol)
        _given_back(session)
    ran = {n: get_ops("cuda").launch_counts.get(n, 0) - before[n] for n in names}
    if dtype == "float32":
        assert not any(ran.values())
        for mode in ("tail", "portions", "mixed"):
            for rid in requests:
                assert torch.equal(results["whole"][rid], results[mode][rid]), (mode, rid)
    else:
        assert all(ran.values()), ran
    get_ops("cuda").check_errors()


def test_the_plain_model_shows_what_the_comparisons_look_for():
    """With the test weights a window that is one token off, a sink that is left out, a state that is lost between
    portions or a convolution that forgets moves the logits by far more than any bound above."""
    cfg = V.MIXED
    weights = V.make_weights(cfg, seed=11)
    toks = _requests(cfg, [60])["r0"]
    want = P.logits_for(cfg, weights, toks)
    size = want.pow(2).mean(-1).sqrt()

    def off(changed_cfg=cfg, changed=None):
        got = P.logits_for(changed_cfg, {**weights, **(changed or {})}, toks)
        return float(((got - want).pow(2).mean(-1).sqrt() / size)[20:].median())

    def mixer(i, **parts):
        layers = [dict(layer) for layer in cfg["layers"]]
        layers[i] = dict(layers[i], mixer={**layers[i]["mixer"], **parts})
        return dict(cfg, layers=layers)

    left = cfg["layers"][0]["mixer"]["left"]
    assert off(mixer(0, left=dict(left, mask={"size": left["mask"]["size"] + 1}))) > 0.03
    assert off(changed={"l1.mix.sink": torch.full((3,), -1e4)}) > 0.03
    assert off(mixer(0, left_scale=1.0)) > 0.03 and off(mixer(0, right_scale=1.0)) > 0.03
    assert off(changed={"l0.mix.right.A_log": torch.full((6,), 8.0)}) > 0.03  # (nothing is remembered)
    unscaled = dict(left, rot=dict(left["rot"], scaling=None))
    assert off(mixer(0, left=unscaled)) > 0.01


# --- what the model is made of ---------------------------------------------------------------------


def test_layout_of_the_model_and_its_caches():
    from inference_engine_b200.config import build_model_spec, config_from_dict
    from inference_engine_b200.engine.model import Model

    model = Model(build_model_spec(config_from_dict(V.MIXED)), "float32", 64)
    assert [type(b).__name__ for b in model.blocks] == ["SandwichResidualBlock"] * 4
    assert [type(b.mixer).__name__ for b in model.blocks] == ["ParallelSum", "LatentAttention", "LatentAttention", "ParallelSum"]
    assert [type(b.feed_forward).__name__ for b in model.blocks] == ["SwiGLU", "NoneType", "SwiGLU", "NoneType"]
    for b in model.blocks:
        assert type(b.norms["pre_mixer"]).__name__ == "NoNorm" and type(b.norms["post_mixer"]).__name__ == "RMSNorm"
    first, last = model.blocks[0].mixer, model.blocks[3].mixer
    assert first.joined and [type(b).__name__ for b in first.branches] == ["SinkAttention", "StateSpace"]
    assert [b.output_scale for b in first.branches] == [0.7, 1.3] and [b.output_scale for b in last.branches] == [1.0, 1.0]
    assert first.branches[0].position.layout == "interleaved" and first.branches[0].position.rotary_dim == 8
    assert first.branches[1].norm_parts == 4 and first.branches[1].groups == 2 and last.branches[1].taps == 2
    latent, plain = model.blocks[1].mixer, model.blocks[2].mixer
    assert latent.q_rank == 28 and "gate" not in latent.names and "sink" in latent.names and not latent.interleaved
    assert latent.position.scaling["kind"] == "yarn" and plain.position.scaling is None and plain.scale == 0.4
    groups = sorted((g.num_kv_heads, g.head_dim, g.value_dim, g.window or 0, g.num_layers) for g in model.paged_groups)
    assert groups == [(1, 32, 0, 0, 1), (1, 36, 0, 0, 1), (2, 12, 20, 9, 1), (4, 16, 8, 13, 1)]
    assert sorted((g.shape, g.num_layers) for g in model.state_groups) == [
        ((4 * 20 * 8 + (80 + 64),), 1), ((6 * 8 * 12 + 3 * (48 + 48),), 1)]
    for name, raw in V.ALL_CONFIGS.items():
        declared = Model(build_model_spec(config_from_dict(raw)), "float32", 64).declared_weights()
        assert {n: d.shape for n, d in declared.items()} == V.tensor_shapes(raw), name


def test_layers_with_equal_rotations_share_a_table():
    from inference_engine_b200.config import build_model_spec, config_from_dict

    a = V.latent(2, 8, 8, 8, 16, 8, scaling=V.yarn(4.0, 32, 8.0, 1.0))
    b = V.latent(2, 8, 8, 8, 16, 8, scaling=V.yarn(4.0, 64, 8.0, 1.0))
    spec = build_model_spec(config_from_dict(V.config(32, 17, [(a, None), (b, None), (a, None)])))
    assert len(spec.positions) == 2
    assert spec.layers[0].mixer.params["position"] == spec.layers[2].mixer.params["position"]


@pytest.mark.parametrize("name", list(V.ALL_CONFIGS))
def test_footprint_formula_counts_what_the_model_declares(name):
    from inference_engine_b200.architectures.kolisun import kolisun_footprint
    from inference_engine_b200.config import build_model_spec, config_from_dict
    from inference_engine_b200.engine.model import Model

    cfg = config_from_dict(V.ALL_CONFIGS[name])
    assert kolisun_footprint(cfg) == Model(build_model_spec(cfg), "float32", 64).footprint()


def test_configuration_errors():
    from inference_engine_b200.config import ConfigError, config_from_dict

    layers = V.MIXED["layers"]

    def changed(i, **mixer):
        return dict(V.MIXED, layers=[dict(layers[i], mixer=dict(layers[i]["mixer"], **mixer))])

    def side(which, **sizes):
        return changed(0, **{which: dict(layers[0]["mixer"][which], **sizes)})

    rot = layers[1]["mixer"]["rot"]
    for raw, match in [
            (dict(V.MIXED, layers=[dict(layers[0], type="other")]), "type"), (dict(V.MIXED, layers=[]), "layers"),
            ({k: v for k, v in V.MIXED.items() if k != "norm"}, "eps"), (dict(V.MIXED, vocab=0), "vocab_size"),
            (dict(V.MIXED, layers=[dict(layers[0], mlp={"kind": "moe"})]), "dense"),
            (dict(V.MIXED, layers=[dict(layers[0], mlp={"kind": "dense", "ff": 0})]), "ff"),
            (changed(1, kv_rank=None), "kv_rank"), (changed(1, q_rank=0), "q_rank"), (changed(1, scale=None), "scale"),
            (changed(1, rot=dict(rot, dims=10)), "rot"), (changed(1, rot=dict(rot, dims=3)), "rot"),
            (changed(1, rot=dict(rot, base=0)), "base"), (changed(1, rot=dict(rot, scaling={"factor": 2.0})), "original"),
            (changed(1, rot=dict(rot, base=1.0)), "base"),
            (side("left", kv_heads=4), "kv_heads"), (side("left", mask={"size": 0}), "mask"), (side("left", vdim=0), "vdim"),
            (side("right", groups=4), "groups"), (side("right", norm_groups=5), "norm_groups"), (side("right", conv=0), "conv"),
            (changed(0, right_scale=None), "right_scale")]:
        with pytest.raises(ConfigError, match=match):
            config_from_dict(raw)


def test_parts_refuse_what_does_not_go_together():
    from inference_engine_b200.config.spec import PartSpec
    from inference_engine_b200.parts.base import BuildEnv
    from inference_engine_b200.parts.registry import build_part

    env = BuildEnv(16, "float32", 8, {})
    names = {"q": "q", "dkv": "d", "latent_norm": "n", "uk": "k", "uv": "v", "o": "o"}
    sizes = dict(heads=2, dim=4, rot_dim=0, vdim=4, kv_rank=8, scale=1.0, eps=1e-5)
    for extra, more in (({"q_rank": 4}, {}), ({}, {"dq": "x", "dq_norm": "y", "uq": "z"})):
        with pytest.raises(ValueError, match="latent"):
            build_part("mixer", PartSpec("latent_attention", {"names": {**names, **more}, **sizes, **extra}), env)
    attn = {"names": {k: k for k in ("q", "k", "v", "o", "q_norm")}, "heads": 2, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0}
    with pytest.raises(ValueError, match="together"):
        build_part("mixer", PartSpec("sink_attention", attn), env)
    attn["names"]["k_norm"] = "k_norm"
    with pytest.raises(ValueError, match="norms over all heads"):
        build_part("mixer", PartSpec("sink_attention", {**attn, "unit_qk": True}), env)
    space = {"names": {}, "heads": 3, "vdim": 4, "state": 4, "groups": 2, "taps": 2, "eps": 1e-5}
    with pytest.raises(ValueError, match="groups"):
        build_part("mixer", PartSpec("state_space", space), env)
    with pytest.raises(ValueError, match="equal parts"):
        build_part("mixer", PartSpec("state_space", {**space, "groups": 1, "norm_parts": 5}), env)
    with pytest.raises(ValueError, match="llama3"):
        build_part("position", PartSpec("rotary", {"rotary_dim": 4, "theta": 10.0, "scaling": {"kind": "yarn"}}), env)


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
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    seq = [i for i, n in enumerate(lens) for _ in range(n)]
    pos = [s + t for s, n in zip(starts, lens) for t in range(n)]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    return SimpleNamespace(num_tokens=cu[-1], num_seqs=len(lens), seq_of_token=i32(seq), positions=i32(pos), cu_q=i32(cu),
                           q_starts=cu[:-1], q_lens=list(lens), start_positions=list(starts), max_q_len=max(lens),
                           ctx_lens=i32([s + n for s, n in zip(starts, lens)]), bounds=None, padded=False,
                           slots=i32(slots if slots is not None else list(range(len(lens)))), ws=ws)


def _paged(x, page_size, pages_total, order, device):
    """Rows [T, G, d] into a cache [pages, G, page_size, d] at the pages `order` names."""
    T, G, d = x.shape
    cache = torch.full((pages_total + 1, G, page_size, d), 9.0, device=device)  # (unused rows hold nonsense)
    for t in range(T):
        cache[order[t // page_size], :, t % page_size] = x[t].to(device)
    return cache


def _table(freqs, positions=64, amplitude=1.0):
    ang = torch.arange(positions, dtype=D)[:, None] * freqs
    return (torch.stack((ang.cos(), ang.sin()), dim=1) * amplitude).float()


SCALINGS = [("llama3", V.llama3(8.0, 1.0, 4.0, 8192)), ("llama3", V.llama3(4.0, 1.0, 4.0, 64)), ("llama3", V.llama3(2.0, 1.5, 1.5, 100)),
            ("llama3", V.llama3(32.0, 0.01, 0.02, 16)), ("yarn", V.yarn(4.0, 32, 8.0, 1.0)), ("yarn", V.yarn(40.0, 4096, 32.0, 1.0)),
            ("yarn", V.yarn(2.0, 100, 1e6, 1e5)), ("yarn", V.yarn(16.0, 1e7, 4.0, 0.5)), ("yarn", V.yarn(1.0, 512, 32.0, 1.0)),
            ("yarn", V.yarn(8.0, 300, 3.0, 3.0)), (None, None)]


@pytest.mark.parametrize("kind,scaling", SCALINGS)
@pytest.mark.parametrize("dims,base", [(2, 10000.0), (16, 1e6), (64, 500.0), (10, 3.0)])
def test_frequencies_and_tables(kind, scaling, dims, base):
    """The 32-bit table the kernels read against the plain formulas in 64-bit: frequencies kept, divided and between,
    ramps that start at once, end late or have no length, and the factor of cos and sin."""
    from inference_engine_b200.parts.base import BuildEnv
    from inference_engine_b200.parts.position import RotaryEncoding

    freqs, amplitude = P.base_frequencies(dims, base), 1.0
    given = scaling
    if kind == "yarn":
        freqs, amplitude = P.yarn(freqs, dims, base, scaling)
        given = {"kind": "yarn", **scaling}
        assert (amplitude == 1.0) == (scaling["factor"] == 1.0)
    elif kind == "llama3":
        freqs = P.by_wavelength(freqs, scaling)
        given = {"factor": scaling["factor"], "low_freq_factor": scaling["low"], "high_freq_factor": scaling["high"],
                 "original_max_position_embeddings": scaling["original"]}
    enc = RotaryEncoding(dims, base, given, 3000, "interleaved", "float64")
    enc.bind({}, BuildEnv(8, "float32", 3000, {}, "cpu"))
    torch.testing.assert_close(enc.rotary_table(), _table(freqs, 3000, amplitude), atol=1e-6, rtol=1e-6)


def test_the_scalings_differ_where_they_should():
    f = P.base_frequencies(64, 10000.0)
    scaled = P.by_wavelength(f, V.llama3(8.0, 1.0, 4.0, 1024))
    ratio = scaled / f
    assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / 8) < 1e-12 and bool(((ratio < 0.99) & (ratio > 0.13)).any())
    ramped, amplitude = P.yarn(f, 64, 10000.0, V.yarn(8.0, 1024, 32.0, 1.0))
    ratio = ramped / f
    assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / 8) < 1e-12 and bool(((ratio < 0.99) & (ratio > 0.13)).any()) and amplitude > 1.2


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,rot,interleaved", [(6, 2, 12, 20, 8, True), (4, 4, 32, 16, 32, True), (3, 1, 10, 7, 10, True),
                                                      (8, 2, 64, 64, 48, False), (5, 5, 6, 11, 4, False), (16, 4, 128, 96, 128, True),
                                                      (2, 1, 16, 8, 0, True), (40, 8, 256, 32, 64, True)])
def test_norms_over_all_heads_before_the_rotation(device, dtype, H, G, d, dv, rot, interleaved):
    """Biases, one norm over all query columns and one over all key columns, heads, rotation, cache rows; values with
    their bias times a factor; columns of another map behind them are left alone.  A norm per head would show."""
    ops, g = _ops(device), torch.Generator().manual_seed(H * d)
    n, ps, eps, factor = 9, 4, 1e-3, 0.7
    size = (H + G) * d + G * dv
    proj = torch.randn(n, size + 8, generator=g) * (10.0 ** torch.linspace(-2, 2, n))[:, None]
    bias = torch.randn(size, generator=g)
    qw, kw = 0.5 + torch.rand(H * d, generator=g), 0.5 + torch.rand(G * d, generator=g)
    pos = torch.tensor([0, 1, 2, 3, 17, 18, 19, 5, 61])
    full = proj[:, :size].to(D) + bias.to(D)
    q = P.rms(full[:, : H * d], eps, qw.to(D)).view(n, H, d)
    k = P.rms(full[:, H * d: (H + G) * d], eps, kw.to(D)).view(n, G, d)
    per_head = P.rms(full[:, : H * d].reshape(n, H, d), eps, qw.to(D).view(H, d))
    if H > 1:
        assert (per_head - q).abs().max() > 0.1
    freqs = P.base_frequencies(rot, 30.0)
    place = lambda x: torch.stack([P.turn(torch.cat([x[i:i + 1].new_zeros(p, *x.shape[1:]), x[i:i + 1]]), freqs, interleaved)[-1]  # noqa: E731
                                   for i, p in enumerate(pos.tolist())])
    q, k = place(q), place(k)
    v = full[:, (H + G) * d:].view(n, G, dv) * factor
    td = getattr(torch, dtype)
    q_out = torch.zeros(n, H * d, device=device, dtype=td)
    kc, vc = torch.zeros(19, G, ps, d, device=device, dtype=td), torch.zeros(19, G, ps, dv, device=device, dtype=td)
    slots = torch.tensor([p + 8 for p in pos.tolist()], dtype=torch.int32, device=device)
    table = _table(freqs).to(device) if rot else None
    ops.qk_norm_rope_write(proj.to(device), pos.to(torch.int32).to(device), table, rot, qw.to(device), kw.to(device), eps,
                           q_out, kc, vc, slots, H, G, d, dv, ps, bias=bias.to(device), interleaved=interleaved,
                           norm_over="all", value_scale=factor)
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == "float32" else dict(atol=1e-2, rtol=1e-2)
    torch.testing.assert_close(q_out.float().cpu(), q.reshape(n, -1).float(), **tol)
    for i, s in enumerate(slots.tolist()):
        torch.testing.assert_close(kc[s // ps, :, s % ps].float().cpu(), k[i].float(), **tol)
        torch.testing.assert_close(vc[s // ps, :, s % ps].float().cpu(), v[i].float(), **tol)
    kept = kc.clone()
    ops.qk_norm_rope_write(-proj.to(device), pos.to(torch.int32).to(device), table, rot, qw.to(device), kw.to(device), eps,
                           q_out, kc, vc, None, H, G, d, dv, ps, interleaved=interleaved, norm_over="all")
    assert torch.equal(kc, kept)  # (a run that borrows a cache writes none; it had no bias either)
    want = place(P.rms(-proj[:, : H * d].to(D), eps, qw.to(D)).view(n, H, d)).reshape(n, -1).float()
    torch.testing.assert_close(q_out.float().cpu(), want, **tol)


def test_wide_norms_refuse_what_they_cannot_do():
    if not torch.cuda.is_available():
        from inference_engine_b200.kernels.cuda_ops import CudaOps, KernelError

        with pytest.raises(KernelError, match="no norm over"):
            CudaOps.qk_norm_rope_write.__wrapped__(SimpleNamespace(), *[None] * 16, norm_over="some")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("window", [1, 7, 16, 40, 64, 65])
def test_window_edges(device, window):
    """Every third query has one key of large score, placed just inside or just outside its window; portions and single
    tokens over scattered pages of 4; the result is some columns of a wider array.  An edge that is one
    position off is checked to show."""
    ops, g = _ops(device), torch.Generator().manual_seed(window)
    T, H, G, d, dv, ps = 90, 4, 2, 12, 20, 4
    k, q = torch.randn(T, G, d, generator=g) * 0.3, torch.randn(T, H, d, generator=g) * 0.3
    for t in range(0, T, 3):
        target = max(t - window + (1 if t % 2 else 0), 0)  # inside / one too far
        k[target, :, t % d] += 1.0
        q[t, :, t % d] += 4.0
    v = torch.randn(T, G, dv, generator=g)
    scale = 0.7
    grouped = lambda x: x.to(D).repeat_interleave(H // G, dim=1)  # noqa: E731
    plain = lambda size: P.softmax_attention(q.to(D), grouped(k), grouped(v), scale, size)  # noqa: E731
    want = plain(window)
    for other in (window - 1, window + 1):
        if other:
            assert ((plain(other) - want)[window:].abs().amax((1, 2)) > 0.02).float().mean() > 0.2
    pages = -(-T // ps)
    order = torch.randperm(pages + 2, generator=g).tolist()[:pages]
    kc, vc = _paged(k, ps, pages + 2, order, device), _paged(v, ps, pages + 2, order, device)
    got, at = [], 0
    for n in [31, 1, 1, 2, 20, 1, 34]:
        # pages wholly behind the first query's window are gone
        table = [page if (i + 1) * ps > at - window + 1 else -1 for i, page in enumerate(order)]
        wide = torch.full((n, 6 + H * dv), 5.0, device=device)
        ops.sink_attention(q[at: at + n].reshape(n, -1).to(device).contiguous(), kc, vc,
                           torch.tensor([table], dtype=torch.int32, device=device), _ctx([n], [at], device), H, G, d, dv, ps,
                           scale, window, None, None, wide[:, 6:])
        got.append(wide[:, 6:].cpu().view(n, H, dv))
        assert bool((wide[:, :6] == 5.0).all())
        at += n
    torch.testing.assert_close(torch.cat(got), want.float(), atol=1e-4, rtol=1e-4)
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("d,dv,heads,kv", [(112, 80, 6, 3), (48, 32, 8, 2), (64, 128, 3, 3), (128, 16, 4, 1)])
@pytest.mark.parametrize("window", [1, 33, 64, 100, 257])
def test_window_edges_on_the_tensor_cores(d, dv, heads, kv, window):
    """The same in bfloat16: portions that start and end inside tiles of 64, single tokens whose window's keys are cut
    among blocks, results beside other columns."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(d + window)
    T, ps = 333, 16
    bf = lambda x: x.to(torch.bfloat16).float()  # noqa: E731
    k, q = torch.randn(T, kv, d, generator=g) * 0.3, torch.randn(T, heads, d, generator=g) * 0.3
    v = bf(torch.randn(T, kv, dv, generator=g))
    for t in range(0, T, 3):
        target = max(t - window + (1 if t % 2 else 0), 0)
        k[target, :, t % d] += 2.0
        q[t, :, t % d] += 5.0
    q, k = bf(q), bf(k)
    grouped = lambda x: x.to(D).repeat_interleave(heads // kv, dim=1)  # noqa: E731
    want = P.softmax_attention(q.to(D), grouped(k), grouped(v), 0.5, window).float()
    pages = -(-T // ps)
    order = torch.randperm(pages + 3, generator=g).tolist()[:pages]
    kc, vc = (_paged(x, ps, pages + 3, order, "cuda").to(torch.bfloat16) for x in (k, v))
    before = ops.launch_counts.get("sink_attention_mma", 0)
    got, at = [], 0
    portions = [70, 33, 1, 2, 5, 130, 1, 8, 83]
    for n in portions:
        table = [page if (i + 1) * ps > at - window + 1 else -1 for i, page in enumerate(order)]
        wide = torch.full((n, heads * dv + 12), 3.0, device="cuda", dtype=torch.bfloat16)
        ops.sink_attention(q[at: at + n].reshape(n, -1).to("cuda", torch.bfloat16), kc, vc,
                           torch.tensor([table], dtype=torch.int32, device="cuda"), _ctx([n], [at], "cuda"), heads, kv, d, dv,
                           ps, 0.5, window, None, None, wide[:, 4: 4 + heads * dv])
        got.append(wide[:, 4: 4 + heads * dv].float().cpu().view(n, heads, dv))
        assert bool((wide[:, :4] == 3.0).all() and (wide[:, 4 + heads * dv:] == 3.0).all())
        at += n
    ops.check_errors()
    assert ops.launch_counts.get("sink_attention_mma", 0) == before + len(portions)
    torch.testing.assert_close(torch.cat(got), want, atol=0.015, rtol=0.01)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("H,dim,rot,rank,q_rank,parts", [(3, 12, 8, 24, 28, 1), (2, 16, 16, 32, 12, 3), (5, 7, 6, 15, 11, 2),
                                                         (4, 32, 0, 48, 64, 1), (16, 128, 64, 512, 768, 8), (1, 48, 2, 20, 9, 5)])
def test_latent_input_stage(device, dtype, interleaved, H, dim, rot, rank, q_rank, parts):
    """The normalised latents of queries and keys, the turned key part in its cache row, gates; then the query rows: each
    head's key matrix on the unrotated part, the turned rotated part behind it.  Inputs whole and in parts."""
    from inference_engine_b200.engine.workspace import Workspace

    ops, g = _ops(device), torch.Generator().manual_seed(rank + parts)
    n, ps, eps, row = 11, 4, 1e-4, rank + rot
    td = getattr(torch, dtype)
    split = lambda t: t[None].repeat(parts, 1, 1) * torch.linspace(0.5, 1.5, parts)[:, None, None] / parts if parts > 1 else t  # noqa: E731
    proj = torch.randn(n, q_rank + row + H, generator=g) * (10.0 ** torch.linspace(-1, 1, n))[:, None]
    q = torch.randn(n, H * (dim + rot), generator=g)
    qw, cw = 0.5 + torch.rand(q_rank, generator=g), 0.5 + torch.rand(rank, generator=g)
    w = torch.randn(H, rank, dim, generator=g).to(td).float() / dim ** 0.5
    pos = torch.tensor([0, 1, 2, 3, 17, 18, 19, 5, 6, 7, 60])
    freqs, amplitude = P.base_frequencies(rot, 50.0), 1.3
    turn = lambda x: torch.stack([P.turn(torch.cat([x[i:i + 1].new_zeros(p, *x.shape[1:]), x[i:i + 1]]), freqs, interleaved, amplitude)[-1]  # noqa: E731
                                  for i, p in enumerate(pos.tolist())])
    dev = lambda t: t.to(device)  # noqa: E731
    table = _table(freqs, 64, amplitude).to(device) if rot else None
    sizes = dict(heads=H, dim=dim, rot_dim=rot, rank=rank, page_size=ps, interleaved=interleaved)
    given = dev(split(proj))
    cache = torch.zeros(20, 1, ps, row, device=device, dtype=td)
    slots = dev(torch.tensor([p + 8 for p in pos.tolist()], dtype=torch.int32))
    cq_out, gate = torch.zeros(n, q_rank, device=device, dtype=td), torch.zeros(n, H, device=device)
    positions = dev(pos.to(torch.int32))
    ops.latent_prep(positions, table, rot, **sizes, eps=eps, cq=given[..., :q_rank], cq_norm_w=dev(qw), cq_out=cq_out,
                    dkv=given[..., q_rank: q_rank + row], norm_w=dev(cw), cache=cache, slot_mapping=slots,
                    gate_pre=given[..., q_rank + row:], gate=gate)
    tol = dict(atol=1e-4, rtol=1e-4) if dtype == "float32" else dict(atol=1e-2, rtol=1e-2)
    x = proj.to(D)
    torch.testing.assert_close(cq_out.float().cpu(), P.rms(x[:, :q_rank], eps, qw.to(D)).float(), **tol)
    torch.testing.assert_close(gate.cpu(), torch.sigmoid(x[:, q_rank + row:]).float(), atol=1e-5, rtol=1e-5)
    rows = torch.cat([P.rms(x[:, q_rank: q_rank + rank], eps, cw.to(D)), turn(x[:, None, q_rank + rank: q_rank + row])[:, 0]], dim=1)
    for i, s in enumerate(slots.tolist()):
        torch.testing.assert_close(cache[s // ps, 0, s % ps].float().cpu(), rows[i].float(), **tol)
    # queries, for few and for many tokens (the products of many go to the library in bfloat16)
    heads = q.to(D).view(n, H, dim + rot)
    plain = heads[..., :dim].to(td).to(D)
    want = torch.cat([torch.einsum("nhk,hok->nho", plain, w.to(D)), turn(heads[..., dim:])], dim=-1).reshape(n, -1).float()
    for times in (1, 4, 14):
        q_abs = torch.zeros(n * times, H * row, device=device, dtype=td)
        ops.latent_queries(dev(split(q.repeat(times, 1))), dev(w).to(td), q_abs, positions.repeat(times), table, rot, **sizes,
                           ws=Workspace(device))
        loose = dict(atol=2e-4, rtol=2e-4) if dtype == "float32" else dict(atol=4e-2, rtol=2e-2)
        torch.testing.assert_close(q_abs.float().cpu(), want.repeat(times, 1), **loose)
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("n", [1, 8, 9, 33, 100, 127, 128, 200])
@pytest.mark.parametrize("heads,o,k", [(3, 40, 48), (2, 64, 512), (5, 16, 16), (16, 128, 256), (1, 100, 1024), (4, 30, 20)])
def test_per_head_products(n, heads, o, k):
    """bfloat16, from and to strided views, with and without a factor per token and head; the result of a token is the same
    number in every batch that the same kernel takes."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(n + o)
    x_all = torch.randn(n, heads, k + 7, generator=g).to(torch.bfloat16).cuda()
    w = (torch.randn(heads, o, k, generator=g) / k ** 0.5).to(torch.bfloat16).cuda()
    scale = torch.rand(n, heads, generator=g).cuda()
    for first, factor in ((0, None), (3, scale)):
        out_all = torch.full((n, heads, o + 5), 2.0, device="cuda", dtype=torch.bfloat16)
        x = x_all[:, :, first: first + k]
        ops.headwise_linear(x, w, out_all[:, :, 5:], row_scale=factor)
        want = torch.einsum("nhk,hok->nho", x.double(), w.double())
        if factor is not None:
            want = want * factor.double()[..., None]
        torch.testing.assert_close(out_all[:, :, 5:].float(), want.float(), atol=2e-2, rtol=1e-2)
        assert bool((out_all[:, :, :5] == 2.0).all())
        if 8 < n < 128:
            again = torch.zeros(n - 1, heads, o, device="cuda", dtype=torch.bfloat16)
            ops.headwise_linear(x[1:], w, again, row_scale=None if factor is None else factor[1:].contiguous())
            assert torch.equal(again, out_all[1:, :, 5:])


def _latent_case(g, T, H, dk, dv, cast):
    """Queries and shared rows [T, ...] in which every third query has a key of large score, near, far or its own; sinks of
    the scores' size that carry some rows."""
    rows, q = torch.randn(T, dk, generator=g) * 0.3, torch.randn(T, H, dk, generator=g) * 0.3
    for t in range(0, T, 3):
        target = [0, t // 2, max(t - 1, 0), t][(t // 3) % 4]
        rows[target, t % dk] += 2.0
        q[t, :, t % dk] += 4.0
    sinks = torch.linspace(-2.0, 4.0, H)
    return cast(q), cast(rows), sinks


@pytest.mark.parametrize("device", DEVICES)
def test_latent_attention_with_a_sink(device):
    """Values that are the first entries of the shared rows, scattered pages of 4, portions and single tokens; a sink
    that is left out, scaled or counted twice shows."""
    ops, g = _ops(device), torch.Generator().manual_seed(6)
    T, H, dk, dv, ps, scale = 45, 5, 14, 9, 4, 0.6
    q, rows, sinks = _latent_case(g, T, H, dk, dv, lambda x: x)
    many = lambda x: x.to(D)[:, None].expand(T, H, x.shape[-1])  # noqa: E731
    plain = lambda s: P.softmax_attention(q.to(D), many(rows), many(rows[:, :dv]), scale, sinks=s)  # noqa: E731
    want = plain(sinks.to(D))
    for other in (None, sinks.to(D) * scale, sinks.to(D) + math.log(2.0)):
        assert (plain(other) - want).abs().max() > 0.05
    order = torch.randperm(14, generator=g).tolist()[:12]
    cache = _paged(rows[:, None], ps, 14, order, device)
    tables = torch.tensor([order], dtype=torch.int32, device=device)
    for given, expect in ((sinks, want), (None, plain(None))):
        got, at = [], 0
        for n in [13, 1, 1, 2, 20, 1, 7]:
            out = torch.zeros(n, H * dv, device=device)
            ops.paged_attention(q[at: at + n].reshape(n, -1).to(device).contiguous(), cache, cache, tables, _ctx([n], [at], device),
                                H, 1, dk, ps, scale, 0, out, value_dim=dv, sinks=None if given is None else given.to(device))
            got.append(out.cpu().view(n, H, dv))
            at += n
        torch.testing.assert_close(torch.cat(got), expect.float(), atol=1e-4, rtol=1e-4)
    # value rows as long as the key rows
    out = torch.zeros(T, H * dk, device=device)
    ops.paged_attention(q.reshape(T, -1).to(device), cache, cache, tables, _ctx([T], [0], device), H, 1, dk, ps, scale, 0, out,
                        value_dim=dk, sinks=sinks.to(device))
    whole = P.softmax_attention(q.to(D), many(rows), many(rows), scale, sinks=sinks.to(D))
    torch.testing.assert_close(out.cpu().view(T, H, dk), whole.float(), atol=1e-4, rtol=1e-4)
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dk,dv,H", [(88, 72, 5), (576, 512, 16), (40, 24, 3), (128, 96, 20), (48, 48, 1), (296, 256, 7)])
def test_latent_attention_with_a_sink_on_the_tensor_cores(dk, dv, H):
    """bfloat16: 64 rows per block for portions, sixteen for steps of few tokens whose context is cut into ranges that a
    second kernel merges with the sink's term; a second request of one token in every step."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(dk)
    T, ps, scale = 333, 16, 0.4
    q, rows, sinks = _latent_case(g, T, H, dk, dv, lambda x: x.to(torch.bfloat16).float())
    many = lambda x: x.to(D)[:, None].expand(T, H, x.shape[-1])  # noqa: E731
    want = P.softmax_attention(q.to(D), many(rows), many(rows[:, :dv]), scale, sinks=sinks.to(D)).float()
    pages = -(-T // ps)
    order = torch.randperm(pages + 3, generator=g).tolist()[:pages]
    cache = _paged(rows[:, None], ps, pages + 3, order, "cuda").to(torch.bfloat16)
    cache[pages + 3] = 0.25  # the second request: one token on the scratch page
    tables = torch.tensor([order, [pages + 3] * pages], dtype=torch.int32, device="cuda")
    own = torch.sigmoid(torch.full((H,), 0.25 * dk * scale) - sinks)  # (its one key against the sink)
    before = ops.launch_counts.get("latent_attention_mma", 0)
    got, at = [], 0
    portions = [70, 33, 1, 2, 5, 130, 1, 8, 83]
    for n in portions:
        qq = torch.cat([q[at: at + n].reshape(n, -1), torch.ones(1, H * dk)]).to("cuda", torch.bfloat16)
        out = torch.zeros(n + 1, H * dv, device="cuda", dtype=torch.bfloat16)
        ops.paged_attention(qq, cache, cache, tables, _ctx([n, 1], [at, 0], "cuda"), H, 1, dk, ps, scale, 0, out, value_dim=dv,
                            sinks=sinks.cuda())
        got.append(out[:n].float().cpu().view(n, H, dv))
        torch.testing.assert_close(out[n].float().cpu().view(H, dv), (0.25 * own)[:, None].expand(H, dv), atol=3e-3, rtol=1e-2)
        at += n
    ops.check_errors()
    assert at == T and ops.launch_counts.get("latent_attention_mma", 0) == before + len(portions)
    torch.testing.assert_close(torch.cat(got), want, atol=0.012, rtol=0.01)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_of_the_latent_attention(dtype):
    """Single tokens and short portions at contexts of thousands of positions: each query's key of large score lies
    thousands of positions back, at a page's or tile's edge or among the first, and carries the result beside a sink."""
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(9)
    T, H, dk, dv, ps, scale, td = 4500, 4, 88, 72, 16, 0.5, getattr(torch, dtype)
    bf = lambda x: x.to(torch.bfloat16).float()  # noqa: E731
    rows, q = bf(torch.randn(T, dk, generator=g) * 0.3), torch.randn(T, H, dk, generator=g) * 0.3
    far = {T - 1: 3, T - 2: 1100, 4099: 4035, 4031: 64, 2500: 0, 70: 63, 3000: 15, 3001: 16}
    for i, (t, target) in enumerate(far.items()):  # (an entry of its own for every probe)
        q[:, :, 76 + i], rows[:, 76 + i] = 0.0, 0.0
        rows[target, 76 + i] = 3.0
        q[t, :, 76 + i] = 10.0
    q, rows, sinks = bf(q), bf(rows), torch.tensor([-1.0, 12.0, 14.0, 10.0])
    order = torch.randperm(-(-T // ps), generator=g).tolist()
    tables = torch.tensor([order], dtype=torch.int32, device="cuda")
    cache = _paged(rows[:, None], ps, len(order), order, "cuda").to(td)
    for t, target in far.items():
        for n in (1, 3):  # (the probe's query is the portion's last)
            first = t - n + 1
            out = torch.zeros(n, H * dv, device="cuda", dtype=td)
            ops.paged_attention(q[first: t + 1].reshape(n, -1).to("cuda", td), cache, cache, tables, _ctx([n], [first], "cuda"),
                                H, 1, dk, ps, scale, 0, out, value_dim=dv, sinks=sinks.cuda())
            s = torch.einsum("hd,td->ht", q[t].to(D), rows[: t + 1].to(D)) * scale
            p = torch.softmax(torch.cat([s, sinks.to(D)[:, None]], dim=1), dim=1)[:, : t + 1]
            assert float(p[0, target]) > 0.3
            want = (p @ rows[: t + 1, :dv].to(D)).float()
            tol = 2e-4 if dtype == "float32" else 0.01
            torch.testing.assert_close(out[-1].float().cpu().view(H, dv), want, atol=tol, rtol=tol)
    ops.check_errors()


# --- the state-space recurrence ------------------------------------------------------------------------


def _space(g, H, p, n, groups, taps):
    inner, channels = H * p, H * p + 2 * groups * n
    return SimpleNamespace(
        H=H, p=p, n=n, groups=groups, taps=taps, inner=inner, channels=channels,
        conv=torch.randn(channels, taps, generator=g) * 0.4 + 0.2, conv_b=torch.randn(channels, generator=g) * 0.3,
        dt_bias=torch.randn(H, generator=g) - 1.0, A_log=torch.linspace(-4.0, 1.5, H) if H > 1 else torch.tensor([-1.0]),
        skip=torch.randn(H, generator=g))


def _space_plain(s, rows, state, weight, parts, eps, rounded):
    """One request's rows of the projection from its state: (normalised result, state afterwards), in 64-bit.  `rounded`:
    the convolved values pass through bfloat16, as they do there."""
    T, H, p, n = rows.shape[0], s.H, s.p, s.n
    matrix, tail = state[: s.inner * n].view(H, p, n).transpose(1, 2), state[s.inner * n:].view(s.taps - 1, s.channels)
    z, xbc, dt = rows.split([s.inner, s.channels, H], dim=1)
    seen = torch.cat([tail, xbc])
    xbc = P.silu(P.causal_conv(seen, s.conv.to(D), s.conv_b.to(D))[s.taps - 1:])
    if rounded:
        xbc = xbc.float().to(torch.bfloat16).to(D)
    x, b, c = xbc.split([s.inner, s.groups * n, s.groups * n], dim=1)
    x, b, c = x.view(T, H, p), b.view(T, s.groups, n), c.view(T, s.groups, n)
    group = torch.arange(H) // (H // s.groups)
    dt = P.softplus(dt + s.dt_bias.to(D))
    decay = torch.exp(-torch.exp(s.A_log.to(D)) * dt)
    S, y = matrix.clone(), []
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * b[t, group][:, :, None] * x[t][:, None, :]
        y.append(torch.einsum("hnp,hn->hp", S, c[t, group]) + s.skip.to(D)[:, None] * x[t])
    y = P.gated_group_norm(torch.stack(y).reshape(T, s.inner), z, weight.to(D), parts, eps)
    return y, torch.cat([S.transpose(1, 2).reshape(-1), seen[seen.shape[0] - (s.taps - 1):].reshape(-1)])


STEPS = [([1, 1, 3], [5, 0, 9]), ([8, 2], [0, 600]), ([150, 1, 64, 63, 65], [0, 100, 7, 3, 64]), ([300], [11]),
         ([2, 9], [64, 0]), ([65], [0]), ([1], [0]), ([16, 17, 2], [3, 0, 0])]
SPACES = [(6, 64, 128, 2, 4, 3), (4, 40, 48, 1, 3, 2), (3, 20, 12, 3, 2, 1), (5, 7, 9, 5, 6, 7), (2, 128, 128, 1, 4, 2), (4, 16, 16, 2, 1, 4),
          (1, 1, 1, 1, 2, 1), (8, 13, 20, 4, 4, 2), (2, 40, 144, 2, 4, 1), (2, 136, 24, 1, 3, 2)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,p,n,groups,taps,parts", SPACES)
def test_state_space_in_every_kind_of_step(device, dtype, H, p, n, groups, taps, parts):
    """Requests of one to hundreds of tokens in one step, from states and kept inputs that others left in scattered slots:
    results (some columns of a wider array, as the projection's are), the slots afterwards, and the slot that
    nobody owns.  Heads that forget at once and heads that hardly forget.  On the GPU in bfloat16 the fused kernels (a
    few tokens per request; chunks), for sizes beyond theirs and in 32-bit convolution, recurrence and norm by themselves."""
    from inference_engine_b200.engine.workspace import Workspace

    ops, g = _ops(device), torch.Generator().manual_seed(H * p + n)
    s, eps, td = _space(g, H, p, n, groups, taps), 1e-4, getattr(torch, dtype)
    weight = 0.5 + torch.rand(s.inner, generator=g)
    dev = lambda t: t.to(device)  # noqa: E731
    small = H * p * n < 4000
    for lens, starts in STEPS if small or device == "cuda" else STEPS[:2]:
        N, floats = sum(lens), s.inner * n + (taps - 1) * s.channels
        proj = torch.randn(N, s.inner + s.channels + H + 4, generator=g)
        state = torch.randn(len(lens) + 1, floats, generator=g)
        slots = torch.randperm(len(lens) + 1, generator=g).tolist()[: len(lens)]
        want, after, at = torch.zeros(N, s.inner, dtype=D), state.to(D).clone(), 0
        for length, slot in zip(lens, slots):
            rows = proj[at: at + length, : s.inner + s.channels + H].to(D)
            want[at: at + length], after[slot] = _space_plain(s, rows, state[slot].to(D), weight, parts, eps,
                                                             dtype == "bfloat16" and max(n, p) <= 128)
            at += length
        got_state, wide = state.clone().to(device), torch.full((N, s.inner + 10), 7.0, device=device, dtype=td)
        ctx = _ctx(lens, starts, device, slots)
        ops.state_space(dev(proj)[:, : s.inner + s.channels + H], ctx, dev(s.conv), dev(s.conv_b), dev(s.dt_bias), dev(s.A_log),
                        dev(s.skip), dev(weight), parts, eps, got_state, ctx.slots, wide[:, 8: 8 + s.inner], H, groups, n, p,
                        Workspace(device))
        tol = dict(atol=5e-4, rtol=5e-4) if dtype == "float32" else dict(atol=2e-2, rtol=2e-2)
        torch.testing.assert_close(wide[:, 8: 8 + s.inner].float().cpu(), want.float(), **tol)
        assert bool((wide[:, :8] == 7.0).all() and (wide[:, 8 + s.inner:] == 7.0).all())
        matrix = s.inner * n
        off = (got_state.cpu() - after)[:, :matrix].abs() / float(after[:, :matrix].abs().max())
        if dtype == "float32":
            assert float(off.max()) < 2e-5
        else:  # (a convolved value next to a rounding edge may round the other way: a row or a column of a state)
            assert float(off.max()) < 3e-3 and float(off.flatten().kthvalue(int(0.98 * off.numel())).values) < 5e-5
        assert torch.equal(got_state.cpu()[:, matrix:], after[:, matrix:].float())  # (the kept inputs are copies)
        idle = next(i for i in range(len(lens) + 1) if i not in slots)
        assert torch.equal(got_state.cpu()[idle], state[idle])
    ops.check_errors()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_space_remembers_its_first_token(device, dtype):
    """A mark that only the first token carries, read hundreds of tokens and several portions later through heads that
    hardly forget: a state or kept inputs lost between portions, chunks or steps show."""
    from inference_engine_b200.engine.workspace import Workspace

    ops, g = _ops(device), torch.Generator().manual_seed(2)
    s, T, eps = _space(g, 4, 16, 32, 2, 3), 290, 1e-5
    s.A_log, s.dt_bias = torch.full((4,), -9.0), torch.full((4,), -1.0)
    s.conv = torch.tensor([[0.2, 0.3, 1.0]]).repeat(s.channels, 1)
    s.conv_b.zero_()
    s.skip.zero_()
    weight, parts = torch.ones(s.inner), 1
    rows = torch.randn(T, s.inner + s.channels + 4, generator=g)
    b_at, c_at = 2 * s.inner, 2 * s.inner + 64
    rows[:, b_at: c_at] *= 0.02
    rows[:, [b_at, b_at + 32]] = -20.0  # (silu of it is nothing: entry 0 is written by the first token alone)
    rows[0, [b_at, b_at + 32]], rows[1:3, [b_at, b_at + 32]] = 8.0, -40.0
    rows[:, [c_at, c_at + 32]] = 6.0
    zero = torch.zeros(s.inner * s.n + 2 * s.channels, dtype=D)
    want, _ = _space_plain(s, rows.to(D), zero, weight, parts, eps, dtype == "bfloat16")
    lost, _ = _space_plain(s, rows[1:].to(D), zero, weight, parts, eps, dtype == "bfloat16")
    assert (lost - want[1:]).abs().amax(-1).min() > 0.3
    dev = lambda t: t.to(device)  # noqa: E731
    cuts = ([290], [1] * 12 + [70, 2, 130, 64, 8, 3, 1], [64, 64, 64, 64, 34], [200] + [1] * 90)
    for portions in cuts[1:2] if device == "cpu" else cuts:
        state, got, at = torch.zeros(2, zero.shape[0], device=device), [], 0
        for n in portions:
            ctx = _ctx([n], [at], device, [1])
            out = torch.zeros(n, s.inner, device=device, dtype=getattr(torch, dtype))
            ops.state_space(dev(rows[at: at + n]), ctx, dev(s.conv), dev(s.conv_b), dev(s.dt_bias), dev(s.A_log), dev(s.skip),
                            dev(weight), parts, eps, state, ctx.slots, out, s.H, s.groups, s.n, s.p, Workspace(device))
            got.append(out.float().cpu())
            at += n
        tol = dict(atol=1e-3, rtol=1e-3) if dtype == "float32" else dict(atol=3e-2, rtol=2e-2)
        torch.testing.assert_close(torch.cat(got), want.float(), **tol)


@pytest.mark.gpu
def test_state_space_in_32_bit_does_not_depend_on_the_cutting():
    from inference_engine_b200.engine.workspace import Workspace
    from inference_engine_b200.kernels import get_ops

    ops, g = get_ops("cuda"), torch.Generator().manual_seed(5)
    s = _space(g, 6, 24, 40, 3, 4)
    rows = torch.randn(130, s.inner + s.channels + 6, generator=g).cuda()
    args = [t.cuda() for t in (s.conv, s.conv_b, s.dt_bias, s.A_log, s.skip, torch.ones(s.inner))]
    results = []
    for portions in ([130], [1] * 20 + [2, 3, 50, 16, 16, 23], [16] * 8 + [2]):
        state, got, at = torch.zeros(1, s.inner * s.n + 3 * s.channels, device="cuda"), [], 0
        for n in portions:
            ctx = _ctx([n], [at], "cuda", [0])
            out = torch.zeros(n, s.inner, device="cuda")
            ops.state_space(rows[at: at + n], ctx, *args, 2, 1e-5, state, ctx.slots, out, s.H, s.groups, s.n, s.p, Workspace("cuda"))
            got.append(out)
            at += n
        results.append((torch.cat(got), state))
    for out, state in results[1:]:
        assert torch.equal(out, results[0][0]) and torch.equal(state, results[0][1])


# --- the stream and the sum of two mixers -----------------------------------------------------------


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [50, 72, 1100, 2048])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_stream_is_handed_on_as_it_is(device, width, dtype):
    """A sublayer's output (whole or in parts) normalised and added, the stream itself handed on in the compute dtype; the first
    reading, where nothing is pending; selected rows leave the stream alone."""
    from inference_engine_b200.engine.workspace import Workspace
    from inference_engine_b200.parts.norm import NoNorm, PostNorm, RMSNorm

    g, n, eps = torch.Generator().manual_seed(width), 7, 1e-4
    h, delta, w = (torch.randn(*shape, generator=g) for shape in ((n, width), (3, n, width), (width,)))
    td = getattr(torch, dtype)
    ctx = SimpleNamespace(ops=_ops(device), ws=Workspace(device))
    norm = RMSNorm("w", width, eps, td)
    norm.weight = w.to(device)
    part = NoNorm(width, td)
    for y in (delta, delta[0].contiguous()):
        total = y.to(D).sum(0) if y.dim() == 3 else y.to(D)
        want = (h.to(D) + P.rms(total, eps, w.to(D))).float()
        hd = h.clone().to(device)
        got = part.add_norm(hd, y.to(device), ctx, delta_post=PostNorm(norm))
        torch.testing.assert_close(hd.cpu(), want, atol=1e-5, rtol=1e-5)
        assert got.dtype == td and torch.equal(got.float().cpu(), hd.cpu().to(td).float())
        rows = torch.tensor([5, 0, 5], dtype=torch.int32, device=device)
        kept = hd.clone()
        got = part.add_norm(hd, y.to(device), ctx, rows=rows, delta_post=PostNorm(norm))
        again = (kept.cpu().to(D) + P.rms(total, eps, w.to(D))).float()[[5, 0, 5]]
        torch.testing.assert_close(got.float().cpu(), again.to(td).float(), atol=1e-5 if dtype == "float32" else 2e-2, rtol=1e-5)
        assert torch.equal(hd, kept)
    hd = h.clone().to(device)
    assert torch.equal(part.add_norm(hd, None, ctx).float().cpu(), h.to(td).float()) and torch.equal(hd.cpu(), h)
    with pytest.raises(ValueError, match="multiplier"):
        part.add_norm(hd, None, ctx, delta_scale=0.5)


@pytest.mark.parametrize("device", DEVICES)
def test_joined_branches_give_the_weighted_sum(device):
    """A sum whose branches share one product each against the same branches run one after the other and added: equal up to
    rounding, and so against the plain functions; factors that are swapped show."""
    from inference_engine_b200.config import build_model_spec, config_from_dict
    from inference_engine_b200.engine.loading import model_from_tensors
    from inference_engine_b200.engine.runner import make_runner
    from inference_engine_b200.engine.batch import StepEntry

    cfg = V.config(40, 31, [(V.parallel(V.attention(3, 1, 10, 6, 5, rot=4), V.recurrence(3, 6, 7, norm_groups=2, conv=3), 0.6, 1.7), None)])
    weights = V.make_weights(cfg, seed=8)
    toks = _requests(cfg, [17])["r0"]
    build_model_spec(config_from_dict(cfg))
    got = {}
    for joined in (True, False):
        model, _ = model_from_tensors(cfg, weights, "float32", device, 32)
        mixer = model.blocks[0].mixer
        assert mixer.joined and mixer.w_in.shape[0] % 4 == 0 and mixer.columns[1][0] % 4 == 0
        if not joined:  # (the same parts again, each with products of its own)
            mixer.joined = False
            for b in mixer.branches:
                b.products_elsewhere, b.output_scale, b.allow_split = False, 1.0, False
                b.bind({n: weights[n].to(device) for n in b.weights()}, model.env)
        runner = make_runner(model, _ops(device), device, 4, 8, 2, 32)
        runner.cache.add_request("a")
        runner.cache.grow("a", 0, len(toks))
        got[joined] = runner.step([StepEntry("a", toks, 0, list(range(len(toks))))]).float().cpu()
    want = P.logits_for(cfg, weights, toks).float()
    torch.testing.assert_close(got[True], want, atol=5e-5, rtol=1e-4)
    torch.testing.assert_close(got[False], want, atol=5e-5, rtol=1e-4)
    swapped = dict(cfg["layers"][0]["mixer"], left_scale=1.7, right_scale=0.6)
    other = P.logits_for(dict(cfg, layers=[dict(cfg["layers"][0], mixer=swapped)]), weights, toks).float()
    assert (other - want).abs().max() > 0.1


# --- long decoding, captured steps and generation through the engine --------------------------------


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding(tmp_path, name, dtype):
    """400 tokens decoded one by one after a short prompt: states that run on, windows that give pages back while the
    latent's pages fill to the pool's last."""
    from inference_engine_b200.kernels import get_ops

    cfg = V.ALL_CONFIGS[name]
    weights = V.make_weights(cfg, seed=3)
    toks = _requests(cfg, [410], seed=5)["r0"]
    want = P.logits_for(cfg, weights, toks, D).float()
    session = _session(tmp_path, cfg, weights, dtype, "cuda", get_ops("cuda"), 448, 16)
    steps = H.trace_decode_tail({"a": toks}, 400)
    steps[-1]["end"] = []
    got = H.collect(session, steps)["a"]
    _check({"a": got}, {"a": want}, dtype, "long decoding", _bound(tmp_path, dtype, cfg, weights, {"a": toks}, {"a": want}))
    for g, spec in enumerate(session.cache.paged_groups):
        table = session.cache.table(g, "a")
        held = [i for i, page in enumerate(table) if page >= 0]
        if spec.window is None:
            assert held == list(range(len(table)))
        else:  # (the next query's window is all that is kept)
            assert held[0] == max(410 - spec.window + 1, 0) // 16 and len(held) == len(table) - held[0]
    session.cache.free("a")
    _given_back(session)


def _greedy_plain(cfg, weights, prompt, count):
    ids = list(prompt)
    for _ in range(count):
        ids.append(int(P.logits_for(cfg, weights, ids, D)[-1].argmax()))
    return ids[len(prompt):]


def _generate(cfg, weights, device, **kw):
    from inference_engine_b200 import SamplingParams
    from inference_engine_b200.engine.llm_engine import LLMEngine
    from inference_engine_b200.engine.loading import model_from_tensors

    model, _ = model_from_tensors(cfg, weights, "float32", device, 128)
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

    weights = V.make_weights(V.MIXED, seed=4)
    _, prompts, got = _generate(V.MIXED, weights, "cpu", ops=RefOps())
    for rid, prompt in prompts.items():
        assert got[rid] == _greedy_plain(V.MIXED, weights, prompt, 10), rid


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "odd", "latent_only", "parallel_only"])
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
    (V.latent(4, 32, 16, 32, 64, 48, base=900.0, scaling=V.yarn(4.0, 64, 8.0, 1.0)), V.dense(64)),
    (V.parallel(V.attention(4, 2, 32, 16, 21, rot=32), V.recurrence(4, 32, 48, groups=2, norm_groups=2, conv=4), 0.8, 1.3), None),
    (V.parallel(V.attention(4, 1, 16, 32, 150), V.recurrence(2, 64, 16, conv=3), 1.1, 0.9), V.dense(48)),
])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_short_steps_with_portions(tmp_path, dtype):
    """Portions and mixed batches replayed through captured launch sequences (launched for bounds,
    padded with tokens that belong to no request and requests without tokens): in bfloat16 the
    recurrence's chunks and the tensor-core attentions are sized by the token bound.  Against the plain
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
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_decoding(tmp_path, dtype):
    """Decode steps through captured launch sequences with padding rows (buckets larger than the batch), after
    prompts run eagerly: the recurrence's step kernel, the cut attentions and their merges."""
    from inference_engine_b200.engine.graphs import DecodeGraphs
    from inference_engine_b200.kernels import get_ops

    cfg = CAPTURED
    weights = V.make_weights(cfg, seed=6)
    requests = _requests(cfg, [80, 33, 64], seed=500)
    want = _want(cfg, weights, requests)
    tol = _bound(tmp_path, dtype, cfg, weights, requests, want)
    session = _session(tmp_path, cfg, weights, dtype, "cuda", get_ops("cuda"), 256, 8)
    graphs = DecodeGraphs(session.runner, 4, 64)
    eager = session.runner.step
    session.runner.step = lambda entries: (graphs.run(entries) if all(len(e.tokens) == 1 for e in entries)
                                           else eager(entries))
    tail = 20
    heads = {rid: len(toks) - tail for rid, toks in requests.items()}
    steps = [{"step": 0, "entries": [{"id": rid, "tokens": toks[: heads[rid]], "want": list(range(heads[rid]))}
                                     for rid, toks in requests.items()], "end": []}]
    for i in range(tail):
        steps.append({"step": i + 1, "entries": [{"id": rid, "tokens": [toks[heads[rid] + i]], "want": [0]}
                                                 for rid, toks in requests.items()], "end": []})
    got = H.collect(session, steps)
    _check(got, want, dtype, "captured decoding", tol)
    get_ops("cuda").check_errors()
