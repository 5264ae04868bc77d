"""The Repolix decoder: its mechanisms one by one against `plain_repolix`, then whole models through the engine's step function,
scheduler and entry points.  The plain implementation shares nothing with the package; it runs in float64 on bfloat16-rounded
random weights."""
import ctypes
import math

import pytest
import torch

import plain_repolix as plain
import repolix_models
from helpers import assert_close, engine_model, run_portions, run_whole, write_model_folder
from test_gelulix import _state_steps              # launch helpers only (no test is imported)
from test_sopetar import _attend, _call, _meta, _pages, _rows_of

BF16 = dict(rmse=0.06, max=0.25, cosine=0.998)


def tokens_for(config, count, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, config["vocab"], (count,), generator=g).tolist()


def plain_logits(config, weights, tokens):
    return plain.forward(config, weights, tokens).float()


def close(got, want, dtype, what):
    """float32: every value.  bfloat16: row by row, and a few rows may be off altogether: where two experts' choice scores are nearly equal,
    the rounding of the router's input lets the choice fall the other way, and that row then differs by an expert's whole output, and with it
    the rows that a convolution's taps or a short window reach from there.  The float32 runs of the same tests allow no such row."""
    if dtype != "bfloat16":
        return assert_close(got, want, dtype, what)
    from helpers import row_metrics
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    m = row_metrics(got, want)
    bad = (m["rmse"] > BF16["rmse"]) | (m["max"] > BF16["max"]) | (m["cosine"] < BF16["cosine"])
    allowed = max(4, got.shape[0] // 10)
    assert int(bad.sum()) <= allowed, (f"{what}: {int(bad.sum())} of {bad.numel()} rows are off (a router's close calls explain up to {allowed}); "
                                       f"worst: rmse {m['rmse'].max():.4f}, max {m['max'].max():.4f}, cosine {m['cosine'].min():.6f}")


# ----------------------------------------------------------------------------- without a GPU
def test_config_and_plan_name_every_tensor():
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dict, plan_for
    from mini_llm_runtime_b200.engine.structure import expected_weights
    for name in repolix_models.ALL:
        config = repolix_models.get(name)
        weights = repolix_models.random_weights(config, 1)
        expected = expected_weights(plan_for(config_from_dict(config)))
        assert set(expected) == set(weights), name
        for key, spec in expected.items():
            assert tuple(spec.shape) == tuple(weights[key].shape), key


def test_ranks_come_from_the_stored_tensors(tmp_path):
    """A configuration that does not name the ranks of the low-rank products takes them from the weights' shapes."""
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dir, plan_for
    from mini_llm_runtime_b200.engine.structure import expected_weights
    config = repolix_models.get("small_a")
    weights = repolix_models.random_weights(config, 1)
    for layer in config["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    write_model_folder(str(tmp_path), config, weights)
    expected = expected_weights(plan_for(config_from_dir(str(tmp_path))))
    assert {k: tuple(s.shape) for k, s in expected.items()} == {k: tuple(t.shape) for k, t in weights.items()}


@pytest.mark.parametrize("path,value,message", [
    (("width",), None, "width"),
    (("norm", "eps"), None, "eps"),
    (("embedding", "scale"), None, "scale"),
    (("layers", 0, "type"), "state", "mamba2"),
    (("layers", 0, "mixer", "groups"), 3, "groups"),
    (("layers", 0, "mixer", "groups"), None, "groups"),
    (("layers", 0, "mixer", "norm_groups"), 7, "norm_groups"),
    (("layers", 0, "mixer", "state"), None, "state"),
    (("layers", 0, "mixer", "conv"), None, "conv"),
    (("layers", 0, "mlp", "kind"), "dense", "moe"),
    (("layers", 0, "mlp", "expert"), None, "expert"),
    (("layers", 0, "mlp", "router", "top"), 9, "cannot give 9"),
    (("layers", 0, "mlp", "router", "groups", "count"), 2, "groups"),
    (("layers", 0, "mlp", "router", "groups", "keep"), None, "keep"),
    (("layers", 1, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 1, "mixer", "diff"), None, "diff"),
    (("layers", 1, "mixer", "scale"), None, "scale"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "dims"),
    (("layers", 1, "mixer", "rot", "scaling", "original"), None, "original"),
    (("layers", 2, "mixer", "dim"), None, "dim"),
])
def test_config_errors_name_the_key(path, value, message):
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.base import ConfigError
    from mini_llm_runtime_b200.config.registry import config_from_dict
    config = repolix_models.get("small_a")
    at = config
    for key in path[:-1]:
        at = at[key]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError, match=message):
        config_from_dict(config)


def test_plain_router_keeps_the_groups_with_the_largest_choice_and_does_not_renormalize():
    scores = torch.tensor([0.30, 0.05, 0.20, 0.20, 0.15, 0.10], dtype=torch.float64)
    shift = torch.tensor([-1.0, -1.0, -1.0, -1.0, -0.7, -1.0], dtype=torch.float64)
    # groups (0, 1), (2, 3), (4, 5): best choices -0.70, -0.80, -0.55; all are negative, so a dropped group's zero would win
    assert plain.choose(scores, shift, 2, 3, 2) == [4, 0]
    assert plain.choose(scores, shift, 4, 3, 2) == [4, 0, 5, 1]
    assert plain.choose(scores, shift, 3, 1, 1) == [4, 0, 2]
    w = {"m.router": torch.zeros(4, 2, dtype=torch.float64), "m.correction": torch.tensor([0.0, 0.0, 1.0, 2.0], dtype=torch.float64)}
    x = torch.tensor([[1.0, -3.0]], dtype=torch.float64)
    got = plain.routed_experts({"router": {"experts": 2, "identity": 2, "top": 2}, "expert": {"limit": 1.0}}, w, "m.", x)
    assert torch.allclose(got, 0.5 * x)             # two identity experts of a quarter each


def test_plain_window_difference_and_rotation():
    q = k = torch.zeros(4, 1, 2, dtype=torch.float64)
    v = torch.tensor([1.0, 2.0, 4.0, 8.0], dtype=torch.float64).view(4, 1, 1)
    assert plain.windowed_attention(q, k, v, 1.0, 2)[:, 0, 0].tolist() == [1.0, 1.5, 3.0, 6.0]
    o = plain.difference(torch.tensor([[[3.0, 1.0]]]), torch.tensor([[[1.0, 1.0]]]), 1.0, 0.25, 2.0)
    assert torch.allclose(o, torch.tensor([[[2.0, 0.0]]]) / 2.0 * 0.75)
    x = torch.tensor([[[1.0, 5.0, 0.0, 7.0, 9.0]]], dtype=torch.float64)
    y = plain.rotate_halves(x, torch.tensor([1]), [math.pi / 2, math.pi], 2.0)
    assert torch.allclose(y, torch.tensor([[[0.0, -10.0, 2.0, -14.0, 9.0]]], dtype=torch.float64), atol=1e-12)


def test_plain_state_space_reads_its_own_write_and_gates_before_the_norm():
    one = lambda *x: torch.tensor(x, dtype=torch.float64)
    y = plain.state_space_recurrence(one([[2.0]], [[0.0]]), one([[1.0, 0.0]], [[0.0, 0.0]]), one([[3.0, 0.0]], [[1.0, 0.0]]), one([0.9], [0.5]), one([0.5], [1.0]))
    assert y[:, 0, 0].tolist() == [3.0, 0.5]
    m = {"heads": 1, "vdim": 2, "state": 1, "groups": 1, "conv": 1, "norm_groups": 2}
    w = {"in": torch.zeros(7, 1), "conv": torch.ones(4, 1), "conv.b": torch.zeros(4), "dt_bias": torch.zeros(1), "A_log": torch.zeros(1), "D": torch.ones(1),
         "norm": torch.ones(2), "o": torch.eye(2)}
    w = {k: t.double() for k, t in w.items()}
    w["in"][:, 0] = torch.tensor([1.0, -1.0, 5.0, 5.0, 0.0, 0.0, 0.0])          # z of both signs, the same value twice
    out = plain.state_space(m, w, "", torch.ones(1, 1, dtype=torch.float64), 0.0)
    assert torch.allclose(out, one([1.0, -1.0]))     # parts of one value: the norm leaves the gate's sign


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps,rot", [
    (4, 2, 16, 24, 4, (8, 100.0, (8.0, 64, 4.0, 1.0))), (3, 1, 7, 5, 6, (4, 30.0, None)), (2, 2, 32, 64, 3, (32, 5000.0, (4.0, 96, 8.0, 2.0))),
    (2, 1, 8, 16, 1, None), (5, 5, 64, 8, 2, (16, 300.0, (32.0, 16, 1.0, 0.1))), (1, 1, 40, 40, 7, (40, 50.0, None))])
@pytest.mark.parametrize("cuts", [[0, 45], [0, 1, 3, 4, 29, 45]])
def test_convolved_and_rotated_projections(dtype, heads, kv_heads, dim, vdim, taps, rot, cuts):
    """Queries into their buffer, keys (both maps of a head side by side) and values into shuffled pages; the taps reach over portions
    through the state, in the form that moves the state on itself and in the one that leaves it to a second launch."""
    from mini_llm_runtime_b200.ops import native
    from mini_llm_runtime_b200.ops.specs import MaskedAttentionSpec
    dev, T, page = "cuda:0", cuts[-1], 8
    g = torch.Generator().manual_seed(dim + taps)
    key_row, channels = 2 * dim, 2 * (heads + kv_heads) * dim + kv_heads * vdim
    x = torch.randn(2 * T, channels + 8, generator=g).to(dtype).to(dev)[:, :channels]      # two requests, interleaved portions below
    weights = torch.randn(channels, taps, generator=g)
    freqs, mult = plain.yarn(rot[0], rot[1], dict(zip(("factor", "original", "fast", "slow"), rot[2])) if rot[2] else None) if rot else ([], 1.0)
    freq = torch.tensor(freqs or [0.0], dtype=torch.float32, device=dev)
    spec = MaskedAttentionSpec(freq=freq.data_ptr() if rot else None, rot_dims=rot[0] if rot else 0, heads=2 * heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                               maps=2, rot_mult=mult)
    wd = weights.to(dev).contiguous()
    for step in (1, 0):
        page_width = kv_heads * (key_row + vdim)
        cache, n_pages, table = _pages(2 * (T + page), page, page_width, dtype, g, dev)
        per = (T + page - 1) // page
        tables = torch.stack([table[0, :per], table[0, per:2 * per]]).contiguous()
        state = torch.zeros(3, max(1, (taps - 1) * channels), device=dev)
        status = torch.zeros(1, dtype=torch.int32, device=dev)
        got_q = torch.full((2, T, 2 * heads * dim), float("nan"), dtype=dtype, device=dev)
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            n = hi - lo
            rows = torch.cat([x[lo:hi], x[T + lo:T + hi]]).contiguous()
            positions, of_row, info = _meta([(0, n, lo, 2), (n, n, lo, 0)], dev)
            q = torch.full((2 * n, 2 * heads * dim), float("nan"), dtype=dtype, device=dev)
            _call("short_conv", "mlr_conv_rotate_cache", ctypes.addressof(spec), rows.data_ptr(), rows.stride(0), q.data_ptr(), q.stride(0),
                  native.is_bf16(q), taps, wd.data_ptr(), state.data_ptr(), state.stride(0), cache.data_ptr(), n_pages, positions.data_ptr(),
                  info.data_ptr(), of_row.data_ptr(), tables.data_ptr(), tables.stride(0), page, 2, 2 * n, step, status.data_ptr(), native.stream())
            if not step:
                _call("short_conv", "mlr_short_conv_state", rows.data_ptr(), rows.stride(0), native.is_bf16(q), channels, taps, state.data_ptr(),
                      state.stride(0), info.data_ptr(), 2, native.stream())
            got_q[0, lo:hi], got_q[1, lo:hi] = q[:n], q[n:]
        assert int(status.item()) == 0 and not state[1].any()
        tol = 2e-5 if dtype is torch.float32 else 2e-2
        held = cache.double().cpu().view(n_pages, -1)
        for i in range(2):
            y = plain.causal_convolution(x[i * T:(i + 1) * T].double().cpu(), weights.double())
            cq, ck, cv = torch.split(y, [2 * heads * dim, 2 * kv_heads * dim, kv_heads * vdim], dim=1)
            at = torch.arange(T)
            want_q = plain.rotate_halves(cq.reshape(T, 2 * heads, dim), at, freqs, mult).reshape(T, -1)
            want_k = plain.rotate_halves(ck.reshape(T, 2 * kv_heads, dim), at, freqs, mult).reshape(T, kv_heads, key_row)
            assert torch.allclose(got_q[i].double().cpu(), want_q, atol=5 * tol, rtol=tol)
            pages = [held[int(tables[i, t // page])] for t in range(T)]
            got_k = torch.stack([p[:kv_heads * page * key_row].view(kv_heads, page, key_row)[:, t % page] for t, p in enumerate(pages)])
            got_v = torch.stack([p[kv_heads * page * key_row:].view(kv_heads, page, vdim)[:, t % page] for t, p in enumerate(pages)])
            assert torch.allclose(got_k, want_k, atol=5 * tol, rtol=tol)
            assert torch.allclose(got_v, cv.reshape(T, kv_heads, vdim), atol=5 * tol, rtol=tol)


ATTENTIONS = [(2, 1, 16, 16, None), (8, 2, 32, 64, 70), (6, 2, 48, 40, 33), (2, 2, 128, 128, 64), (18, 1, 16, 8, None), (3, 3, 7, 5, 20), (2, 1, 64, 96, 1),
              (1, 1, 24, 160, 50)]
HOWS = ["rows", ("tiles", 77), ("split", 1, 64, 4, 1), ("split", 1, 128, 2, 4)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("how", HOWS)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window", ATTENTIONS)
@pytest.mark.parametrize("loud", [None, 0, 63, 64, "last_in", "last_out"])
def test_difference_of_two_maps(dtype, how, heads, kv_heads, dim, vdim, window, loud):
    """Both maps' softmaxes over shuffled pages and their normed difference, on every kernel; with one key made loud for one of the
    maps: at the first place, on both sides of a tile's border, the last one inside the last row's window and the first one outside."""
    from mini_llm_runtime_b200.ops import native
    from mini_llm_runtime_b200.ops.specs import MaskedAttentionSpec
    dev, T, page, diff, factor, eps, scale = "cuda:0", 200, 8, 0.3, 0.6, 1e-3, 0.8 / math.sqrt(dim)
    tiled = native.module("attention_masked").mlr_attention_masked_tiles_fit(2 * dim, vdim) and dim % 16 == 0
    if how[0] == "tiles" and not (tiled and dtype is torch.bfloat16):
        pytest.skip("these sizes run on the row kernel")
    if window is None and loud in ("last_in", "last_out"):
        pytest.skip("no window")
    g = torch.Generator().manual_seed(dim + vdim)
    q, k, v = torch.randn(T, 2 * heads, dim, generator=g), torch.randn(T, kv_heads, 2, dim, generator=g), torch.randn(T, kv_heads, vdim, generator=g)
    if loud is not None:
        at = {"last_in": T - (window or 0), "last_out": T - 1 - (window or 0)}.get(loud, loud)
        k[at, :, 0] *= 3.0
        own = k[at].repeat_interleave(heads // kv_heads, dim=0)          # the last row's first map asks for that key
        q[T - 1].view(heads, 2, dim)[:, 0] = 2.0 * own[:, 0] / own[:, 0].norm(dim=-1, keepdim=True) * math.sqrt(dim)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    cache, n_pages, table = _pages(T, page, kv_heads * (2 * dim + vdim), dtype, g, dev)
    for t in range(T):
        row = cache[int(table[0, t // page])]
        row[:kv_heads * page * 2 * dim].view(kv_heads, page, 2 * dim)[:, t % page] = k[t].reshape(kv_heads, 2 * dim).to(dev)
        row[kv_heads * page * 2 * dim:].view(kv_heads, page, vdim)[:, t % page] = v[t].to(dev)
    spec = MaskedAttentionSpec(heads=2 * heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window or 0, maps=2, scale=scale, out_scale=1.0 - diff,
                               map_weight=factor, map_eps=eps)
    out = torch.full((T, heads * vdim), float("nan"), dtype=dtype, device=dev)
    qd = q.reshape(T, -1).to(dev)
    _attend(spec, qd, None, out, cache, n_pages, table, page, T, how, kv_heads, vdim)
    wide = [t.double() for t in (q, k, v)]
    vv = wide[2].repeat_interleave(heads // kv_heads, dim=1)
    maps = [plain.windowed_attention(wide[0].view(T, heads, 2, dim)[:, :, i], wide[1][:, :, i].repeat_interleave(heads // kv_heads, dim=1), vv, scale, window)
            for i in range(2)]
    want = plain.difference(maps[0], maps[1], factor, diff, eps).reshape(T, -1)
    rows = _rows_of(how, T)
    tol = 3e-5 if dtype is torch.float32 else 2e-2
    assert torch.allclose(out.double().cpu()[rows], want[rows], atol=2 * tol, rtol=tol), float((out.double().cpu()[rows] - want[rows]).abs().max())
    if loud in (0, 63, 64, "last_in") and (window is None or T - 1 - at < window):
        assert torch.allclose(maps[0][T - 1], vv[at], atol=0.2), "the loud key must carry the row"


def _mixer(kind, mixer, width, eps, dtype, seed):
    """The part of a one-layer configuration, its weights and a runtime."""
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dict, plan_for
    from mini_llm_runtime_b200.csrc import build
    from mini_llm_runtime_b200.engine.runtime import Runtime
    from mini_llm_runtime_b200.engine.structure import build_part
    config = {"architecture": "Repolix", "vocab": 8, "width": width, "norm": {"eps": eps}, "embedding": {"scale": 1.0},
              "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}
    weights = repolix_models.random_weights(config, seed)
    part = build_part("mixer", plan_for(config_from_dict(config)).layers[0].mixer)
    rt = Runtime(dtype)
    build.ensure(part.kernel_modules(dtype))
    return part, weights, rt, config


STATES = [
    ("mamba2", dict(heads=3, groups=1, state=10, vdim=7, conv=5, norm_groups=7)),
    ("mamba2", dict(heads=4, groups=2, state=32, vdim=56, conv=3, norm_groups=1)),
    ("mamba2", dict(heads=6, groups=6, state=64, vdim=20, conv=1, norm_groups=4)),
    ("mamba2", dict(heads=2, groups=1, state=128, vdim=64, conv=4, norm_groups=2)),
    ("mamba2", dict(heads=3, groups=3, state=100, vdim=16, conv=7, norm_groups=3)),
    ("mamba2", dict(heads=2, groups=2, state=256, vdim=32, conv=2, norm_groups=8)),
    ("mamba2", dict(heads=1, groups=1, state=96, vdim=160, conv=4, norm_groups=5)),
    ("mamba2", dict(heads=40, groups=4, state=32, vdim=40, conv=2, norm_groups=10)),       # more blocks than SMs: two state columns a lane
    ("channel_delta", dict(heads=6, kv_heads=2, dim=12, vdim=20, conv=4, decay_rank=7, gate_rank=9)),
    ("channel_delta", dict(heads=2, kv_heads=2, dim=64, vdim=32, conv=3, decay_rank=16, gate_rank=8)),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("kind,mixer", STATES)
def test_recurrences_alone_in_both_forms(dtype, fused, kind, mixer):
    """Three unequal requests in one batch, in portions (down to one token) that carry the state; the form for few rows and the prepared
    walk for many.  An eps of the size of the squares shows whether it stands inside the root."""
    width, eps = 40, 0.05
    part, weights, rt, config = _mixer(kind, mixer, width, eps, dtype, seed=mixer.get("state", 5))
    rt.recurrence_fused_rows = 1 << 30 if fused else 0
    part.bind(weights, rt)
    g = torch.Generator().manual_seed(5)
    lengths = [75, 1, 38]
    x = [torch.randn(n, width, generator=g).to(dtype) for n in lengths]
    wide = {k: v.double() for k, v in weights.items()}
    want = [plain.MIXERS[kind](config["layers"][0]["mixer"], wide, "l0.mix.", r.double(), eps) for r in x]
    tol = 3e-4 if dtype is torch.float32 else 0.1
    for cuts in ([0, 80], [0, 1, 3, 36, 37, 69, 80]):
        got, state = _state_steps(part, rt, x, lengths, cuts)
        assert not state[:2].any()                       # slots of nobody stay as they are
        for a, b in zip(got, want):
            size = float(b.pow(2).mean().sqrt())
            assert torch.allclose(a, b, atol=tol * max(1.0, size), rtol=tol), (cuts, float((a - b).abs().max()), size)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,identity,groups,keep,top", [(6, 3, 3, 2, 3), (5, 0, 1, 1, 2), (10, 6, 4, 3, 5), (1, 7, 2, 1, 3), (64, 16, 8, 3, 8), (3, 2, 5, 2, 2),
                                                              (40, 24, 64, 32, 32), (7, 1, 1, 1, 8)])
@pytest.mark.parametrize("rows,width", [(37, 24), (601, 18)])            # one token a block, and four
def test_router_with_groups_and_identity_experts(dtype, experts, identity, groups, keep, top, rows, width):
    from mini_llm_runtime_b200.ops import native
    dev = "cuda:0"
    everyone = experts + identity
    g = torch.Generator().manual_seed(everyone)
    x = torch.randn(rows, width, generator=g).to(dtype).to(dev)
    router, correction = torch.randn(everyone, width, generator=g).to(dev), (0.3 * torch.randn(everyone, generator=g) - 1.0).to(dev)      # choices below zero
    chosen = torch.empty(rows, top, dtype=torch.int32, device=dev)
    place = torch.empty_like(chosen)
    weights, passed = torch.empty(rows, top, device=dev), torch.full((rows,), float("nan"), device=dev)
    counts = torch.zeros(experts, dtype=torch.int32, device=dev)
    _call("experts", "mlr_experts_route", x.data_ptr(), x.stride(0), native.is_bf16(x), router.data_ptr(), correction.data_ptr(), rows, width,
          everyone, experts, groups, keep, top, 0, chosen.data_ptr(), weights.data_ptr(), place.data_ptr(), counts.data_ptr(), None,
          passed.data_ptr() if identity else None, 2, native.stream())
    scores = torch.softmax(x.double().cpu() @ router.double().cpu().T, dim=-1)
    for t in list(range(37)) + list(range(37, rows, 41)) + [rows - 1]:
        want = plain.choose(scores[t], correction.double().cpu(), top, groups, keep)
        assert chosen[t].tolist() == want
        assert torch.allclose(weights[t].double().cpu(), scores[t, want], atol=1e-6)
        if identity:
            assert float(passed[t]) == pytest.approx(float(sum(scores[t, e] for e in want if e >= experts)), abs=1e-6)
    real = chosen.cpu().flatten()
    assert counts.cpu().tolist() == torch.bincount(real[real < experts].long(), minlength=experts).tolist()
    for e in range(experts):
        mine = place.cpu()[chosen.cpu() == e]
        assert sorted(mine.tolist()) == list(range(len(mine)))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [1, 3, 70, 700])
@pytest.mark.parametrize("shape", [(24, 6, 3, (3, 2), 3, 56), (32, 8, 0, None, 2, None), (10, 2, 6, (2, 1), 2, 12)])
def test_routed_experts_part_against_the_plain_function(dtype, rows, shape):
    """The part by hand, run twice: counters return to zero, tokens whose experts are all identity experts among them."""
    from mini_llm_runtime_b200.csrc import build
    from mini_llm_runtime_b200.engine.runtime import Runtime
    from mini_llm_runtime_b200.engine.structure import build_part
    from mini_llm_runtime_b200.config.registry import config_from_dict, plan_for
    from mini_llm_runtime_b200.parts.base import StepContext
    ff, experts, identity, groups, top, shared = shape
    mlp = repolix_models._moe(ff, 1.2, experts, top, identity, groups, (shared, 0.8) if shared else None)
    config = {"architecture": "Repolix", "vocab": 8, "width": 40, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
              "layers": [{"type": "mamba2", "mixer": dict(heads=1, groups=1, state=4, vdim=4, conv=1, norm_groups=1), "mlp": mlp}]}
    weights = repolix_models.random_weights(config, rows)
    part = build_part("feed_forward", plan_for(config_from_dict(config)).layers[0].feed_forward)
    rt = Runtime(dtype)
    build.ensure(part.kernel_modules(dtype))
    part.bind(weights, rt)
    x = torch.randn(rows, 40, generator=torch.Generator().manual_seed(rows)).to(dtype)
    wide = {k: v.double() for k, v in weights.items()}
    want = plain.routed_experts(mlp, wide, "l0.mlp.", x.double())
    for _ in range(2):
        step = StepContext(rt=rt, num_rows=rows, segments=[], token_ids=None, positions=None, segment_of_row=None, segment_info=None, slots=None, tables={},
                           page_size=16, status=torch.zeros(1, dtype=torch.int32, device=rt.device))
        got = part.forward(x.to(rt.device), step).double().cpu()
        assert not part.counts.any()
        wrong = ((got - want).abs() > (2e-4 if dtype is torch.float32 else 0.06) * (1.0 + want.abs())).any(dim=1)
        assert int(wrong.sum()) <= (0 if dtype is torch.float32 else rows // 100), int(wrong.sum())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,top,streams,shared,identity", [(5, 40, 3, 1, True, True), (3, 37, 1, 1, False, True), (70, 64, 8, 1, True, False),
                                                                    (4, 4096, 4, 1, True, True), (6, 48, 2, 3, False, True)])
def test_pieces_of_routed_experts_joined_by_the_stream_and_by_the_combine_kernel(dtype, rows, width, top, streams, shared, identity):
    """x <- x + scale .* (the pieces added up), with the norm that reads the stream next, in one launch; and the pieces added up alone."""
    from mini_llm_runtime_b200.ops import native
    dev = "cuda:0"
    g = torch.Generator().manual_seed(width)
    h, y = torch.randn(rows, streams * width, generator=g), torch.randn(rows * top, width, generator=g)
    place = torch.randperm(rows * top, generator=g).to(torch.int32).view(rows, top)
    if identity:
        place[0, 0] = place[-1, top - 1] = -1
    weights, passed = torch.rand(rows, top, generator=g), torch.rand(rows, generator=g)
    x, other = torch.randn(rows, width + 4, generator=g).to(dtype), torch.randn(rows, width, generator=g)
    scale, norm_w = torch.randn(width, generator=g), torch.randn(width, generator=g)
    mix = torch.randn(streams, streams, generator=g) if streams > 1 else torch.ones(1, 1)
    w_out, w_in = (torch.randn(streams, generator=g) if streams > 1 else torch.ones(1) for _ in range(2))
    on = [t.to(dev).contiguous() for t in (h, y, place, weights, other, x, passed, scale, mix, w_out, w_in, norm_w)]
    hd, yd, pd, wd, od, xd, sd, cd, md, outd, ind, nd = on
    pieces = (yd.data_ptr(), width, pd.data_ptr(), wd.data_ptr(), top, od.data_ptr() if shared else None, width if shared else 0, None,
              xd.data_ptr() if identity else None, xd.stride(0), native.is_bf16(xd), sd.data_ptr() if identity else None)
    alone = torch.full((rows, width), float("nan"), device=dev)
    _call("experts", "mlr_experts_combine", *pieces, alone.data_ptr(), width, rows, width, native.stream())
    out = torch.full((rows, width), float("nan"), dtype=dtype, device=dev)
    _call("streams", "mlr_streams_step_pieces", hd.data_ptr(), *pieces, cd.data_ptr(), md.data_ptr(), outd.data_ptr(), ind.data_ptr(), nd.data_ptr(), 0.01,
          out.data_ptr(), width, native.is_bf16(out), rows, width, streams, native.stream())
    total = torch.zeros(rows, width, dtype=torch.float64)
    for t in range(rows):
        for j in range(top):
            if place[t, j] >= 0:
                total[t] += float(weights[t, j]) * y[int(place[t, j])].double()
    if identity:
        total += passed.double()[:, None] * x[:, :width].double()
    if shared:
        total += other.double()
    assert torch.allclose(alone.double().cpu(), total, atol=1e-5, rtol=1e-5)
    old = h.double().view(rows, streams, width)
    new = torch.einsum("rsw,st->rtw", old, mix.double()) + w_out.double()[None, :, None] * (scale.double() * total)[:, None, :]
    assert torch.allclose(hd.double().cpu().view(rows, streams, width), new, atol=5e-5, rtol=5e-5)
    read = torch.einsum("rtw,t->rw", new, w_in.double())
    tol = 1e-4 if dtype is torch.float32 else 2e-2
    assert torch.allclose(out.double().cpu(), plain.rms_norm(read, norm_w.double(), 0.01), atol=tol, rtol=tol)


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module", params=sorted(repolix_models.ALL))
def case(request, tmp_path_factory):
    config = repolix_models.get(request.param)
    weights = repolix_models.random_weights(config, seed=14)
    folder = str(tmp_path_factory.mktemp(request.param))
    stored = repolix_models.get(request.param)
    for layer in stored["layers"]:               # the file leaves the ranks to the tensors' shapes
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    write_model_folder(folder, stored, weights)
    return folder, config, weights


@pytest.mark.gpu
def test_every_layer_of_a_short_prompt(case):
    """The stream after every layer, float32, with the steps driven from Python part by part."""
    from mini_llm_runtime_b200.engine.model import StepEntry
    folder, config, weights = case
    model = engine_model(folder, "float32", num_pages=8, page_size=8, max_requests=1)
    model._native = None
    seen = []
    for run in model.runs:
        def wrapped(h, pending, step, ctx, inner=run.block.forward):
            result = inner(h, pending, step, ctx)
            seen.append(h.double().cpu())
            return result
        run.block.forward = wrapped
    tokens = tokens_for(config, 19, 2)
    slot = model.open_request()
    model.step([StepEntry(slot, tokens, [18])])
    want = []
    plain.forward(config, weights, tokens, want)
    assert len(seen) == len(want)
    for i, (a, b) in enumerate(zip(seen, want)):
        assert torch.allclose(a, b, atol=2e-4, rtol=2e-4), (i, float((a - b).abs().max()))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_portions_and_decoding_agree_with_the_plain_implementation(case, dtype):
    folder, config, weights = case
    model = engine_model(folder, dtype, num_pages=24, page_size=8, max_requests=2)
    assert model._native is not None, "the model must run in the native step executor"
    tokens = tokens_for(config, 150, 4)
    want = plain_logits(config, weights, tokens)
    whole = run_whole(model, tokens)
    close(whole, want, dtype, "whole")
    for sizes in ([1], [2], [3, 2, 7], [64, 1], [65, 2, 70], [149, 1], [11, 2, 2, 30, 1, 5]):      # [1]: decoding from the first token on
        got = run_portions(model, tokens, sizes)
        close(got, want, dtype, f"portions {sizes}")
        if dtype == "float32":      # how a prompt is cut changes nothing but the order of a few sums
            assert float((got - whole).abs().max()) <= 2e-4 * max(1.0, float(whole.abs().max())), sizes
    assert model.cache.free_slots() == 2


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_of_unequal_requests_equals_each_alone_and_slots_are_used_again(case, dtype):
    from mini_llm_runtime_b200.engine.model import StepEntry
    folder, config, weights = case
    model = engine_model(folder, dtype, num_pages=40, page_size=8, max_requests=3)
    lengths = [70, 9, 33, 2, 51, 20, 64]
    requests = [tokens_for(config, n, 100 + n) for n in lengths]
    alone = [plain_logits(config, weights, t) for t in requests]
    got = [[] for _ in requests]
    # Three live requests at a time; a finished one gives its slot and its pages to the next.
    waiting, live = list(range(len(requests))), {}
    sizes = [5, 1, 2, 13, 1, 1, 30, 3]
    turn = 0
    while waiting or live:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = [model.open_request(), 0]
        entries, who = [], []
        for i, (slot, at) in live.items():
            if (turn + i) % 4 == 3 and len(live) > 1:
                continue                                  # this request sits the step out
            n = min(sizes[(turn + i) % len(sizes)], len(requests[i]) - at)
            entries.append(StepEntry(slot, requests[i][at:at + n], list(range(n))))
            who.append((i, n))
        if entries:
            logits = model.step(entries).float().cpu()
            row = 0
            for i, n in who:
                got[i].append(logits[row:row + n])
                row += n
                live[i][1] += n
                if live[i][1] == len(requests[i]):
                    model.close_request(live.pop(i)[0])
        turn += 1
    model.check_status()
    for i in range(len(requests)):
        close(torch.cat(got[i]), alone[i], dtype, f"request {i}")
    assert model.cache.free_slots() == 3


@pytest.mark.gpu
def test_long_decoding_through_the_graphs(case):
    """Two requests decoded token by token from their first token on, through several graph buckets of the smallest size."""
    from mini_llm_runtime_b200.engine.model import StepEntry
    folder, config, weights = case
    model = engine_model(folder, "float32", num_pages=64, page_size=8, max_requests=2)
    a, b = tokens_for(config, 260, 1), tokens_for(config, 200, 2)
    sa, sb = model.open_request(), model.open_request()
    got_a, got_b = [], []
    for t in range(len(a)):
        entries = [StepEntry(sa, [a[t]], [0])] + ([StepEntry(sb, [b[t]], [0])] if t < len(b) else [])
        logits = model.step(entries).float().cpu()
        got_a.append(logits[0])
        if t < len(b):
            got_b.append(logits[1])
    model.check_status()
    assert model._graphs, "single-token steps did not reach the CUDA graphs"
    assert_close(torch.stack(got_a), plain_logits(config, weights, a), "float32", "a")
    assert_close(torch.stack(got_b), plain_logits(config, weights, b), "float32", "b")


WINDOW = 37


def _loud_model(kind):
    """One layer in which token 0 asks for token 1: the query of token 0 points at the key of token 1 (in one map of every head),
    decays are nearly none, and the logits of a token 0 behind a token 1 therefore show that token's value."""
    mixers = {"attention": dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, diff=0.4, conv=3, mask={"size": WINDOW},
                                rot={"base": 1000.0, "dims": 4, "scaling": {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0}}),
              "mamba2": dict(heads=4, groups=2, state=48, vdim=24, conv=2, norm_groups=2),
              "channel_delta": dict(heads=4, kv_heads=2, dim=48, vdim=24, conv=2, decay_rank=6, gate_rank=5)}
    config = {"architecture": "Repolix", "vocab": 64, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
              "layers": [{"type": kind, "mixer": mixers[kind], "mlp": None}]}
    w = repolix_models.random_weights(config, 3)
    m, p = config["layers"][0]["mixer"], "l0.mix."
    H = m["heads"]
    x = plain.rms_norm(w["embed"].double(), w["l0.norm1"].double(), 1e-5)
    w["l0.ls1"] = 3.0 * w["l0.ls1"]
    asker = x[0] / (x[0] @ x[0])
    last_tap = lambda n: torch.eye(m["conv"])[-1].repeat(n, 1).bfloat16()
    if kind == "attention":
        G, D = m["kv_heads"], m["dim"]
        for role, n in (("q", 2 * H * D), ("k", 2 * G * D), ("v", G * m["vdim"])):
            w[p + role + ".conv"] = last_tap(n)
        key = (w[p + "k"].double() @ x[1]).view(G, 2, D).repeat_interleave(H // G, dim=0)
        q = w[p + "q"].double().view(H, 2, D, -1)
        q[:, 0] += 3.0 * key[:, 0, :, None] * asker
        q[:, :, :4] = 0.0                             # nothing of the question is rotated
        w[p + "q"] = q.reshape(2 * H * D, -1).bfloat16()
    elif kind == "mamba2":
        inner, N, G = H * m["vdim"], m["state"], m["groups"]
        w[p + "conv"], w[p + "conv.b"] = last_tap(inner + 2 * G * N), torch.zeros(inner + 2 * G * N).bfloat16()
        rows = w[p + "in"].double()
        key = plain.silu(rows[2 * inner:2 * inner + G * N] @ x[1])
        rows[2 * inner + G * N:2 * inner + 2 * G * N] = 8.0 * (key - key.mean())[:, None] * asker
        w[p + "in"] = rows.bfloat16()
        w[p + "A_log"], w[p + "dt_bias"], w[p + "D"] = torch.full((H,), -9.0).bfloat16(), torch.zeros(H).bfloat16(), torch.zeros(H).bfloat16()
    else:
        G, D = m["kv_heads"], m["dim"]
        w[p + "q.conv"], w[p + "k.conv"] = last_tap(G * D), last_tap(G * D)
        w[p + "q"] = (w[p + "q"].double() + 4.0 * (w[p + "k"].double() @ x[1]).reshape(-1, 1) * asker).bfloat16()
        w[p + "dt_bias"] = torch.full((H * D,), -9.0).bfloat16()
        w[p + "b"] *= 0.0
    return config, w


LOUD_LENGTH = {"attention": 210, "mamba2": 40, "channel_delta": 60}       # a state of 48 x 24 holds so many other writes before they drown one key


def _loud_places(kind):
    n = LOUD_LENGTH[kind]
    if kind == "attention":           # by the distance to the asking token: just inside, on and just outside the window; the pages of 8 around
        return [n - 1 - d for d in (1, 2, 8, 9, 17, WINDOW - 2, WINDOW - 1, WINDOW, WINDOW + 1)]
    return [p for p in (0, 1, 7, 8, 15, 16, 31, 32, n - 2) if p < n - 1]


def _loud_shift(kind, config, weights, at):
    g = torch.Generator().manual_seed(8)
    rest = torch.randint(2, config["vocab"], (LOUD_LENGTH[kind],), generator=g).tolist()
    tokens = list(rest)
    tokens[at], tokens[-1] = 1, 0
    want = plain_logits(config, weights, tokens)[-1:]
    without = plain_logits(config, weights, rest[:-1] + [0])[-1:]
    return tokens, want, float((want - without).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


@pytest.mark.parametrize("kind", sorted(LOUD_LENGTH))
def test_the_loud_token_shows_in_the_plain_logits_exactly_where_it_is_seen(kind):
    config, weights = _loud_model(kind)
    for at in _loud_places(kind):
        shift = _loud_shift(kind, config, weights, at)[2]
        outside = kind == "attention" and LOUD_LENGTH[kind] - 1 - at >= WINDOW
        assert shift == 0.0 if outside else shift > 0.1, (at, shift)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", sorted(LOUD_LENGTH))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_loud_token_shows_wherever_it_stands(kind, dtype, tmp_path):
    """A token asked for at the end of the prompt, or by a decoded token, from places around page, tile and window borders."""
    from mini_llm_runtime_b200.engine.model import StepEntry
    config, weights = _loud_model(kind)
    write_model_folder(str(tmp_path), config, weights)
    model = engine_model(str(tmp_path), dtype, num_pages=64, page_size=8, max_requests=2)
    n = LOUD_LENGTH[kind]
    for at in _loud_places(kind):
        tokens, want, _ = _loud_shift(kind, config, weights, at)
        for cuts in ([n], [n - 1, 1], [20, n - 21, 1], [n - 2, 2]):
            slot, pos = model.open_request(), 0
            for c in cuts:
                got = model.step([StepEntry(slot, tokens[pos:pos + c], [c - 1])]).float().cpu()
                pos += c
            model.check_status()
            model.close_request(slot)
            from helpers import row_metrics
            if dtype == "float32":
                assert_close(got, want, dtype, f"{kind} at {at}, portions {cuts}")
            else:
                found = row_metrics(got, want)
                assert float(found["rmse"]) <= BF16["rmse"] and float(found["cosine"]) >= BF16["cosine"], (kind, at, cuts, found)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(case, dtype):
    from mini_llm_runtime_b200 import LLM
    folder, config, weights = case
    prompts = [tokens_for(config, n, 50 + n) for n in (3, 41, 18, 77, 1)]
    llm = LLM(folder, dtype=dtype, max_model_len=128, max_requests=3, num_pages=48, page_size=8, max_batch_tokens=24, prefill_chunk=16)
    results = llm.generate(prompts, max_tokens=12, ignore_eos=True)
    off = 0
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 12
        tokens = list(prompt)
        for step, token in enumerate(result.token_ids):
            row = plain_logits(config, weights, tokens)[-1]
            best = int(torch.argmax(row))
            if token != best:       # two logits closer than the precision's rounding may change places
                margin = 1e-3 if dtype == "float32" else 2 * BF16["max"] * float(row.double().pow(2).mean().sqrt())
                if float(row[best] - row[token]) > margin:
                    off += 1
                    assert dtype == "bfloat16" and off <= 2, (len(prompt), step, token, best)     # a router's close call
            tokens.append(token)
    assert llm.model.cache.free_slots() == 3


@pytest.mark.gpu
def test_trace_replay_with_a_pool_that_is_used_again(case, tmp_path):
    """Through `bin/trace_run` as a user runs it: up to four live requests in a pool sized for them, not for all."""
    import trace_tools
    folder, config, weights = case
    requests = {f"r{i}": tokens_for(config, n, 300 + i) for i, n in enumerate((90, 5, 130, 64, 31, 17, 100))}
    trace = trace_tools.mixed(requests, seed=9)
    logits = trace_tools.run_trace(folder, "float32", trace, str(tmp_path), config["vocab"])
    for name, tokens in requests.items():
        assert_close(trace_tools.stack(logits, name, len(tokens)), plain_logits(config, weights, tokens), "float32", name)
