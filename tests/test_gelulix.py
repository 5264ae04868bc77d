"""The Gelulix decoder: its mechanisms one by one against `plain_gelulix`, then whole models through the engine's step function,
scheduler and entry points.  The plain implementation shares nothing with the package; it runs in float64 on bfloat16-rounded
random weights."""
import math

import pytest
import torch

import gelulix_models
import plain_gelulix as plain
from helpers import assert_close, assert_rows_close, engine_model, run_portions, run_whole, write_model_folder
from test_sopetar import _call, _meta, _pages     # launch helpers only (no test is imported)

BF16 = dict(rmse=0.06, max=0.25, cosine=0.998)


def tokens_for(config, count, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, config["vocab"], (count,), generator=g).tolist()


def plain_logits(config, weights, tokens):
    return plain.forward(config, weights, tokens).float()


def close(got, want, dtype, what):
    if dtype == "bfloat16":
        return assert_rows_close(got, want, what, BF16)
    return assert_close(got, want, dtype, what)


# ----------------------------------------------------------------------------- without a GPU
def test_config_and_plan_name_every_tensor():
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dict, plan_for
    from mini_llm_runtime_b200.engine.structure import expected_weights
    for name in gelulix_models.ALL:
        config = gelulix_models.get(name)
        weights = gelulix_models.random_weights(config, 1)
        expected = expected_weights(plan_for(config_from_dict(config)))
        assert set(expected) == set(weights), name
        for key, spec in expected.items():
            assert tuple(spec.shape) == tuple(weights[key].shape), key


def test_ranks_come_from_the_stored_tensors(tmp_path):
    """A configuration that does not name the ranks of the low-rank products takes them from the weights' shapes."""
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dir, plan_for
    from mini_llm_runtime_b200.engine.structure import expected_weights
    config = gelulix_models.get("small_a")
    weights = gelulix_models.random_weights(config, 1)
    for layer in config["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    write_model_folder(str(tmp_path), config, weights)
    expected = expected_weights(plan_for(config_from_dir(str(tmp_path))))
    assert {k: tuple(s.shape) for k, s in expected.items()} == {k: tuple(t.shape) for k, t in weights.items()}


@pytest.mark.parametrize("path,value,message", [
    (("width",), None, "width"),
    (("norm", "eps"), None, "eps"),
    (("postln_alpha",), None, "postln_alpha"),
    (("layers", 0, "type"), "delta", "channel_delta"),
    (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "conv"), None, "conv"),
    (("layers", 0, "mlp", "kind"), "moe", "dense"),
    (("layers", 0, "mlp", "ff"), None, "ff"),
    (("layers", 1, "mixer", "rot"), None, "rot"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "dims"),
    (("layers", 1, "mixer", "rot", "scaling", "slow"), None, "slow"),
    (("layers", 1, "mixer", "kv_rank"), None, "kv_rank"),
    (("layers", 2, "mixer", "tau"), 0, "tau"),
    (("layers", 3, "mixer", "vdim"), None, "vdim"),
])
def test_config_errors_name_the_key(path, value, message):
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.base import ConfigError
    from mini_llm_runtime_b200.config.registry import config_from_dict
    config = gelulix_models.get("small_a")
    at = config
    for key in path[:-1]:
        at = at[key]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError, match=message):
        config_from_dict(config)


YARNS = [(8, 100.0, (8.0, 64, 4.0, 1.0)), (32, 5000.0, (4.0, 96, 8.0, 2.0)), (64, 300.0, (32.0, 16, 1.0, 0.1)), (64, 1e4, (40.0, 4096, 32.0, 1.0)),
         (2, 10.0, (2.0, 64, 2.0, 1.0)), (6, 50.0, (1.0, 10, 3.0, 1.0)), (16, 20.0, (0.5, 1000000, 1.0, 1.0))]


@pytest.mark.parametrize("dims,base,scaling", YARNS)
def test_yarn_frequencies(dims, base, scaling):
    from mini_llm_runtime_b200.parts.rotary import yarn_frequencies
    s = dict(zip(("factor", "original", "fast", "slow"), scaling))
    want, mult = plain.yarn(dims, base, s)
    got, magnitude = yarn_frequencies(base, dims, **s)
    assert magnitude == pytest.approx(mult, rel=1e-12) and got.tolist() == pytest.approx(want, rel=1e-12)


def test_plain_yarn_keeps_quick_pairs_and_slows_the_slow_ones():
    s = {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    bare, one = plain.yarn(64, 1e4, None)
    f, mult = plain.yarn(64, 1e4, s)
    turns = [4096 * x / (2 * math.pi) for x in bare]
    assert one == 1.0 and math.isclose(mult, 1.0 + 0.1 * math.log(40.0))
    assert all(math.isclose(a, b) for a, b, t in zip(f, bare, turns) if t > 40) and any(t > 40 for t in turns)
    assert all(math.isclose(a, b / 40.0) for a, b, t in zip(f, bare, turns) if t < 0.7) and any(t < 0.7 for t in turns)
    middle = [(a, b) for a, b, t in zip(f, bare, turns) if 2 < t < 20]
    assert middle and all(b / 40.0 < a < b for a, b in middle)


def test_plain_sink_counts_once_is_not_scaled_and_has_no_value():
    q = k = torch.zeros(3, 1, 2, dtype=torch.float64)
    v = torch.ones(3, 1, 1, dtype=torch.float64)
    out = plain.causal_attention(q, k, v, 77.0, torch.tensor([math.log(3.0)], dtype=torch.float64))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 4, 2 / 5, 3 / 6], dtype=torch.float64))


def test_plain_decays_act_on_key_channels_and_the_read_sees_the_write():
    one = lambda *x: torch.tensor(x, dtype=torch.float64)
    q, k = one([[1.0, 1.0]], [[1.0, 0.0]]), one([[1.0, 2.0]], [[0.0, 0.0]])
    v, decay = one([[3.0]], [[0.0]]), one([[0.9, 0.9]], [[0.5, 0.25]])
    assert plain.channel_decay_recurrence(q, k, v, decay)[:, 0, 0].tolist() == [9.0, 1.5]
    out = plain.delta_recurrence(q, k, v, decay, one([1.0], [1.0]))
    assert out[:, 0, 0].tolist() == [9.0, 1.5]
    k2, v2 = one([[1.0, 0.0]], [[1.0, 0.0]]), one([[4.0]], [[6.0]])
    out = plain.delta_recurrence(one([[1.0, 0.0]], [[1.0, 0.0]]), k2, v2, one([[1.0, 1.0]], [[0.5, 1.0]]), one([1.0], [0.5]))
    assert out[:, 0, 0].tolist() == [4.0, 2.0 + 0.5 * (6.0 - 2.0)]          # the state decays before the value it holds is taken off


def test_plain_convolution_and_norm_of_the_sum():
    x = torch.tensor([[1.0], [2.0], [5.0]], dtype=torch.float64)
    y = plain.causal_convolution(x, torch.tensor([[10.0, 1.0]], dtype=torch.float64))
    assert torch.allclose(y, plain.silu(torch.tensor([[1.0], [12.0], [25.0]], dtype=torch.float64)))
    z = plain.residual_norm(torch.tensor([1.0, 2.0], dtype=torch.float64), torch.tensor([1.0, -2.0], dtype=torch.float64), 3.0, torch.ones(2, dtype=torch.float64), 2.0)
    assert torch.allclose(z, torch.tensor([4.0, 4.0], dtype=torch.float64) / math.sqrt(18.0))


def test_a_rotation_with_a_factor_is_refused_where_the_kernels_have_none():
    from mini_llm_runtime_b200.config.base import ConfigError, PartSpec
    from mini_llm_runtime_b200.engine.structure import build_part
    position = build_part("position", PartSpec("rotary_frequencies", {"base": 100.0, "dims": 8, "yarn": {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0}}))
    retention = build_part("mixer", PartSpec("retention", {"hidden_size": 16, "num_heads": 1, "head_dim": 8, "value_dim": 8, "decay": [0.9], "eps": 1e-5,
                                                           "position": "p"}, {}))
    with pytest.raises(ConfigError, match="factor"):
        retention.attach_positions({"p": position})


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,rows,a,bias,then", [(48, 5, 3.0, True, "plain"), (37, 3, 0.5, False, "plain"), (64, 70, 1.0, False, "norm"),
                                                    (6000, 3, -1.5, True, "norm"), (256, 9, 2.5, True, None)])
def test_the_norm_behind_the_sum(dtype, width, rows, a, bias, then):
    """h = norm(a h + delta + bias) * w in one launch, with what the next reader takes of it: the stream, a norm of it, nothing."""
    from mini_llm_runtime_b200.ops import native
    dev, eps = "cuda:0", 0.3                     # an eps of the size of the squares shows whether it stands inside the root
    g = torch.Generator().manual_seed(width)
    h, delta = torch.randn(rows, width, generator=g), 2.0 * torch.randn(rows, width + 8, generator=g)
    b, w, w_next = (torch.randn(width, generator=g) for _ in range(3))
    hd, dd, bd, wd, nd = (t.to(dev) for t in (h, delta, b, w, w_next))
    out = torch.full((rows, width), float("nan"), dtype=dtype, device=dev)
    _call("norm_grouped", "mlr_group_rmsnorm_sum", hd.data_ptr(), a, dd.data_ptr(), dd.stride(0), bd.data_ptr() if bias else None, wd.data_ptr(),
          nd.data_ptr() if then == "norm" else None, out.data_ptr() if then else None, out.stride(0), native.is_bf16(out), rows, width, 1, eps,
          int(then == "plain"), native.stream())
    want = plain.residual_norm(h.double(), delta[:, :width].double() + (b.double() if bias else 0.0), a, w.double(), eps)
    assert torch.allclose(hd.double().cpu(), want, atol=1e-5, rtol=1e-5)
    if then:
        shown = plain.rms_norm(want, w_next.double(), eps) if then == "norm" else want
        tol = 1e-5 if dtype is torch.float32 else 1e-2
        assert torch.allclose(out.double().cpu(), shown, atol=tol, rtol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dims,base,scaling", [y for y in YARNS if y[0] >= 6] + [(10, 30.0, None)])
def test_rotated_parts_carry_the_factor_of_the_scaling(dtype, dims, base, scaling):
    """Queries and the shared key part are turned pair by pair with scaled frequencies, cosine and sine times the scaling's factor; the
    latent beside the key part and the values past the rotated ones are not."""
    from mini_llm_runtime_b200.ops import native
    dev, T, page, rank, heads, dim = "cuda:0", 45, 8, 12, 3, 5
    rot = dims + 2                                 # two values more than are rotated
    g = torch.Generator().manual_seed(dims)
    down, q = torch.randn(T, rank + rot, generator=g).to(dtype).to(dev), torch.randn(T, heads * (dim + rot), generator=g).to(dtype).to(dev)
    weight = torch.ones(rank, device=dev)
    freqs, mult = plain.yarn(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None)
    freq = torch.tensor(freqs + [mult], dtype=torch.float32, device=dev)
    cache, n_pages, table = _pages(T, page, rank + rot, dtype, g, dev)
    positions, of_row, _ = _meta([(0, T, 0, 0)], dev)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    key = rank + rot
    out = torch.zeros(T, heads * key, dtype=dtype, device=dev)
    _call("latent", "mlr_latent_rot_cache", down.data_ptr(), down.stride(0), native.is_bf16(down), weight.data_ptr(), 1e-5, rank, rot, dims, 3,
          freq.data_ptr(), q.data_ptr(), q.stride(0), dim, dim + rot, heads, out.data_ptr(), out.stride(0), rank, key, cache.data_ptr(), n_pages,
          positions.data_ptr(), of_row.data_ptr(), table.data_ptr(), table.stride(0), page, 1, T, status.data_ptr(), native.stream())
    assert int(status.item()) == 0
    at = torch.arange(T)
    want_q = plain.rotate_pairs(q.double().cpu().view(T, heads, dim + rot)[..., dim:], at, freqs, mult)
    want_k = plain.rotate_pairs(down.double().cpu()[:, rank:].view(T, 1, rot), at, freqs, mult)[:, 0]
    tol = 2e-5 if dtype is torch.float32 else 2e-2
    assert torch.allclose(out.double().cpu().view(T, heads, key)[..., rank:], want_q, atol=tol, rtol=tol)
    held = cache.double().cpu().view(n_pages, page, key)
    got = torch.stack([held[int(table[0, t // page]), t % page] for t in range(T)])
    assert torch.allclose(got[:, rank:], want_k, atol=tol, rtol=tol)
    assert torch.allclose(got[:, :rank], plain.rms_norm(down.double().cpu()[:, :rank], None, 1e-5), atol=tol, rtol=tol)


def _mixer(kind, mixer, width, eps, dtype, seed):
    """The part of a one-layer configuration, its weights (by the mixer's own names, float64) and a runtime."""
    from mini_llm_runtime_b200 import models  # noqa: F401
    from mini_llm_runtime_b200.config.registry import config_from_dict, plan_for
    from mini_llm_runtime_b200.csrc import build
    from mini_llm_runtime_b200.engine.runtime import Runtime
    from mini_llm_runtime_b200.engine.structure import build_part
    config = {"architecture": "Gelulix", "vocab": 8, "width": width, "norm": {"eps": eps}, "postln_alpha": 1.0,
              "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}
    weights = gelulix_models.random_weights(config, seed)
    part = build_part("mixer", plan_for(config_from_dict(config)).layers[0].mixer)
    rt = Runtime(dtype)
    build.ensure(part.kernel_modules(dtype))
    return part, weights, rt, config


STATES = [
    ("gla", dict(heads=3, dim=10, vdim=6, tau=16.0, decay_rank=3)),
    ("gla", dict(heads=2, dim=32, vdim=48, tau=1.0, decay_rank=16)),
    ("gla", dict(heads=1, dim=128, vdim=256, tau=5.0, decay_rank=33)),
    ("gla", dict(heads=4, dim=200, vdim=20, tau=8.0, decay_rank=8)),
    ("gla", dict(heads=2, dim=256, vdim=128, tau=16.0, decay_rank=64)),
    ("channel_delta", dict(heads=6, kv_heads=2, dim=12, vdim=20, conv=4, decay_rank=7, gate_rank=9)),
    ("channel_delta", dict(heads=5, kv_heads=5, dim=64, vdim=6, conv=1, decay_rank=1, gate_rank=24)),
    ("channel_delta", dict(heads=2, kv_heads=1, dim=96, vdim=64, conv=7, decay_rank=24, gate_rank=1)),
    ("channel_delta", dict(heads=2, kv_heads=2, dim=128, vdim=128, conv=2, decay_rank=32, gate_rank=16)),
    ("channel_delta", dict(heads=3, kv_heads=1, dim=32, vdim=40, conv=3, decay_rank=12, gate_rank=8)),
]


def _state_steps(part, rt, x, requests, cuts):
    """Runs each request's rows of x [T, W] in steps at `cuts` with their states in slots; returns the rows' results."""
    from mini_llm_runtime_b200.parts.base import RunContext, Segment, StepContext
    state = torch.zeros(len(requests) + 2, *part.state_need().shape, device=rt.device)
    slots = [len(requests) + 1 - i for i in range(len(requests))]
    got = [[] for _ in requests]
    for lo, hi in zip(cuts[:-1], cuts[1:]):
        rows, segments, who = [], [], []
        for i, r in enumerate(requests):
            piece = x[i][min(lo, r):min(hi, r)]
            if len(piece):
                segments.append(Segment(slots[i], min(lo, r), len(piece), sum(len(p) for p in rows)))
                rows.append(piece)
                who.append(i)
        if not rows:
            continue
        h = torch.cat(rows).to(rt.dtype).to(rt.device)
        positions, of_row, info = _meta([(s.row, s.count, s.start, s.slot) for s in segments], rt.device)
        step = StepContext(rt=rt, num_rows=h.shape[0], segments=segments, token_ids=None, positions=positions, segment_of_row=of_row, segment_info=info,
                           slots=None, tables={}, page_size=16, status=torch.zeros(1, dtype=torch.int32, device=rt.device))
        y = part.forward(h, step, RunContext(state=state)).double().cpu()
        for i, s in zip(who, segments):
            got[i].append(y[s.row:s.row + s.count])
    return [torch.cat(p) for p in got], state


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("kind,mixer", STATES)
def test_recurrences_alone_in_both_forms(dtype, fused, kind, mixer):
    """Three unequal requests in one batch, in portions (down to one token) that carry the state; one kernel for few rows, the prepared
    walk for many."""
    width, eps = 40, 1e-3
    part, weights, rt, config = _mixer(kind, mixer, width, eps, dtype, seed=mixer["dim"])
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


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module", params=sorted(gelulix_models.ALL))
def case(request, tmp_path_factory):
    config = gelulix_models.get(request.param)
    weights = gelulix_models.random_weights(config, seed=14)
    folder = str(tmp_path_factory.mktemp(request.param))
    stored = gelulix_models.get(request.param)
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
            assert float((got - whole).abs().max()) <= 1e-4 * max(1.0, float(whole.abs().max())), sizes
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


def _loud_model(kind):
    """One layer in which token 0 asks for token 1: the query of token 0 points at the key of token 1, decays are nearly none, and the
    logits of a token 0 far behind a token 1 therefore show that token's value."""
    mixers = {"gla": dict(heads=2, dim=48, vdim=24, tau=16.0, decay_rank=6),
              "channel_delta": dict(heads=4, kv_heads=2, dim=48, vdim=24, conv=2, decay_rank=6, gate_rank=5),
              "latent_attention": dict(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=32, scale=0.3, rot={"base": 1000.0, "dims": 8, "scaling": {
                  "factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0}})}
    config = {"architecture": "Gelulix", "vocab": 64, "width": 64, "norm": {"eps": 1e-5}, "postln_alpha": 1.0,
              "layers": [{"type": kind, "mixer": mixers[kind], "mlp": None}]}
    w = gelulix_models.random_weights(config, 3)
    m, p = config["layers"][0]["mixer"], "l0.mix."
    H, D = m["heads"], m["dim"]
    x = w["embed"].double()
    w[p + "o"] = 3.0 * w[p + "o"]
    asker = x[0] / (x[0] @ x[0])
    if kind == "latent_attention":
        latent = plain.rms_norm(x[1] @ w[p + "dkv"].double()[:m["kv_rank"]].T, w[p + "dkv.norm"].double(), 1e-5)
        key = (w[p + "uk"].double() @ latent).view(H, D)
        q = w[p + "q"].double().view(H, D + m["rot_dim"], -1).clone()
        q[:, :D] += 3.0 * key[:, :, None] * asker
        w[p + "q"] = q.reshape(-1, q.shape[-1]).bfloat16()
    elif kind == "gla":
        key = (w[p + "k"].double() @ x[1]).view(H, D)
        w[p + "q"] = (w[p + "q"].double() + 8.0 * key.reshape(-1, 1) * asker).bfloat16()
        w[p + "a2.b"] = torch.full((H * D,), 9.0).bfloat16()
    else:
        G = m["kv_heads"]
        w[p + "q.conv"] = torch.tensor([[0.0, 1.0]]).repeat(G * D, 1).bfloat16()
        w[p + "k.conv"] = w[p + "q.conv"].clone()
        w[p + "q"] = (w[p + "q"].double() + 4.0 * (w[p + "k"].double() @ x[1]).reshape(-1, 1) * asker).bfloat16()
        w[p + "dt_bias"] = torch.full((H * D,), -9.0).bfloat16()
        w[p + "b"] *= 0.0
    return config, w


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["gla", "channel_delta", "latent_attention"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_loud_token_far_back_shows_wherever_it_stands(kind, dtype, tmp_path):
    """A token asked for at the end of the prompt, or by a decoded token, from the first place, both sides of page borders and of the
    walk's and the tiles' borders, and just before the end; its logits are the plain implementation's and differ from those of
    a prompt without it."""
    from mini_llm_runtime_b200.engine.model import StepEntry
    config, weights = _loud_model(kind)
    write_model_folder(str(tmp_path), config, weights)
    model = engine_model(str(tmp_path), dtype, num_pages=64, page_size=8, max_requests=2)
    g = torch.Generator().manual_seed(8)
    n = 210 if kind == "latent_attention" else 60       # a state of 48 x 24 holds so many other writes before they drown one key
    rest = torch.randint(2, config["vocab"], (n,), generator=g).tolist()
    for at in [p for p in (0, 1, 7, 8, 15, 16, 31, 32, 63, 64, 127, 128, n - 2) if p < n - 1]:
        tokens = list(rest)
        tokens[at], tokens[-1] = 1, 0
        want = plain_logits(config, weights, tokens)[-1:]
        without = plain_logits(config, weights, rest[:-1] + [0])[-1:]
        shift = float((want - without).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
        assert shift > 0.1, (at, shift)
        for cuts in ([n], [n - 1, 1], [40, n - 41, 1]):
            slot, pos = model.open_request(), 0
            for c in cuts:
                got = model.step([StepEntry(slot, tokens[pos:pos + c], [c - 1])]).float().cpu()
                pos += c
            model.check_status()
            model.close_request(slot)
            close(got, want, dtype, f"{kind} at {at}, portions {cuts}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(case, dtype):
    from mini_llm_runtime_b200 import LLM
    folder, config, weights = case
    prompts = [tokens_for(config, n, 50 + n) for n in (3, 41, 18, 77, 1)]
    llm = LLM(folder, dtype=dtype, max_model_len=128, max_requests=3, num_pages=48, page_size=8, max_batch_tokens=24, prefill_chunk=16)
    results = llm.generate(prompts, max_tokens=12, ignore_eos=True)
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 12
        tokens = list(prompt)
        for step, token in enumerate(result.token_ids):
            row = plain_logits(config, weights, tokens)[-1]
            best = int(torch.argmax(row))
            if token != best:       # two logits closer than the precision's rounding may change places; nothing else may
                margin = 1e-3 if dtype == "float32" else 2 * BF16["max"] * float(row.double().pow(2).mean().sqrt())
                assert float(row[best] - row[token]) <= margin, (len(prompt), step, token, best)
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
