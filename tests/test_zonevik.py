"""The Zonevik decoder in the engine against the plain implementation of ``plain_zonevik.py``: each mechanism's kernel alone,
then whole models of several small configurations through the step function (whole prompts, token by token, portions down
to two tokens, unequal batches, pages and slots used again, long decoding), the replay program, and greedy generation through
``LLMEngine`` and its scheduler.  Where random weights would hide a fault (one key among hundreds, a window's edge, the kept first
tokens, a page border) the weights are made so that one score stands out."""
import json
import math
import random

import numpy as np
import pytest
import torch

import plain_zonevik as P
from trace_tools import TraceBuilder, mixed_trace, peak_tokens, run_trace

gpu = pytest.mark.gpu


def _attn(heads, kv_heads, dim, vdim, scale, rot=None, yarn=None, mask=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if yarn is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return m


def _ssd(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def _moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# Six configurations that differ in every size and option.  a: every kind of layer, the middle ones run three times, values wider
# than keys, YaRN over part of a head with all three bands, a window that is no multiple of a page, three taps.  b: no loop, no
# rotation, no mask, one tap (no convolution state), groups of one expert, one expert a token, one norm part.  c: sizes that the
# tensor-core products and attention take, sixteen query heads a key/value head, kept tokens that fill a page, a loop of one pass
# over the whole model.  d: more than sixteen query heads a key/value head and odd sizes (the plain attention kernel on both
# paths), more kept tokens than the window is wide, five taps, every expert chosen.  e: a window of one token, keys and values as
# many as heads, equal key and value sizes, a loop that opens with the first layer, a stretched rotation whose ramp has no width.
# f: a width that is no multiple of 8 (the CUDA-core products on both paths), sixteen taps, heads wider than the tensor-core
# attention takes, one group kept, plain rotation over an odd number of pairs.
ZN = {
    "a": dict(seed=41, config={
        "architecture": "Zonevik", "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.5},
        "layers": [
            _layer("attention", _attn(4, 2, 16, 24, 0.3, rot=(500.0, 12), yarn=(3.0, 64, 8.0, 0.5)), _moe(6, 2, 24, groups=(3, 2))),
            _layer("parallel", {"left": _attn(4, 2, 12, 20, 0.25, mask=(20, 3)), "right": _ssd(6, 10, 12, 3, 3, 2)}, _moe(8, 3, 16, groups=(2, 1))),
            _layer("delta", _delta(4, 2, 12, 20, 3), _moe(6, 2, 24, groups=(3, 2))),
            _layer("attention", _attn(2, 1, 24, 8, 0.35, rot=(500.0, 24), yarn=(2.0, 40, 16.0, 1.0)), None),
        ], "loop": {"start": 1, "stop": 3, "times": 3}}),
    "b": dict(seed=42, config={
        "architecture": "Zonevik", "vocab": 157, "width": 40, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "loop": None,
        "layers": [
            _layer("delta", _delta(3, 1, 20, 9, 1), _moe(5, 1, 16, groups=(5, 3))),
            _layer("attention", _attn(3, 3, 12, 20, 0.35), _moe(4, 4, 12)),
            _layer("parallel", {"left": _attn(3, 1, 12, 12, 0.3), "right": _ssd(4, 6, 40, 1, 1, 1)}, None),
        ]}),
    "c": dict(seed=43, config={
        "architecture": "Zonevik", "vocab": 509, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 4.0},
        "layers": [
            _layer("delta", _delta(4, 2, 64, 32, 4), _moe(16, 4, 32, groups=(4, 2))),
            _layer("parallel", {"left": _attn(8, 4, 32, 64, 0.18, mask=(64, 16)), "right": _ssd(4, 64, 48, 2, 4, 4)}, _moe(12, 2, 40, groups=(3, 3))),
            _layer("attention", _attn(16, 1, 128, 128, 0.09, rot=(10000.0, 64), yarn=(4.0, 128, 32.0, 1.0)), _moe(16, 4, 32, groups=(4, 2))),
            _layer("parallel", {"left": _attn(4, 4, 64, 64, 0.125, mask=(40, 2)), "right": _ssd(8, 32, 128, 8, 4, 1)}, None),
        ], "loop": {"start": 0, "stop": 4, "times": 1}}),
    "d": dict(seed=44, config={
        "architecture": "Zonevik", "vocab": 97, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.5},
        "layers": [
            _layer("parallel", {"left": _attn(20, 1, 7, 5, 0.4, mask=(25, 30)), "right": _ssd(3, 7, 5, 1, 5, 3)}, _moe(4, 4, 12, groups=(2, 2))),
            _layer("delta", _delta(5, 5, 7, 11, 5), _moe(4, 1, 12, groups=(2, 1))),
        ], "loop": {"start": 0, "stop": 2, "times": 2}}),
    "e": dict(seed=45, config={
        "architecture": "Zonevik", "vocab": 131, "width": 80, "norm": {"eps": 1e-6}, "embedding": {"scale": 3.0},
        "layers": [
            _layer("parallel", {"left": _attn(4, 4, 24, 24, 0.2, mask=(1, 0)), "right": _ssd(4, 16, 16, 4, 2, 4)}, _moe(2, 2, 16, groups=(1, 1))),
            _layer("delta", _delta(2, 2, 16, 16, 2), _moe(2, 1, 16, groups=(2, 1))),
            _layer("attention", _attn(2, 2, 16, 16, 0.25, rot=(100.0, 16), yarn=(8.0, 2000, 1.0, 1.0)), _moe(3, 2, 24, groups=(1, 1))),
        ], "loop": {"start": 0, "stop": 1, "times": 2}}),
    "f": dict(seed=46, config={
        "architecture": "Zonevik", "vocab": 83, "width": 100, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5},
        "layers": [
            _layer("attention", _attn(2, 1, 160, 192, 0.08, rot=(2000.0, 10)), _moe(8, 2, 20, groups=(4, 1))),
            _layer("parallel", {"left": _attn(6, 3, 40, 36, 0.16, mask=(50, 12)), "right": _ssd(2, 50, 33, 2, 16, 2)}, _moe(8, 2, 20, groups=(2, 1))),
            _layer("delta", _delta(6, 3, 36, 18, 16), None),
        ], "loop": {"start": 1, "stop": 3, "times": 2}}),
}
TOL = {"float32": 2e-4, "bfloat16": 6e-2}      # largest difference over the largest logit
CUTS = 8e-6                                     # between two cuts of one prompt in float32


def agrees(got, want, dtype, what=""):
    """32-bit: every position within the tolerance.  bfloat16: a router's close call may fall the other way for a token, which
    swaps a whole expert there (and colours what a later token reads of it), so the criterion is one of counts: nine
    positions in ten are within the tolerance and the median within half of it."""
    err = np.abs(got - want).max(axis=-1) / np.abs(want).max()
    if dtype == "float32":
        assert err.max() < TOL[dtype], f"{what}: position {int(err.argmax())} differs by {float(err.max()):.2e}"
    elif len(err) < 20:
        assert (err < TOL[dtype]).mean() >= 0.5, f"{what}: {err}"
    else:
        assert np.median(err) < TOL[dtype] / 2 and (err > TOL[dtype]).mean() <= 0.1, \
            f"{what}: median {float(np.median(err)):.2e}, {float((err > TOL[dtype]).mean()):.2f} over, worst {float(err.max()):.2e} at {int(err.argmax())}"


def write_model(folder, cfg, w):
    from safetensors.torch import save_file

    with open(folder / "config.json", "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
    return str(folder)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (model folder, config, weights in float64); written with the safetensors library, not with the package's writer."""
    out = {}
    for name, case in ZN.items():
        w = P.random_weights(case["config"], case["seed"])
        out[name] = (write_model(tmp_path_factory.mktemp(f"zn_{name}"), case["config"], w), case["config"], P.as_float64(w))
    return out


_PLAIN = {}


def plain_logits(name, models, tokens):
    key = (name, tuple(tokens))
    if key not in _PLAIN:
        _, cfg, w = models[name]
        _PLAIN[key] = P.forward(cfg, w, list(tokens)).numpy()
    return _PLAIN[key]


def tokens_of(name, n, salt=0):
    rng = random.Random(ZN[name]["seed"] * 1000 + n + salt)
    return [rng.randrange(ZN[name]["config"]["vocab"]) for _ in range(n)]


def make_runner(model_dir, dtype, page_size=16, num_pages=64, max_num_seqs=4, graphs=True):
    from spyinfer_b200.config import EngineConfig, load_model_config
    from spyinfer_b200.engine.model import Model
    from spyinfer_b200.engine.runner import ModelRunner

    spec = load_model_config(model_dir).to_spec()
    config = EngineConfig(dtype=dtype, kvcache_block_size=page_size, num_kvcache_blocks=num_pages, max_num_seqs=max_num_seqs,
                          max_model_len=num_pages * page_size, max_num_batched_tokens=num_pages * page_size, use_cuda_graphs=graphs)
    model = Model(spec, torch.bfloat16 if dtype == "bfloat16" else torch.float32, config.device, config.max_model_len)
    model.load(model_dir)
    return ModelRunner(model, config)


def run_cuts(runner, rid, tokens, cuts, finish=True):
    """The logits of every position of one request fed in portions of the given sizes."""
    from spyinfer_b200.engine.batch import StepEntry

    rows, at = [], 0
    for c in cuts:
        rows.append(runner.step([StepEntry(rid, tokens[at:at + c], list(range(c)))]).float().cpu().numpy().copy())
        at += c
    assert at == len(tokens)
    runner.check_status()
    if finish:
        runner.finish(rid)
    return np.concatenate(rows)


def cycle_cuts(n, sizes):
    cuts, left = [], n
    while left:
        cuts.append(min(left, sizes[len(cuts) % len(sizes)]))
        left -= cuts[-1]
    return cuts


# ---- configuration, cache bookkeeping, the plain mechanisms (no GPU) -------------------------------------------

def test_config_is_found_by_its_architecture_key_and_declares_the_checkpoints_tensors():
    from spyinfer_b200.config import ConfigError, ZonevikConfig, config_from_json
    from spyinfer_b200.engine.model import declared_weights

    for name, case in ZN.items():
        cfg = config_from_json(case["config"])
        assert isinstance(cfg, ZonevikConfig)
        spec = cfg.to_spec()
        declared = {d.name: tuple(d.shape) for d in declared_weights(spec)}
        assert declared == P.tensor_shapes(case["config"]), name
        assert [(e.layer, e.before is not None) for e in spec.run_order] == P.run_order(case["config"]), name
        assert config_from_json(cfg.to_json()).to_json() == cfg.to_json()
    base = ZN["a"]["config"]

    def broken(change):
        c = json.loads(json.dumps(base))
        change(c)
        with pytest.raises(ConfigError):
            config_from_json(c).to_spec()

    broken(lambda c: c["layers"][0].update(type="mamba1"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))                   # 4 heads do not group over 3
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18))               # wider than a head
    broken(lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"))
    broken(lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0))
    broken(lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1))
    broken(lambda c: c["layers"][1]["mixer"]["right"].update(groups=4))            # 6 heads do not form 4 groups
    broken(lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7))
    broken(lambda c: c["layers"][1]["mixer"].pop("right"))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][2]["mixer"].pop("conv"))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))                # more than there are experts
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4))    # 6 experts do not form 4 groups
    broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=5))                # one group of four cannot give five experts
    broken(lambda c: c["loop"].update(stop=5))
    broken(lambda c: c["loop"].update(stop=1))
    broken(lambda c: c["loop"].update(times=0))
    broken(lambda c: c.pop("norm"))


def test_every_pass_of_the_loop_has_a_cache_and_states_of_its_own():
    from spyinfer_b200.cache import CacheManager
    from spyinfer_b200.config import CompositeCacheNeed, PagedCacheNeed, StateCacheNeed, config_from_json
    from spyinfer_b200.engine.model import Model

    model = Model(config_from_json(ZN["a"]["config"]).to_spec(), torch.float32, None, 256)
    needs, cache_of = model.cache_needs()
    assert len(needs) == 8 and cache_of == [None] * 8
    state = lambda n: StateCacheNeed((n,), "float32")
    par = CompositeCacheNeed((PagedCacheNeed(2, 24, 20, keep_first=3), CompositeCacheNeed((state(6 * 12 * 10), state(2 * (60 + 2 * 3 * 12))))))
    delta = CompositeCacheNeed((state(4 * 12 * 20), state(2 * (2 * 2 * 12 + 4 * 20))))
    assert needs[0] == PagedCacheNeed(2, 24, None) and needs[7] == PagedCacheNeed(1, 24, None)       # rows of max(dim, vdim), rounded up to 8
    assert needs[1:7] == [par, delta] * 3
    cache = CacheManager(needs, 8, 40, 2, 320, device=None, cache_of=cache_of, max_step_tokens=16)
    views = [cache.view(i) for i in range(8)]
    windows = [views[i].parts[0] for i in (1, 3, 5)]
    assert len({id(v) for v in windows}) == 3 and all(v.writes for v in windows)
    # one tap leaves no convolution state
    needs, _ = Model(config_from_json(ZN["b"]["config"]).to_spec(), torch.float32, None, 256).cache_needs()
    assert needs[0] == state(3 * 20 * 9) and needs[2] == CompositeCacheNeed((PagedCacheNeed(1, 16, None), state(4 * 40 * 6)))


def test_what_the_plain_mechanisms_do_on_inputs_known_by_hand():
    f64 = lambda *v: torch.tensor(v, dtype=P.F)
    # the norm: no statistics, a row's elements do not see one another
    W = {"n": f64(2.0, 3.0), "n.b": f64(0.5, -1.0), "n.alpha": torch.tensor(0.5, dtype=P.F)}
    assert torch.allclose(P.dynamic_tanh(f64(1.0, -4.0), W, "n"), f64(2.0 * math.tanh(0.5) + 0.5, 3.0 * math.tanh(-2.0) - 1.0))
    # visibility: the window counts the query's own position; kept tokens stay; nothing later is seen
    assert [P.visible(10, j, 3, 2) for j in range(12)] == [True, True, False, False, False, False, False, False, True, True, True, False]
    v = P.visibility(12, 3, 2)
    assert all(bool(v[i, j]) == P.visible(i, j, 3, 2) for i in range(12) for j in range(12))
    # YaRN: the fastest pair keeps its frequency, the slowest is divided by the factor, cos and sin grow
    freqs, mag = P.yarn_frequencies(16, 10000.0, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0})
    plain, one = P.yarn_frequencies(16, 10000.0, None)
    assert one == 1.0 and math.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    assert freqs[0] == plain[0] and math.isclose(freqs[-1], plain[-1] / 4.0) and all(p / 4.0 - 1e-15 <= f <= p for f, p in zip(freqs, plain))
    lo = math.floor(16 * math.log(512 / (2 * math.pi * 32)) / (2 * math.log(10000.0)))
    hi = math.ceil(16 * math.log(512 / (2 * math.pi)) / (2 * math.log(10000.0)))
    ramp = (2 - lo) / (hi - lo)
    assert 0 < ramp < 1 and math.isclose(freqs[2], plain[2] / 4.0 * ramp + plain[2] * (1 - ramp))
    # the convolution's last column meets the current token
    h = torch.tensor([[1.0], [10.0], [100.0]], dtype=P.F)
    assert P.time_conv(h, torch.tensor([[3.0, 2.0]], dtype=P.F)).flatten().tolist() == [2.0, 23.0, 230.0]
    # the delta rule writes what the state lacks: with beta 1, no decay and a unit key the read-out is the value itself
    k = f64(0.6, 0.8).reshape(1, 1, 2).repeat(2, 1, 1)
    val = f64(5.0, -3.0).reshape(2, 1, 1)
    o, S = P.delta_state_walk(k, k, val, torch.ones(2, 1, dtype=P.F), torch.ones(2, 1, dtype=P.F))
    assert torch.allclose(o.flatten(), f64(5.0, -3.0)) and torch.allclose(S.flatten(), f64(-1.8, -2.4))
    o, _ = P.delta_state_walk(k, k, val, torch.full((2, 1), 0.5, dtype=P.F), torch.full((2, 1), 0.25, dtype=P.F))
    assert torch.allclose(o.flatten(), f64(1.25, 0.625 + 0.25 * (-3.0 - 0.625)))      # the decay comes before the read of what is removed
    # the state-space scan by hand
    B, C, x = f64(2.0).reshape(1, 1, 1).repeat(2, 1, 1), f64(3.0).reshape(1, 1, 1).repeat(2, 1, 1), f64(1.0, 4.0).reshape(2, 1, 1)
    o, S = P.ssd_state_walk(B, C, x, f64(0.5, 0.25).reshape(2, 1), f64(math.log(2.0)), f64(10.0))
    s1 = 0.5 * 2.0 * 1.0
    s2 = math.exp(-0.5) * s1 + 0.25 * 2.0 * 4.0
    assert torch.allclose(o.flatten(), f64(3.0 * s1 + 10.0, 3.0 * s2 + 40.0)) and math.isclose(float(S), s2)
    # the choice: the group whose two best scores have the larger sum wins over the one that holds the best expert
    r = {"experts": 4, "top": 1, "groups": {"count": 2, "keep": 1}}
    logit = lambda p: math.log(p / (1.0 - p))
    W = {"router": f64(logit(0.9), logit(0.1), logit(0.6), logit(0.55)).reshape(4, 1)}
    idx, w = P.route(torch.ones(1, 1, dtype=P.F), r, W, "")
    assert idx.tolist() == [[2]] and torch.allclose(w, f64(0.6).reshape(1, 1))
    r["groups"] = {"count": 4, "keep": 2}                                   # groups of one: a group's score is its only expert's
    assert P.route(torch.ones(1, 1, dtype=P.F), r, W, "")[0].tolist() == [[0]]
    # the loop: every pass starts from a projection of the stream and the embedding output
    assert P.run_order(ZN["a"]["config"]) == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]


# ---- kernels alone ---------------------------------------------------------------------------------------

@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_dynamic_tanh_adds_a_result_and_norms_the_stream(dtype):
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(4)
    for rows, n, splits in ((5, 40, 1), (3, 200, 3), (9, 1000, 2), (4, 4096, 7), (601, 256, 2), (2, 50, 1), (7, 6145, 1), (1, 3, 4), (514, 37, 1)):
        h, y = torch.randn(rows, n, generator=g) * 2, torch.randn(splits, rows, n, generator=g)
        ty, tx = ((torch.rand(1, generator=g) + 0.3, (1.0 + 0.3 * torch.randn(n, generator=g)).to(torch.bfloat16), (0.3 * torch.randn(n, generator=g)).to(torch.bfloat16))
                  for _ in range(2))
        name = lambda t: {"n": t[1].double(), "n.b": t[2].double(), "n.alpha": t[0].double()}
        ys = y.double().sum(0) if splits > 1 else y[0].to(dtype).double()
        want_h = h.double() + 0.5 * P.dynamic_tanh(ys, name(ty), "n")
        want_x = P.dynamic_tanh(want_h, name(tx), "n")
        dev = lambda t: tuple(v.cuda() for v in t)
        hd, out = h.cuda(), torch.empty((rows, n), dtype=dtype, device="cuda")
        kernels.dynamic_tanh(hd, y=y.cuda() if splits > 1 else y[0].to(dtype).cuda(), y_norm=dev(ty), y_scale=0.5, norm=dev(tx), out=out)
        tol = dict(atol=2e-6, rtol=2e-6) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
        assert torch.allclose(hd.cpu().double(), want_h, atol=5e-6, rtol=1e-6), (rows, n)
        assert torch.allclose(out.cpu().double(), want_x, **tol)
        # the stream's own sum is 32-bit in both formats, from tiny to saturated arguments
        ramp = torch.cat([torch.logspace(-6, 1.3, n // 2), -torch.logspace(-6, 1.3, n - n // 2)])[None].repeat(rows, 1)
        acc = torch.zeros(rows, n, device="cuda")
        one = (torch.ones(1), torch.ones(n).to(torch.bfloat16), torch.zeros(n).to(torch.bfloat16))
        kernels.dynamic_tanh(acc, y=ramp.cuda(), y_norm=dev(one), norm=dev(tx), out=torch.empty((rows, n), dtype=dtype, device="cuda"))
        assert torch.allclose(acc.cpu().double(), torch.tanh(ramp.double()), rtol=1e-6, atol=1e-12)
        before = hd.clone()
        pick = torch.tensor([rows - 1, 0], dtype=torch.int32, device="cuda")           # gathered rows: the pending result counts, the stream stays
        few = torch.empty((2, n), dtype=torch.float32, device="cuda")
        kernels.dynamic_tanh(hd, y=y[0].cuda(), y_norm=dev(ty), norm=dev(tx), out=few, rows=pick)
        want = P.dynamic_tanh(before.cpu().double() + P.dynamic_tanh(y[0].double(), name(ty), "n"), name(tx), "n")[[rows - 1, 0]]
        assert torch.allclose(few.cpu().double(), want, atol=5e-6) and torch.equal(hd, before)
        kernels.dynamic_tanh(hd, y=y[0].cuda(), y_norm=dev(ty))                        # the sum alone
        assert torch.allclose(hd.cpu().double(), before.cpu().double() + P.dynamic_tanh(y[0].double(), name(ty), "n"), atol=5e-6)


@gpu
@pytest.mark.parametrize("theirs,own", [(torch.float32, torch.bfloat16), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
def test_two_norms_of_one_launch_may_be_stored_in_different_types(theirs, own):
    """What a norm in the one type left behind is formed by one in the other, and neither's weights are rounded."""
    from spyinfer_b200.config import PartSpec
    from spyinfer_b200.parts import BuildContext, build_part

    g = torch.Generator().manual_seed(6)
    n, rows = 72, 5
    ctx = BuildContext(device="cuda", dtype=torch.float32, max_model_len=8)
    norms, plain = [], []
    for dtype in (theirs, own):
        w = {"n": (1.0 + 0.3 * torch.randn(n, generator=g)).to(dtype), "n.b": (0.3 * torch.randn(n, generator=g)).to(dtype), "n.alpha": torch.tensor(0.7).to(dtype)}
        norms.append(build_part(PartSpec("dynamic_tanh", {"size": n, "weight": "n"}), ctx))
        norms[-1].bind({k: v.cuda() for k, v in w.items()})
        plain.append({k: v.double() for k, v in w.items()})
    h, y = torch.randn(rows, n, generator=g), torch.randn(rows, n, generator=g)
    hd = h.cuda()
    out = norms[1].forward_add(hd, norms[0].defer(y.cuda(), 0.5))
    want = h.double() + 0.5 * P.dynamic_tanh(y.double(), plain[0], "n")
    assert torch.allclose(hd.cpu().double(), want, atol=3e-6)
    assert torch.allclose(out.cpu().double(), P.dynamic_tanh(want, plain[1], "n"), atol=3e-6)


@gpu
@pytest.mark.parametrize("dims,base,yarn", [(12, 500.0, (3.0, 64, 8.0, 0.5)), (64, 10000.0, (4.0, 512, 32.0, 1.0)), (16, 100.0, (8.0, 2000, 1.0, 1.0)),
                                            (8, 1e6, (1.0, 4096, 32.0, 1.0)), (24, 10000.0, None), (2, 10.0, (2.0, 5, 64.0, 0.001))])
def test_the_stretched_rotations_table(dims, base, yarn):
    from spyinfer_b200.config import PartSpec
    from spyinfer_b200.parts import BuildContext, build_part

    scaling = dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None
    params = {"theta": base, "rotary_dim": dims}
    if scaling:
        params["yarn_scaling"] = scaling
    table = build_part(PartSpec("rotary_interleaved", params), BuildContext(torch.float32, torch.device("cuda"), 700)).rotation_table().cpu().double()
    freqs, mag = P.yarn_frequencies(dims, base, scaling)
    angle = torch.arange(700, dtype=P.F)[:, None] * torch.tensor(freqs, dtype=P.F)[None]
    assert float((table[..., 0] - mag * torch.cos(angle)).abs().max()) < 7e-5 * mag       # angles of up to 700 radians in 32-bit
    assert float((table[..., 1] - mag * torch.sin(angle)).abs().max()) < 7e-5 * mag


def _paged_setup(lens, page_size, nkv, hd, dtype, seed=0):
    """Block tables of requests of the given lengths over shuffled pages, and an empty cache."""
    rng = random.Random(seed)
    per = [-(-n // page_size) for n in lens]
    ids = list(range(sum(per) + 3))
    rng.shuffle(ids)
    table = torch.full((len(lens), max(per) + 1), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor(ids[at:at + n], dtype=torch.int32)
        at += n
    pages = torch.zeros((len(ids), 2, nkv, page_size, hd), dtype=dtype, device="cuda")
    return table.cuda(), pages


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,page_size,splits,pairing", [
    (4, 2, 16, 24, 8, 8, 1, "interleaved"), (3, 1, 12, 20, 12, 4, 3, "interleaved"), (8, 4, 32, 64, 16, 16, 2, "interleaved"), (16, 1, 128, 128, 64, 16, 1, "interleaved"),
    (20, 1, 7, 5, 4, 8, 2, "interleaved"), (2, 2, 10, 6, 0, 16, 1, "interleaved"), (4, 2, 16, 16, 8, 8, 1, "half"), (2, 1, 160, 192, 10, 16, 4, "interleaved")])
def test_queries_and_cache_rows_of_a_projection(dtype, heads, kv_heads, dim, vdim, rot, page_size, splits, pairing):
    """Two requests' tokens in one batch, at positions that are not the batch's order, from a projection that may be a stack of
    partial sums: queries and cache rows equal the plain rotation of the biased projection, rows are zero behind their content,
    nothing else is written; the gate reads its columns of the same projection."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(heads * 100 + dim)
    hd = (max(dim, vdim) + 7) // 8 * 8
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    lens = [37, 21]
    pos = torch.tensor(list(range(30, 37)) + list(range(5, 21)), dtype=torch.int32)
    seq = torch.tensor([0] * 7 + [1] * 16, dtype=torch.int32)
    T = pos.shape[0]
    proj = torch.randn(splits, T, nq + nk + nv + heads * vdim, generator=g)
    bias = torch.randn(proj.shape[2], generator=g)
    stack = proj.cuda() if splits > 1 else proj[0].to(dtype).cuda()
    pd = (proj.double().sum(0) if splits > 1 else proj[0].to(dtype).double())
    biased = pd + bias.double()
    table, pages = _paged_setup(lens, page_size, kv_heads, hd, dtype)
    rope, spec = None, None
    if rot:
        spec = {"base": 300.0, "dims": rot}
        ang = torch.arange(64, dtype=torch.float64)[:, None] * torch.tensor([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)[None]
        rope = torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).float().cuda()
    q_out = torch.full((T, heads * hd), 7.0, dtype=dtype, device="cuda")
    kernels.qkv_store(stack, 0, nq, nq + nk, bias.cuda(), rope, pos.cuda(), seq.cuda(), q_out, table, pages, heads, kv_heads, dim, vdim, pairing=pairing)

    def rotated(x):
        if pairing == "half" and rot:                      # the same rotation on pairs (i, i + r): reorder, rotate neighbours, reorder back
            order = [e for i in range(rot // 2) for e in (i, i + rot // 2)] + list(range(rot, dim))
            back = [order.index(e) for e in range(dim)]
            return P.rotate_pairs(x[..., order], pos, spec)[..., back]
        return P.rotate_pairs(x, pos, spec)

    q, k = rotated(biased[:, :nq].reshape(T, heads, dim)), rotated(biased[:, nq:nq + nk].reshape(T, kv_heads, dim))
    v = biased[:, nq + nk:nq + nk + nv].reshape(T, kv_heads, vdim)
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=1e-2)
    got_q = q_out.cpu().double().reshape(T, heads, hd)
    assert torch.allclose(got_q[..., :dim], q, **tol) and float(got_q[..., dim:].abs().max() if hd > dim else 0.0) == 0.0
    table_h, pages_h = table.cpu(), pages.cpu().double()
    for t in range(T):
        page, slot = int(table_h[seq[t], pos[t] // page_size]), int(pos[t]) % page_size
        assert torch.allclose(pages_h[page, 0, :, slot, :dim], k[t], **tol) and torch.allclose(pages_h[page, 1, :, slot, :vdim], v[t], **tol)
        assert float(pages_h[page, 0, :, slot, dim:].abs().sum()) == 0.0 and float(pages_h[page, 1, :, slot, vdim:].abs().sum()) == 0.0
    written = {(int(table_h[seq[t], pos[t] // page_size]), int(pos[t]) % page_size) for t in range(T)}
    assert int((pages_h.abs().sum(dim=(1, 2, 4)) > 0).sum()) == len(written)
    # the gate
    attn = torch.randn(T, heads, hd, generator=g).to(dtype)
    want = attn.double()[..., :vdim] * torch.sigmoid(pd[:, nq + nk + nv:]).reshape(T, heads, vdim)
    out = torch.empty((T, heads * vdim), dtype=dtype, device="cuda")
    kernels.gate_heads(attn.reshape(T, heads * hd).cuda(), hd, stack, nq + nk + nv, out, heads, vdim)
    assert torch.allclose(out.cpu().double().reshape(T, heads, vdim), want, **tol)


@gpu
@pytest.mark.parametrize("path", ["plain32", "plain16", "tensor"])
@pytest.mark.parametrize("heads,kv_heads,hd,window,keep,page_size", [(4, 2, 24, 20, 3, 8), (8, 4, 64, 64, 4, 16), (16, 1, 128, 40, 16, 16), (2, 1, 32, 7, 0, 8),
                                                                     (2, 2, 16, 25, 30, 16), (4, 1, 8, 1, 1, 8), (2, 1, 64, 130, 20, 16)])
def test_window_with_kept_first_keys_under_an_ordinary_softmax(path, heads, kv_heads, hd, window, keep, page_size):
    """A portion of a long prompt, a whole prompt and one decoded token over shuffled pages; a few queries point at one key with
    nearly all their weight: the window's oldest key and the one before it, the last kept key and the one after it, a page's
    first and last place."""
    from spyinfer_b200 import kernels

    dtype = torch.float32 if path == "plain32" else torch.bfloat16
    if path == "tensor" and not kernels.attention_tc_takes(heads, kv_heads, hd, dtype):
        pytest.skip("sizes the tensor-core kernels do not take")
    g = torch.Generator().manual_seed(hd + heads)
    lens = [300, 40, 261]
    keys = [torch.randn(n, kv_heads, hd, generator=g).to(dtype).double() for n in lens]
    values = [torch.randn(n, kv_heads, hd, generator=g).to(dtype).double() for n in lens]
    table, pages = _paged_setup(lens, page_size, kv_heads, hd, dtype, seed=3)
    pages_h = pages.cpu()
    for s, n in enumerate(lens):
        for j in range(n):
            page = int(table[s, j // page_size])
            pages_h[page, 0, :, j % page_size], pages_h[page, 1, :, j % page_size] = keys[s][j].to(dtype), values[s][j].to(dtype)
    pages.copy_(pages_h)
    spans = [(2, 260, 261), (0, 150, 300), (1, 0, 40)]            # the decoded token first, as the step function lays a mixed batch out
    pos = torch.tensor([p for _, a, b in spans for p in range(a, b)], dtype=torch.int32)
    seq = torch.tensor([i for i, (_, a, b) in enumerate(spans) for _ in range(a, b)], dtype=torch.int32)
    T = pos.shape[0]
    q = torch.randn(T, heads, hd, generator=g) * 0.5
    first = 1                                                     # the row of request 0's position 150
    for p, target in ((170, 170 - window + 1), (171, 171 - window), (180, keep - 1), (181, keep), (190, (190 // page_size) * page_size),
                      (191, (190 // page_size) * page_size - 1), (210, 0), (299, 299)):
        if 0 <= target <= p:
            q[first + p - 150, 0] = keys[0][target, 0].float() * (12.0 / hd ** 0.5)
    q = q.to(dtype)
    scale, rep, want, at = hd ** -0.5, heads // kv_heads, [], 0
    for s, a, b in spans:                                         # the plain attention of the span's rows over the request's keys
        seen = P.visibility(b, window, keep)[a:b]
        k, v = keys[s][:b].repeat_interleave(rep, dim=1), values[s][:b].repeat_interleave(rep, dim=1)
        sc = torch.einsum("ihd,jhd->hij", q[at:at + b - a].double(), k) * scale
        want.append(torch.einsum("hij,jhd->ihd", torch.softmax(sc.masked_fill(~seen[None], -math.inf), dim=-1), v))
        at += b - a
    want = torch.cat(want)
    table_d = table[[s for s, _, _ in spans]].contiguous()
    qd, out = q.reshape(T, heads * hd).cuda(), torch.empty((T, heads * hd), dtype=dtype, device="cuda")
    if path != "tensor":
        kernels.attention_generic(qd, heads, hd, out, pages, table_d, pos.cuda(), seq.cuda(), scale, window=window, keep_first=keep)
    else:
        q_start = torch.tensor([0, 1, 151, 191], dtype=torch.int32).cuda()
        lse = torch.empty((T, heads), dtype=torch.float32, device="cuda")
        kernels.attention_decode(qd, heads, hd, out, pages, table_d[:1], pos.cuda(), q_start[:2], 1, scale, window=window, lse=lse)
        kernels.attention_tc(qd, heads, hd, out, pages, table_d[1:], pos.cuda(), q_start[1:], 2, scale, window=window, lse=lse)
        kernels.sink_merge(qd, heads, hd, out, lse, pages, table_d, pos.cuda(), seq.cuda(), scale, window, keep, False)
    worst = (out.cpu().double().reshape(T, heads, hd) - want).abs().amax(dim=(1, 2))
    assert float(worst.max()) < (2e-5 if dtype == torch.float32 else 4e-2), f"token {int(worst.argmax())} (position {int(pos[int(worst.argmax())])}): {float(worst.max()):.3e}"


def _scan_case(kind, heads, share, dk, dv, lens, seed, slow):
    """Inputs of one scan for requests of the given lengths and the plain walk's results: (proj columns, gates, parameters, want)."""
    g = torch.Generator().manual_seed(seed)
    T, G = sum(lens), heads // share
    q, k, v = torch.randn(T, G, dk, generator=g), torch.randn(T, G, dk, generator=g), torch.randn(T, heads, dv, generator=g)
    gates = torch.randn(T, 2 * heads, generator=g)
    a_log = 0.5 * torch.randn(heads, generator=g)
    dt_bias = (-6.0 if slow else -2.0) + torch.randn(heads, generator=g)
    d_skip = torch.randn(heads, generator=g)
    S = [torch.randn(heads, dk, dv, generator=g).double() for _ in lens]
    d = lambda t: t.double()
    rep = lambda t: d(t).repeat_interleave(share, dim=1)
    dt = P.softplus(d(gates[:, heads:]) + d(dt_bias))
    want, last, at = [], [], 0
    for i, n in enumerate(lens):
        sl = slice(at, at + n)
        if kind == "delta":
            o, Sn = P.delta_state_walk(P.unit_vector(rep(q[sl])) * dk ** -0.5, P.unit_vector(rep(k[sl])), d(v[sl]), torch.exp(-torch.exp(d(a_log)) * dt[sl]),
                                       torch.sigmoid(d(gates[sl, :heads])), S[i])
        else:
            o, Sn = P.ssd_state_walk(rep(k[sl]), rep(q[sl]), d(v[sl]), dt[sl], d(a_log), d(d_skip), S[i])
        want.append(o)
        last.append(Sn)
        at += n
    proj = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1)
    return proj, gates, a_log, dt_bias, d_skip, S, want, last


SCAN_SIZES = [(4, 2, 12, 20), (3, 3, 20, 9), (6, 1, 64, 32), (8, 4, 128, 64), (2, 1, 128, 128), (5, 1, 7, 11), (4, 4, 33, 50), (2, 2, 256, 40), (16, 8, 16, 64), (2, 1, 300, 24), (1, 1, 643, 16)]


@gpu
@pytest.mark.parametrize("kind", ["delta", "ssd"])
@pytest.mark.parametrize("slow", [False, True])
@pytest.mark.parametrize("heads,share,dk,dv", SCAN_SIZES)
def test_scans_with_one_decay_a_head_in_every_cut(kind, slow, heads, share, dk, dv):
    """Three requests of unequal lengths from states that are not zero, in one step, in portions, and token by token, in slots that
    are not in the batch's order: outputs and states equal the plain walk's, and the slots of other requests are not touched."""
    from spyinfer_b200 import kernels

    lens = [70, 1, 301]
    proj, gates, a_log, dt_bias, d_skip, S, want, last = _scan_case(kind, heads, share, dk, dv, lens, heads * 1000 + dk, slow)
    G = heads // share
    starts = [0, 70, 71]
    slots = [3, 0, 2]
    par = [t.cuda() for t in (a_log, dt_bias, d_skip)]

    def run(state, pieces, longest=None):
        """pieces: (request, first, end) of this step."""
        rows = torch.cat([torch.arange(starts[r] + a, starts[r] + b) for r, a, b in pieces])
        x, gt = proj[rows].cuda(), gates[rows].cuda()
        q_start = torch.tensor(np.cumsum([0] + [b - a for _, a, b in pieces]), dtype=torch.int32).cuda()
        slot = torch.tensor([slots[r] for r, _, _ in pieces], dtype=torch.int32).cuda()
        out = torch.empty((len(rows), heads * dv), dtype=torch.float32, device="cuda")
        status = torch.zeros(2, dtype=torch.int32, device="cuda")
        if kind == "delta":
            kernels.gated_delta_scan(x, (0, G * dk, 2 * G * dk), gt, 0, heads, par[0], par[1], state, q_start, slot, len(pieces), out, heads, share, dk, dv, dk ** -0.5,
                                     status=status, longest=longest)
        else:
            kernels.ssd_scan(x, (2 * G * dk, G * dk, 0), gt, heads, par[0], par[1], par[2], state, q_start, slot, len(pieces), out, heads, share, dk, dv,
                             status=status, longest=longest)
        assert status.cpu().tolist() == [0, 0]
        return {(r, a + i): row for (r, a, b), block in zip(pieces, out.cpu().double().split([b - a for _, a, b in pieces])) for i, row in enumerate(block)}

    def fresh():
        state = torch.full((5, heads * dk * dv), 7.0, device="cuda")
        for s, S0 in zip(slots, S):
            state[s] = S0.reshape(-1).float().cuda()
        return state

    def check(got, state, what):
        scale = max(float(w.abs().max()) for w in want)
        for (r, t), row in got.items():
            err = float((row - want[r][t].reshape(-1)).abs().max()) / scale
            assert err < 2e-5, f"{what}: request {r} token {t} differs by {err:.2e}"
        for s, Sn in zip(slots, last):
            err = float((state[s].cpu().double() - Sn.reshape(-1)).abs().max() / Sn.abs().max())
            assert err < 2e-5, f"{what}: state of slot {s} differs by {err:.2e}"
        assert bool((state[[1, 4]] == 7.0).all()), what

    state = fresh()
    check(run(state, [(0, 0, 70), (1, 0, 1), (2, 0, 301)]), state, "whole")
    state, got, at = fresh(), {}, [0, 0, 0]
    for n in (2, 3, 64, 1, 17, 128, 5, 2, 33, 63, 31, 65, 40, 40):
        pieces = [(r, at[r], min(at[r] + n + r, lens[r])) for r in range(3) if at[r] < lens[r]]
        if not pieces:
            break
        got.update(run(state, pieces, longest=500 if n % 2 else None))
        for r, _, b in pieces:
            at[r] = b
    assert at == lens
    check(got, state, "portions")
    state, got = fresh(), {}
    got.update(run(state, [(0, 0, 40), (2, 0, 280)]))
    for t in range(30):
        pieces = [(0, 40 + t, 41 + t)] + ([(1, 0, 1)] if t == 4 else []) + ([(2, 280 + t, 281 + t)] if t < 21 else [])
        got.update(run(state, pieces, longest=1))
    check(got, state, "decoded")


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_gate_ahead_of_a_norm_in_parts_and_the_sum_of_two_normed_outputs(dtype):
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(2)
    for T, size, groups in ((5, 60, 2), (3, 24, 1), (300, 256, 4), (2, 21, 3), (7, 8192, 8), (4, 6000, 1)):
        o, proj, w = torch.randn(T, size, generator=g) * 2, torch.randn(T, size + 12, generator=g), 1.0 + 0.3 * torch.randn(size, generator=g)
        for off in (4, 7):
            y = o.double() * P.silu(proj[:, off:off + size].double())
            want = P.unit_rms(y.reshape(T, groups, size // groups), 1e-5).reshape(T, size) * w.double()
            out = torch.empty((T, size), dtype=dtype, device="cuda")
            kernels.gate_group_norm(o.cuda(), proj.cuda(), off, w.cuda(), out, groups, 1e-5)
            assert torch.allclose(out.cpu().double(), want, atol=2e-5 if dtype == torch.float32 else 3e-2, rtol=1e-5 if dtype == torch.float32 else 1e-2)
    for T, n, sa, sb in ((5, 64, 1, 1), (3, 100, 3, 1), (40, 4096, 1, 4), (2, 2050, 2, 2), (1, 7, 1, 1)):
        a, b = torch.randn(sa, T, n, generator=g) * 3, torch.randn(sb, T, n, generator=g) * 0.1
        wa, wb = 1.0 + torch.randn(n, generator=g), torch.randn(n, generator=g)
        ad, bd = (t.double().sum(0) if t.shape[0] > 1 else t[0].to(dtype).double() for t in (a, b))
        want = 0.5 * P.unit_rms(ad, 1e-6) * wa.double() + 0.25 * P.unit_rms(bd, 1e-6) * wb.double()
        out = torch.empty((T, n), dtype=torch.float32, device="cuda")
        dev = lambda t: t.cuda() if t.shape[0] > 1 else t[0].to(dtype).cuda()
        kernels.normed_sum(out, dev(a), wa.cuda(), 0.5, dev(b), wb.cuda(), 0.25, 1e-6)
        assert torch.allclose(out.cpu().double(), want, atol=1e-5, rtol=1e-5)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_stream_beside_the_embedding_output(dtype):
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(6)
    for T, n in ((5, 40), (33, 256), (2, 101)):
        h, table = torch.randn(T, n, generator=g), torch.randn(19, n, generator=g).to(torch.bfloat16)
        ids = torch.randint(0, 19, (T,), generator=g, dtype=torch.int32)
        out = torch.empty((T, 2 * n), dtype=dtype, device="cuda")
        status = torch.zeros(2, dtype=torch.int32, device="cuda")
        kernels.stream_concat(h.cuda(), table.cuda(), ids.cuda(), 2.5, out, status)
        want = torch.cat([h.double(), 2.5 * table[ids.long()].double()], dim=1)
        assert torch.allclose(out.cpu().double(), want, atol=1e-6 if dtype == torch.float32 else 4e-2) and status.cpu().tolist() == [0, 0]
        ids[1] = 19                                                # an id outside the table is refused, not read
        kernels.stream_concat(h.cuda(), table.cuda(), ids.cuda(), 2.5, out, status)
        assert status.cpu().tolist() == [1, 1] and float(out[1, n:].abs().max()) == 0.0


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,groups", [(6, 2, 24, (3, 2)), (8, 3, 16, (2, 1)), (5, 1, 16, (5, 3)), (4, 4, 12, None), (16, 4, 32, (4, 2)), (4, 4, 12, (2, 2)),
                                                   (2, 1, 16, (2, 1)), (60, 6, 8, (10, 3)), (3, 2, 24, (1, 1))])
def test_sigmoid_scores_and_groups_by_their_two_best(dtype, experts, top, ff, groups):
    """The kernel's weights equal the plain choice's (an expert that is not chosen weighs exactly zero), its activations are
    weight * silu(gate) * up; the sorted pairs hold the same choice."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(experts * 10 + top)
    T = 60
    logits = torch.randn(T, experts, generator=g) * 1.5
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    idx, w = P.route(logits.double(), r, {"router": torch.eye(experts, dtype=P.F)}, "")
    want_w = torch.zeros(T, experts, dtype=P.F).scatter_(1, idx, w)
    gu = torch.randn(T, 2 * experts * ff, generator=g).to(dtype)
    y = torch.empty((T, experts * ff), dtype=dtype, device="cuda")
    weights = torch.empty((T, experts + 1), dtype=torch.float32, device="cuda")
    kernels.moe_activation(gu.cuda(), logits.cuda(), y, experts, top, ff, 0.0, weights_out=weights, groups=groups, activation="silu", scoring="sigmoid",
                           group_score="best_two")
    got_w = weights.cpu().double()[:, :experts]
    assert torch.equal(got_w != 0, want_w != 0) and torch.allclose(got_w, want_w, atol=1e-6)
    a = gu.double().reshape(T, experts, 2, ff)
    want = (want_w[:, :, None] * P.silu(a[:, :, 0]) * a[:, :, 1]).reshape(T, -1)
    assert torch.allclose(y.cpu().double(), want, atol=1e-5 if dtype == torch.float32 else 2e-2, rtol=1e-5 if dtype == torch.float32 else 1e-2)
    offsets, slot, row_token, row_w, _, _ = kernels.moe_route_general(logits.cuda(), experts, top, 0, None, groups, False, scoring="sigmoid", group_score="best_two")
    offsets, slot, row_token, row_w = offsets.cpu().tolist(), slot.cpu(), row_token.cpu(), row_w.cpu()
    assert offsets[experts] == T * top
    for e in range(experts):
        rows = range(offsets[e], offsets[e + 1])
        assert [int(row_token[i]) for i in rows] == [t for t in range(T) if want_w[t, e] != 0]
        assert np.allclose([float(row_w[i]) for i in rows], [float(x) for x in want_w[:, e] if x != 0], atol=1e-6)


@gpu
@pytest.mark.parametrize("experts,top,hidden,ff,T", [(6, 2, 64, 24, 50), (8, 3, 136, 200, 700), (1, 1, 256, 64, 300), (5, 1, 40, 16, 9), (16, 4, 512, 320, 1100)])
def test_one_launch_multiplies_every_tile_with_its_own_experts_weight(experts, top, hidden, ff, T):
    """Pairs sorted by expert into runs of whole tiles: every pair has a row of its own expert's run, the rows between belong to nobody,
    and the two products (row parts of one fused weight, column parts of another) equal each expert's own; an expert that nobody
    chose has no tile."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(T + ff)
    logits = torch.randn(T, experts, generator=g) * 1.5
    if experts > 2:
        logits[:, 1] = -30.0                                       # an expert without rows
    idx = torch.topk(torch.sigmoid(logits), top, dim=-1).indices.sort(dim=-1).values
    pad = kernels.grouped_tile_rows()
    offsets, slot, row_token, row_w, _, _, tiles = kernels.moe_route_general(logits.cuda(), experts, top, scoring="sigmoid", pad=pad)
    starts, slots, tokens, owner = offsets.cpu().tolist(), slot.cpu(), row_token.cpu(), tiles.cpu().tolist()
    assert all(v % pad == 0 for v in starts) and tokens.shape[0] == len(owner) * pad >= starts[experts]
    for t in range(T):
        for k in range(top):
            r = int(slots[t, k])
            assert int(tokens[r]) == t and owner[r // pad] == int(idx[t, k])
    assert int((tokens >= 0).sum()) == T * top and owner[starts[experts] // pad:] == [-1] * (len(owner) - starts[experts] // pad)
    x = torch.randn(T, hidden, generator=g).to(torch.bfloat16)
    w = (torch.randn(experts * 2 * ff, hidden, generator=g) / hidden ** 0.5).to(torch.bfloat16)
    rows = kernels.gather_rows(x.cuda(), row_token, torch.empty((tokens.shape[0], hidden), dtype=torch.bfloat16, device="cuda"))
    gu = kernels.gemm_grouped(rows, w.cuda(), tiles, experts, 2 * ff, row_step=2 * ff)
    d = (torch.randn(hidden, experts * ff, generator=g) / ff ** 0.5).to(torch.bfloat16)
    y = torch.randn(tokens.shape[0], ff, generator=g).to(torch.bfloat16)
    down = kernels.gemm_grouped(y.cuda(), d.cuda(), tiles, experts, hidden, col_step=ff, out_dtype=torch.float32)
    gu, down = gu.float().cpu().double(), down.cpu().double()
    for e in range(experts):
        mine = [r for r in range(starts[e], starts[e + 1]) if tokens[r] >= 0]
        if not mine:
            continue
        want = x[tokens[mine].long()].double() @ w[2 * ff * e:2 * ff * (e + 1)].double().T
        assert torch.allclose(gu[mine], want, atol=2e-2, rtol=1e-2), e
        assert torch.allclose(down[mine], y[mine].double() @ d[:, ff * e:ff * (e + 1)].double().T, atol=1e-4, rtol=1e-4), e


# ---- whole models through the step function ---------------------------------------------------------------

@gpu
@pytest.mark.parametrize("name", sorted(ZN))
def test_the_stream_after_every_layer(models, name):
    """The 32-bit path's residual stream after every layer run (what a layer left pending added) equals the plain model's."""
    from spyinfer_b200.engine.batch import StepEntry

    runner = make_runner(models[name][0], "float32", graphs=False)
    toks = tokens_of(name, 45)
    got, blocks = [], {id(l.block): l.block for l in runner.model.layers}

    def watch(block):
        inner = block.forward

        def forward(hidden, delta, batch, cache):
            hidden, delta = inner(hidden, delta, batch, cache)
            got.append(block.settle(hidden.clone(), delta).cpu().double())
            return hidden, delta
        block.forward = forward

    for b in blocks.values():
        watch(b)
    runner.step([StepEntry("r", toks, [44])])
    streams = []
    P.forward(models[name][1], models[name][2], toks, streams=streams)
    assert len(got) == len(streams) == len(runner.model.spec.run_order)
    for i, (a, b) in enumerate(zip(got, streams)):
        assert float((a - b).abs().max() / b.abs().max()) < 1e-4, f"layer run {i}"


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ZN))
def test_whole_prompts_token_by_token_and_portions_agree_with_the_plain_model(models, name, dtype):
    runner = make_runner(models[name][0], dtype)
    for n in (1, 2, 3, 47, 150):
        toks = tokens_of(name, n)
        want = plain_logits(name, models, toks)
        whole = run_cuts(runner, "w", toks, [n])
        agrees(whole, want, dtype, f"{n} tokens at once")
        if n >= 47:
            one_by_one = run_cuts(runner, "d", toks, [n - 40] + [1] * 40)
            agrees(one_by_one, want, dtype, f"{n} tokens, the last 40 one by one")
            portions = run_cuts(runner, "p", toks, cycle_cuts(n, [2, 3, 2, 17, 2, 5, 31, 2, 64]))
            agrees(portions, want, dtype, f"{n} tokens in portions")
            if dtype == "float32":                      # the cut must not show beyond rounding
                scale = np.abs(whole).max()
                assert np.abs(one_by_one - whole).max() / scale < CUTS and np.abs(portions - whole).max() / scale < CUTS
    runner.cache.check_invariants()
    assert runner.cache.num_free_slots() == 4


@gpu
@pytest.mark.parametrize("name", sorted(ZN))
def test_long_decoding_passes_windows_and_pages(models, name):
    """260 tokens, all but the first three one by one (through the decode graphs): every window passes over decoded tokens,
    every page border is crossed by a decoded token, and the windowed groups give their pages back but for the first ones."""
    runner = make_runner(models[name][0], "float32", page_size=8, num_pages=40)
    toks = tokens_of(name, 260, salt=1)
    got = run_cuts(runner, "long", toks, [3] + [1] * 257)
    agrees(got, plain_logits(name, models, toks), "float32", "decoded")
    assert runner.graph_steps > 200


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ZN))
def test_unequal_batches_with_pages_and_slots_used_again(models, name, dtype):
    """Up to three live requests, portions of some beside decoded tokens of others, in a pool so small that every page
    and slot that is given back is needed again; each row equals the plain model's row for its request and position."""
    from spyinfer_b200.engine.batch import StepEntry

    rng = random.Random(9)
    reqs = {f"q{n}": tokens_of(name, n, salt=2) for n in (90, 5, 61, 2, 130, 33, 75)}
    b = TraceBuilder()
    mixed_trace(b, reqs, {r: max(1, len(t) - 25) for r, t in reqs.items()}, rng, max_live=3, portion_sizes=(7, 2, 19, 3, 40, 2))
    pages = -(-peak_tokens(b, round_to=8) // 8)
    runner = make_runner(models[name][0], dtype, page_size=8, num_pages=pages, max_num_seqs=3)
    got, want = [], []
    for st, rows in zip(b.steps, b.rows):
        logits = runner.step([StepEntry(e["id"], e["tokens"], e["want"]) for e in st["entries"]]).float().cpu().numpy()
        for (rid, pos), row in zip(rows, logits):
            got.append(row)
            want.append(plain_logits(name, models, reqs[rid])[pos])
        for rid in st["end"]:
            runner.finish(rid)
    runner.check_status()
    agrees(np.stack(got), np.stack(want), dtype, "mixed steps")
    runner.cache.check_invariants()
    assert runner.cache.num_free_slots() == 3


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "c", "d"])
def test_four_decoding_requests_beside_a_prompt_portion(models, name, dtype):
    """From four one-token requests on, a mixed step lays them out first and their attention takes the kernel made for
    decoding while the portion beside them takes the one for portions; every row still equals the plain model's."""
    from spyinfer_b200.engine.batch import StepEntry

    runner = make_runner(models[name][0], dtype, page_size=16, num_pages=60, max_num_seqs=5)
    olds = {f"o{n}": tokens_of(name, n, salt=5) for n in (70, 90, 33, 120)}
    new = tokens_of(name, 150, salt=6)
    for rid, toks in olds.items():                       # all but the last ten tokens of each
        runner.step([StepEntry(rid, toks[:-10], [])])
    got, want, at = [], [], 0
    for k, n in enumerate((37, 2, 41, 16, 3, 20, 5, 9, 11, 6)):
        entries = [StepEntry("new", new[at:at + n], list(range(n)))]
        entries[1:1] = [StepEntry(rid, [toks[len(toks) - 10 + k]], [0]) for rid, toks in olds.items()]     # the portion first, then the four
        logits = runner.step(entries).float().cpu().numpy()
        got += [logits[:n]] + [logits[n + j][None] for j in range(4)]
        want += [plain_logits(name, models, new)[at:at + n]] + [plain_logits(name, models, toks)[len(toks) - 10 + k][None] for toks in olds.values()]
        at += n
    runner.check_status()
    assert at == len(new)
    agrees(np.concatenate(got), np.concatenate(want), dtype, "four decoding beside a portion")


def _pointing_model(tmp_path, kind, window, keep, dim=32):
    """A one-layer model without a feed-forward whose weights are made so that the token ``A`` as a query points at the token ``B``
    as a key with a large score on its first head: the key projection takes B's normed input to the direction of A's query.  In
    a rotated layer both lie in the elements that are not rotated, so the two may stand anywhere.  The second head's queries are
    so small that it weighs all visible keys nearly alike, so its result moves when one key too many or too few is seen."""
    if kind == "parallel":
        mixer = {"left": _attn(2, 1, dim, 12, 1.0, mask=(window, keep) if window else None), "right": _ssd(2, 8, 8, 1, 2, 1)}
        p = "l0.mix.left."
    else:
        mixer, p = _attn(2, 1, dim, 12, 1.0, rot=(1000.0, 8), yarn=(4.0, 64, 8.0, 1.0)), "l0.mix."
    cfg = {"architecture": "Zonevik", "vocab": 60, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "loop": None,
           "layers": [_layer(kind, mixer, None)]}
    w = P.as_float64(P.random_weights(cfg, 77))
    A, B = 58, 59
    h = P.dynamic_tanh(w["embed"], w, "l0.norm1")
    w[p + "q"][dim:] *= 1e-3
    w[p + "q"][:8] = 0.0                                             # the rotated elements of the first head take no part
    q = w[p + "q"][:dim] @ h[A]
    if kind == "parallel":
        w[p + "q.b"].zero_()
        w[p + "k.b"].zero_()
        w["l0.mix.right.out"] *= 1e-2
    w[p + "k"] *= 0.05
    b = h[B] - h.mean(0)                                             # what sets B's input apart from the others'
    w[p + "k"] += 25.0 / float(q @ q) * torch.outer(q, b / (b @ h[B]))
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    d_ = tmp_path / f"point_{kind}_{window}_{keep}"
    d_.mkdir()
    return write_model(d_, cfg, w), cfg, P.as_float64(w), A, B


def _pointing_case(tmp_path, kind, window, keep):
    model_dir, cfg, w, A, B = _pointing_model(tmp_path, kind, window, keep)
    rng = random.Random(5)
    n = 400
    toks = [rng.randrange(50) for _ in range(n)]
    if window:
        # keys among the kept first tokens (the last kept place) and right behind them; far back; at a page's first and last place.
        # queries: the key is the window's oldest place, one before it, just kept, just not kept
        keys = [keep - 1, keep, 200, 303, 304]
        asks = [200 + window - 1, 200 + window, 150, 390, 305, 304 + window, 10]
        sees = [[200, keep - 1], [keep - 1], [keep - 1], [keep - 1], [303, 304, keep - 1], [keep - 1], [keep - 1, keep]]
    else:
        keys = [300, 1]
        asks = [301, 399, 304, 303, 350, 2, 17]
        sees = [[300, 1], [300, 1], [300, 1], [300, 1], [300, 1], [1], [1]]
    for k in keys:
        toks[k] = B
    for a in asks:
        toks[a] = A
    probs = []
    want = P.forward(cfg, w, toks, probs=probs).numpy()
    first_head = probs[0][0]                                       # [query, key] of the first head
    for a, seen in zip(asks, sees):
        seen = [k for k in seen if k <= a]
        unseen = [k for k in keys if k not in seen]
        on_seen = float(first_head[a, seen].sum()) if seen else 1.0
        assert on_seen > 0.8 and float(first_head[a, unseen].sum() if unseen else 0.0) < 1e-9, (a, on_seen)
    return model_dir, toks, want, asks, keys


POINTING = [("attention", None, 0), ("parallel", None, 0), ("parallel", 40, 6), ("parallel", 24, 17)]


def test_the_plain_model_points_where_the_test_wants_it_to(tmp_path):
    for case in POINTING:
        _pointing_case(tmp_path, *case)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,window,keep", POINTING)
def test_a_query_that_points_at_one_key_finds_it_far_back_and_at_every_edge(tmp_path, dtype, kind, window, keep):
    """The key token stands a few times in a sequence of 400 others; the query token is asked at places where the key is far
    back, at a page's first or last place, at the window's oldest place and one beyond it, and among the kept first tokens
    or right behind them.  The engine's logits equal the plain model's, whole, in portions that cut windows and pages
    anywhere, and decoded one by one."""
    model_dir, toks, want, asks, keys = _pointing_case(tmp_path, kind, window, keep)
    n = len(toks)
    runner = make_runner(model_dir, dtype, page_size=16, num_pages=30)
    tol = TOL[dtype]

    def check(got, what):
        worst = np.abs(got - want).max(axis=1) / np.abs(want).max()
        assert worst[asks].max() < tol, f"{what}: asked position {asks[int(worst[asks].argmax())]}: {worst[asks].max():.2e}"
        assert worst.max() < tol, f"{what}: position {int(worst.argmax())}: {worst.max():.2e}"

    check(run_cuts(runner, "w", toks, [n]), "whole")
    check(run_cuts(runner, "d", toks, [99, 2] + [1] * (n - 101)), "decoded")
    check(run_cuts(runner, "p", toks, cycle_cuts(n, [3, 61, 2, 16, 2, 45, 7])), "portions")
    if window:                                                     # portions that end and start exactly where the window's edge passes a key
        check(run_cuts(runner, "e", toks, [keep, 200 - keep, window - 1, 1, 1, n - 200 - window - 1]), "portions at the edges")


@gpu
def test_the_replay_program_runs_the_model(models, tmp_path):
    name = "a"
    rng = random.Random(2)
    reqs = {f"r{n}": tokens_of(name, n, salt=3) for n in (40, 3, 77, 25)}
    b = TraceBuilder()
    b.whole("whole", reqs["r77"])
    mixed_trace(b, reqs, {r: max(1, len(t) - 10) for r, t in reqs.items()}, rng, max_live=4, portion_sizes=(5, 2, 16))
    for dtype in ("float32", "bfloat16"):
        out = run_trace(models[name][0], dtype, b, str(tmp_path / dtype), peak_tokens(b), ZN[name]["config"]["vocab"])
        keys = sorted(out)
        got = np.stack([out[k] for k in keys])
        want = np.stack([plain_logits(name, models, reqs["r77" if rid == "whole" else rid])[pos] for rid, pos in keys])
        agrees(got, want, dtype, "replayed")


@gpu
@pytest.mark.parametrize("name", ["a", "b", "e"])
def test_greedy_generation_through_the_engine_and_its_scheduler(models, name):
    """Five prompts of unequal length, three slots, prompts cut by a small token budget, pages so few that requests wait
    and are preempted: the tokens equal the plain model's greedy continuation."""
    from spyinfer_b200 import LLMEngine, SamplingParams

    model_dir, cfg, w = models[name]
    prompts = [tokens_of(name, n, salt=4) for n in (30, 3, 55, 1, 18)]
    new = 12
    engine = LLMEngine(model_dir, dtype="float32", max_num_seqs=3, max_num_batched_tokens=24, kvcache_block_size=8, num_kvcache_blocks=20,
                       max_model_len=128)
    got = engine.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    for prompt, out in zip(prompts, got):
        toks = list(prompt)
        for i in range(new):
            logits = P.forward(cfg, w, toks)[-1]
            top = torch.topk(logits, 2).values
            if (top[0] - top[1]).item() < 1e-3:                    # the greedy choice must not hang on rounding: follow the engine from here
                assert out[i] in torch.topk(logits, 2).indices.tolist()
                toks.append(out[i])
                continue
            toks.append(int(logits.argmax()))
            assert out[i] == toks[-1], (i, out, toks[len(prompt):])
    assert engine.stats()["free_slots"] == 3


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ZN))
def test_the_routed_mixture_agrees_with_the_plain_model_and_with_the_dense_form(models, name, dtype, monkeypatch):
    """Steps of eight tokens or more take the routed form (each expert's products on its own rows), shorter ones and decoding the
    dense one; both agree with the plain model, and in float32 with each other to rounding."""
    toks = tokens_of(name, 150, salt=8)
    want = plain_logits(name, models, toks)
    dense = run_cuts(make_runner(models[name][0], dtype), "w", toks, [150])
    monkeypatch.setenv("SPYINFER_MOE_ROUTED_FROM", "8")
    runner = make_runner(models[name][0], dtype, graphs=False)
    whole = run_cuts(runner, "w", toks, [150])
    agrees(whole, want, dtype, "routed, whole")
    portions = run_cuts(runner, "p", toks, cycle_cuts(150, [2, 31, 8, 3, 64, 9]))
    agrees(portions, want, dtype, "routed and dense portions")
    if dtype == "float32":
        scale = np.abs(dense).max()
        assert np.abs(whole - dense).max() / scale < CUTS and np.abs(portions - dense).max() / scale < CUTS


# ---- configurations drawn at random -------------------------------------------------------------------------

def random_config(rng):
    """A configuration with every size, option and layer order drawn at random."""
    def divisor(n):
        return rng.choice([d for d in range(1, n + 1) if n % d == 0])

    def attention(masked):
        heads, dim = rng.choice([1, 2, 4, 8, 16, 3, 6, 20, 32]), rng.choice([8, 16, 32, 64, 128, 24, 48, 192, 10])
        rot = yarn = mask = None
        if not masked and rng.random() < 0.85:
            rot = (rng.choice([10000.0, 500000.0, 100.0]), rng.choice(range(2, dim + 1, 2)))
            if rng.random() < 0.8:
                yarn = (rng.choice([1.0, 2.0, 4.0, 16.0]), rng.choice([32, 128, 512]), rng.choice([32.0, 8.0, 2.0]), rng.choice([1.0, 0.5]))
        if masked and rng.random() < 0.9:
            mask = (rng.choice([1, 5, 16, 17, 33, 64, 100, 200, 1000]), rng.choice([0, 1, 2, 4, 8, 16, 17, 40]))
        return _attn(heads, divisor(heads), dim, rng.choice([8, 16, 32, 64, 128, 40, dim, dim]), rng.choice([dim ** -0.5, 0.13, 0.2]), rot, yarn, mask)

    def mixer(kind):
        if kind == "attention":
            return attention(False)
        if kind == "delta":
            heads = rng.choice([1, 2, 3, 4, 6, 8])
            return _delta(heads, divisor(heads), rng.choice([8, 16, 32, 64, 128, 20]), rng.choice([8, 16, 32, 64, 128, 18]), rng.choice([1, 2, 3, 4, 4, 6]))
        heads, vdim = rng.choice([1, 2, 4, 6, 8, 12]), rng.choice([8, 16, 32, 64, 10])
        return {"left": attention(True), "right": _ssd(heads, vdim, rng.choice([8, 16, 32, 64, 128, 24]), divisor(heads), rng.choice([1, 2, 3, 4, 4, 6]),
                                                       divisor(heads * vdim))}

    def mlp():
        if rng.random() < 0.12:
            return None
        count = rng.randrange(1, 5)
        experts = count * rng.randrange(1, 6)
        keep = rng.randrange(1, count + 1)
        return _moe(experts, rng.randrange(1, min(keep * (experts // count), 5) + 1), rng.choice([16, 32, 64, 24, 12]), groups=(count, keep))

    layers = [_layer(kind, mixer(kind), mlp()) for kind in (rng.choice(["attention", "delta", "parallel"]) for _ in range(rng.randrange(2, 7)))]
    cfg = {"architecture": "Zonevik", "vocab": rng.randrange(50, 600), "width": rng.choice([64, 96, 128, 160, 192, 256, 320]),
           "norm": {"eps": rng.choice([1e-5, 1e-6])}, "embedding": {"scale": rng.choice([1.0, 2.0, 4.0, 0.5, 7.5])}, "layers": layers, "loop": None}
    if rng.random() < 0.8:
        start = rng.randrange(0, len(layers))
        cfg["loop"] = {"start": start, "stop": rng.randrange(start + 1, len(layers) + 1), "times": rng.randrange(1, 4)}
    return cfg


@gpu
@pytest.mark.parametrize("seed", [3, 11, 19, 27, 42, 58, 77, 91])
def test_configurations_drawn_at_random_agree_with_the_plain_model_in_every_cut(tmp_path, seed):
    """Whole, the last 60 tokens one by one, and portions down to two tokens, in both formats; in float32 the cuts agree with each
    other to rounding."""
    rng = random.Random(seed)
    cfg = random_config(rng)
    w = P.random_weights(cfg, seed)
    model_dir = write_model(tmp_path, cfg, w)
    n = 330
    toks = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    want = P.forward(cfg, P.as_float64(w), toks).numpy()
    for dtype in ("float32", "bfloat16"):
        runner = make_runner(model_dir, dtype, page_size=16, num_pages=64)
        whole = run_cuts(runner, "w", toks, [n])
        one_by_one = run_cuts(runner, "d", toks, [n - 60] + [1] * 60)
        portions = run_cuts(runner, "p", toks, cycle_cuts(n, [2, 3, 2, 17, 2, 5, 31, 2, 64, 129]))
        for what, got in (("whole", whole), ("decoded", one_by_one), ("portions", portions)):
            agrees(got, want, dtype, f"{json.dumps(cfg)}: {what}")
        if dtype == "float32":
            scale = np.abs(whole).max()
            assert np.abs(one_by_one - whole).max() / scale < CUTS and np.abs(portions - whole).max() / scale < CUTS
