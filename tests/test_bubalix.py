"""The Bubalix decoder in the engine against the plain implementation of ``plain_bubalix.py``: each mechanism's kernel alone,
then whole models of several small configurations through the step function (whole prompts, token by token, portions down
to two tokens, unequal batches, pages and slots used again, long decoding), the replay program, and greedy generation through
``LLMEngine`` and its scheduler.  Where random weights would hide a fault (one key among hundreds, a window's edge, a sink, a page
border) the weights are made so that one score stands out."""
import json
import math
import random

import numpy as np
import pytest
import torch

import plain_bubalix as P
from trace_tools import TraceBuilder, mixed_trace, peak_tokens, run_trace

gpu = pytest.mark.gpu


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=None, yarn=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if base is not None:
        m["rot"] = {"base": base, "dims": rot_dim}
        if yarn is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return m


def _attn(heads, kv_heads, dim, vdim, scale, conv, cap=None, temp=None, window=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if cap is not None:
        m["softcap"] = cap
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def _moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _layer(mixer, mlp):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def _config(vocab, width, eps, scale, side, layers):
    cfg = {"architecture": "Bubalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


# Six configurations that differ in every size and option.  a: both kinds of layer in turns, values wider and narrower than keys, all
# three bands of the stretched rotation, a window that is no multiple of a page, three taps, two experts a token and a shared one.
# b: no mask, no cap, no temperature, one tap (no convolution state), a plain rotation, one expert a token, no shared expert, a layer
# without experts, no stretch of the embedding.  c: sizes that the tensor-core products and attention take, sixteen heads on one
# latent, caps below and above the one that may serve as the softmax's reference, a window of whole pages.  d: more heads than the
# tensor-core attention takes and odd sizes (the plain attention kernel on both paths), five taps, every expert chosen, no token
# input.  e: a window of one token, keys and values as many as heads, no rotated part at all and one wider than the latent.  f: a width that is no
# multiple of 8 (the CUDA-core products on both paths), sixteen taps, heads and a cache row wider than the tensor-core attention takes.
BX = {
    "a": dict(seed=51, config=_config(211, 64, 1e-5, 2.5, 12, [
        _layer(_latent(4, 12, 8, 20, 24, 0.25, 500.0, (3.0, 64, 8.0, 0.5)), _moe(6, 2, 24, 40)),
        _layer(_attn(4, 2, 16, 24, 0.3, 3, cap=12.0, temp=(0.4, 16), window=20), _moe(5, 2, 16, 24)),
        _layer(_attn(6, 3, 24, 8, 0.25, 3, cap=8.0, temp=(0.7, 33), window=37), _moe(6, 3, 24, 40)),
        _layer(_latent(2, 24, 12, 8, 20, 0.2, 10000.0, (2.0, 40, 16.0, 1.0)), _moe(6, 2, 24, 16)),
    ])),
    "b": dict(seed=52, config=_config(157, 40, 1e-6, 1.0, 8, [
        _layer(_attn(3, 1, 12, 20, 0.35, 1), _moe(4, 1, 16)),
        _layer(_latent(1, 16, 6, 24, 10, 0.3, 100.0), None),
        _layer(_attn(3, 3, 20, 12, 0.25, 1, window=300), _moe(3, 1, 12)),
    ])),
    "c": dict(seed=53, config=_config(509, 128, 1e-6, 4.0, 32, [
        _layer(_attn(8, 4, 64, 64, 0.125, 4, cap=30.0, temp=(0.3, 50), window=64), _moe(8, 2, 32, 64)),
        _layer(_latent(16, 32, 32, 48, 96, 0.125, 500000.0, (8.0, 128, 32.0, 1.0)), _moe(8, 1, 64, 32)),
        _layer(_attn(16, 1, 128, 128, 0.09, 4, cap=50.0, window=96), None),
        _layer(_attn(4, 4, 64, 32, 0.125, 2, temp=(0.5, 10)), _moe(16, 4, 32)),
        _layer(_latent(8, 64, 16, 64, 48, 0.11, 10000.0, (4.0, 64, 16.0, 0.5)), _moe(8, 2, 32, 64)),
    ])),
    "d": dict(seed=54, config=_config(97, 48, 1e-5, 0.5, 0, [
        _layer(_attn(20, 1, 7, 5, 0.4, 5, cap=5.0, temp=(1.5, 3), window=25), _moe(4, 4, 12, 7)),
        _layer(_latent(20, 9, 2, 11, 13, 0.3, 50.0, (8.0, 20, 4.0, 1.0)), _moe(2, 2, 20)),
    ])),
    "e": dict(seed=55, config=_config(131, 80, 1e-6, 3.0, 20, [
        _layer(_attn(4, 4, 24, 24, 0.2, 2, cap=20.0, temp=(0.5, 64), window=1), _moe(2, 1, 16, 8)),
        _layer(_latent(4, 16, 0, 16, 32, 0.25), _moe(3, 2, 24, 16)),
        _layer(_latent(2, 8, 24, 16, 16, 0.2, 100.0, (8.0, 2000, 1.0, 1.0)), _moe(2, 1, 16)),
    ])),
    "f": dict(seed=56, config=_config(83, 100, 1e-5, 1.5, 10, [
        _layer(_latent(2, 40, 20, 50, 150, 0.13, 2000.0, (2.0, 30, 6.0, 1.0)), _moe(7, 2, 20, 12)),
        _layer(_attn(2, 1, 160, 192, 0.08, 16, cap=18.0, temp=(0.2, 7), window=50), _moe(4, 3, 20)),
        _layer(_attn(6, 3, 40, 36, 0.16, 6, cap=40.0), None),
    ])),
}
TOL = {"float32": 2e-4, "bfloat16": 6e-2}      # largest difference over the largest logit
CUTS = 8e-6                                     # between two cuts of one prompt in float32


def agrees(got, want, dtype, what=""):
    err = np.abs(got - want).max(axis=-1) / np.abs(want).max()
    assert err.max() < TOL[dtype], f"{what}: position {int(err.argmax())} differs by {float(err.max()):.2e} (median {float(np.median(err)):.2e})"


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
    for name, case in BX.items():
        w = P.random_weights(case["config"], case["seed"])
        out[name] = (write_model(tmp_path_factory.mktemp(f"bx_{name}"), case["config"], w), case["config"], P.as_float64(w))
    return out


_PLAIN = {}


def plain_logits(name, models, tokens):
    key = (name, tuple(tokens))
    if key not in _PLAIN:
        _, cfg, w = models[name]
        _PLAIN[key] = P.forward(cfg, w, list(tokens)).numpy()
    return _PLAIN[key]


def tokens_of(name, n, salt=0):
    rng = random.Random(BX[name]["seed"] * 1000 + n + salt)
    return [rng.randrange(BX[name]["config"]["vocab"]) for _ in range(n)]


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


def run_cuts(runner, rid, tokens, cuts):
    """The logits of every position of one request fed in portions of the given sizes."""
    from spyinfer_b200.engine.batch import StepEntry

    rows, at = [], 0
    for c in cuts:
        rows.append(runner.step([StepEntry(rid, tokens[at:at + c], list(range(c)))]).float().cpu().numpy().copy())
        at += c
    assert at == len(tokens)
    runner.check_status()
    runner.finish(rid)
    return np.concatenate(rows)


def cycle_cuts(n, sizes):
    cuts, left = [], n
    while left:
        cuts.append(min(left, sizes[len(cuts) % len(sizes)]))
        left -= cuts[-1]
    return cuts


# ---- configuration, cache bookkeeping, weights, the plain mechanisms (no GPU) ------------------------------------

def test_config_is_found_by_its_architecture_key_and_declares_the_checkpoints_tensors():
    from spyinfer_b200.config import BubalixConfig, ConfigError, config_from_json
    from spyinfer_b200.engine.model import declared_weights

    for name, case in BX.items():
        cfg = config_from_json(case["config"])
        assert isinstance(cfg, BubalixConfig)
        decls = declared_weights(cfg.to_spec())
        assert {d.name: tuple(d.shape) for d in decls} == P.tensor_shapes(case["config"]), name
        assert len({d.name for d in decls}) == len(decls), name                     # the table that the layers share is declared once
        assert {d.name for d in decls if d.integer} == {n for n in P.tensor_shapes(case["config"]) if n.endswith(".table")}
        assert config_from_json(cfg.to_json()).to_json() == cfg.to_json()
    base = BX["a"]["config"]

    def broken(change):
        c = json.loads(json.dumps(base))
        change(c)
        with pytest.raises(ConfigError):
            config_from_json(c).to_spec()

    broken(lambda c: c["layers"][0].update(type="mamba1"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mixer"].pop("kv_rank"))
    broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10))                # wider than the rotated part
    broken(lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"))
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=3))                    # 4 heads do not group over 3
    broken(lambda c: c["layers"][1]["mixer"].pop("conv"))
    broken(lambda c: c["layers"][1]["mixer"].update(conv=17))
    broken(lambda c: c["layers"][1]["mixer"].update(softcap=-1.0))
    broken(lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0))
    broken(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))                 # more than there are experts
    broken(lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0))
    broken(lambda c: c["token_side"].update(dim=0))
    broken(lambda c: c["norm"].pop("eps"))
    broken(lambda c: c.pop("layers"))


def test_what_each_layer_keeps_between_steps():
    from spyinfer_b200.cache import CacheManager
    from spyinfer_b200.config import CompositeCacheNeed, PagedCacheNeed, StateCacheNeed, config_from_json
    from spyinfer_b200.engine.model import Model

    needs, cache_of = Model(config_from_json(BX["a"]["config"]).to_spec(), torch.float32, None, 256).cache_needs()
    assert cache_of == [None] * 4
    state = lambda n: StateCacheNeed((n,), "float32")
    assert needs[0] == PagedCacheNeed(1, 24 + 8, planes=1) and needs[3] == PagedCacheNeed(1, 20 + 12, planes=1)      # a latent and the shared key part
    assert needs[1] == CompositeCacheNeed((PagedCacheNeed(2, 24, 20), state(2 * (4 * 16 + 2 * 16 + 2 * 24))))
    assert needs[2] == CompositeCacheNeed((PagedCacheNeed(3, 24, 37), state(2 * (6 * 24 + 3 * 24 + 3 * 8))))
    cache = CacheManager(needs, 8, 40, 2, 320, device=None, cache_of=cache_of, max_step_tokens=16)
    assert cache.num_groups() == 3                              # the two latent layers have rows of equal width, so they share their pages' ids
    assert cache.view(0).group == cache.view(3).group
    needs, _ = Model(config_from_json(BX["b"]["config"]).to_spec(), torch.float32, None, 256).cache_needs()
    assert needs[0] == PagedCacheNeed(1, 24) and needs[2] == PagedCacheNeed(3, 24, 300)      # one tap leaves no state


def test_random_tables_of_experts_hold_different_entries_in_a_row():
    from spyinfer_b200.weights.loader import WeightDecl
    from spyinfer_b200.weights.random_init import random_tensor

    t = random_tensor(WeightDecl("t", (300, 3), init="choice:5", integer=True), 7, 0.02, 0.05, "cpu")
    assert t.dtype == torch.int32 and tuple(t.shape) == (300, 3) and int(t.min()) == 0 and int(t.max()) == 4
    assert all(len(set(row)) == 3 for row in t.tolist())
    assert torch.equal(t, random_tensor(WeightDecl("t", (300, 3), init="choice:5", integer=True), 7, 0.02, 0.05, "cpu"))
    with pytest.raises(ValueError):
        random_tensor(WeightDecl("t", (4, 6), init="choice:5", integer=True), 7, 0.02, 0.05, "cpu")


def test_a_random_model_folder_is_read_back_with_its_tables(tmp_path):
    from spyinfer_b200.config import config_from_json
    from spyinfer_b200.engine.model import declared_weights
    from spyinfer_b200.weights import write_model_folder
    from spyinfer_b200.weights.loader import load_checkpoint

    cfg = config_from_json(BX["a"]["config"])
    write_model_folder(str(tmp_path), cfg, 3)
    w = load_checkpoint(str(tmp_path), declared_weights(cfg.to_spec()), "cpu")
    assert w["l0.mlp.table"].dtype == torch.int32 and int(w["l0.mlp.table"].max()) < 6 and w["side.embed"].dtype == torch.bfloat16


def test_a_table_that_names_an_expert_there_is_not_is_refused():
    from spyinfer_b200.config import PartSpec
    from spyinfer_b200.parts import BuildContext, build_part

    part = build_part(PartSpec("expert_mixture", {"hidden_size": 8, "experts": 2, "top": 1, "ff": 8, "activation": "silu", "scoring": "table", "vocab_size": 3}),
                      BuildContext(torch.float32, torch.device("cpu"), 8))
    w = {d.name: torch.zeros(d.shape, dtype=torch.int32 if d.integer else torch.float32) for d in part.weight_decls()}
    part.bind(w)
    for bad in (2, -1):
        w["table"][1, 0] = bad
        with pytest.raises(ValueError, match="table"):
            part.bind(w)


def test_what_the_plain_mechanisms_do_on_inputs_known_by_hand():
    f64 = lambda *v: torch.tensor(v, dtype=P.F)
    # the norm's stored weight is the gain's distance from one
    assert torch.allclose(P.centred_norm(f64(3.0, -4.0), f64(0.0, 1.0), 0.0), f64(3.0, -8.0) / math.sqrt(12.5))
    # visibility: the window counts the query's own position
    assert [P.visible(10, j, 3) for j in range(12)] == [False] * 8 + [True] * 3 + [False]
    assert [P.visible(2, j, None) for j in range(4)] == [True, True, True, False]
    v = P.visibility(12, 3)
    assert all(bool(v[i, j]) == P.visible(i, j, 3) for i in range(12) for j in range(12))
    # slopes: the last head's is 2^-8 whatever the number of heads
    assert P.distance_slope(0, 8) == 0.5 and P.distance_slope(7, 8) == 2.0 ** -8 and P.distance_slope(0, 1) == 2.0 ** -8
    # the temperature grows by whole multiples: position every - 1 is the first whose queries are warmer
    t = P.query_temperature(torch.tensor([0, 14, 15, 31, 46, 47]), {"coef": 0.5, "every": 16})
    assert torch.allclose(t, f64(1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(4)))
    # the sink is one more in the denominator and takes no value
    s = f64(1.0, 2.0, 9.0).reshape(1, 3)
    w = P.softmax_with_sink(s, torch.tensor([[True, True, False]]), 0.5)
    z = math.exp(1.0) + math.exp(2.0) + math.exp(0.5)
    assert torch.allclose(w, f64(math.exp(1.0) / z, math.exp(2.0) / z, 0.0).reshape(1, 3))
    # the convolution's last column meets the current token
    h = torch.tensor([[1.0], [10.0], [100.0]], dtype=P.F)
    assert P.time_conv(h, torch.tensor([[3.0, 2.0]], dtype=P.F)).flatten().tolist() == [2.0, 23.0, 230.0]
    # halves: element i turns with element i + dims / 2
    x = f64(1.0, 2.0, 3.0, 4.0, 5.0).reshape(1, 1, 5)
    y = P.rotate_halves(x, torch.tensor([1]), {"dims": 4, "base": 100.0})[0, 0]
    c0, s0, c1, s1 = math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1)
    assert torch.allclose(y, f64(c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + s0, 4 * c1 + 2 * s1, 5.0))
    # the fastest pair keeps its frequency, the slowest is divided by the factor, cos and sin grow
    freqs, mag = P.stretched_frequencies({"dims": 16, "base": 10000.0, "scaling": {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}})
    plain, one = P.stretched_frequencies({"dims": 16, "base": 10000.0})
    assert one == 1.0 and math.isclose(mag, 0.1 * math.log(4.0) + 1.0) and freqs[0] == plain[0] and math.isclose(freqs[-1], plain[-1] / 4.0)
    # experts by table: the mean of the chosen ones' results, and the shared expert's on top
    g = torch.Generator().manual_seed(1)
    W = {f"{e}.{n}": torch.randn(2, 2, generator=g).double() for e in ("e0", "e1", "e2", "shared") for n in ("gate", "up", "down")}
    W["table"] = torch.tensor([[0, 2], [1, 2]], dtype=torch.int32)
    x = torch.randn(2, 2, generator=g).double()
    y = P.mixture(x, torch.tensor([1, 0]), W, "", {"router": {"experts": 3, "top": 2}, "shared": {"ff": 2}})
    by = {e: P.expert(x, W, e + ".") for e in ("e0", "e1", "e2", "shared")}
    assert torch.allclose(y[0], (by["e1"][0] + by["e2"][0]) / 2 + by["shared"][0]) and torch.allclose(y[1], (by["e0"][1] + by["e2"][1]) / 2 + by["shared"][1])


# ---- kernels alone ---------------------------------------------------------------------------------------

@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_two_results_join_the_stream_and_the_token_input_follows(dtype):
    """The sum of two sublayers' results (each possibly a stack of partial sums) and its copy; the pending normed input that the next
    norm of the stream adds in its launch, with a gain stored around zero; gathered rows for the head."""
    from spyinfer_b200 import kernels
    from spyinfer_b200.config import PartSpec
    from spyinfer_b200.parts import BuildContext, NormedDelta, build_part

    g = torch.Generator().manual_seed(4)
    for rows, n, sa, sb in ((5, 40, 1, 3), (3, 201, 2, 1), (9, 1000, 3, 0), (4, 4096, 7, 4), (301, 256, 1, 1), (1, 3, 2, 2)):
        h, a, b = torch.randn(rows, n, generator=g), torch.randn(sa, rows, n, generator=g), torch.randn(max(sb, 1), rows, n, generator=g)
        put = lambda t, s: t.cuda() if s > 1 else t[0].to(dtype).cuda()
        of = lambda t, s: t.double().sum(0) if s > 1 else t[0].to(dtype).double()
        want = h.double() + of(a, sa) + (of(b, sb) if sb else 0.0)
        hd, copy = h.cuda(), torch.empty((rows, n), dtype=torch.bfloat16, device="cuda")
        kernels.stream_sum(hd, put(a, sa), put(b, sb) if sb else None, copy)
        assert torch.allclose(hd.cpu().double(), want, atol=1e-5, rtol=1e-6), (rows, n)
        assert torch.equal(copy, hd.to(torch.bfloat16))
        # a pending input
        norm = build_part(PartSpec("group_rms_norm", {"size": n, "eps": 1e-5, "weight": "w", "weight_offset": 1.0}), BuildContext(dtype, torch.device("cuda"), 8))
        w, yw = (0.3 * torch.randn(n, generator=g)).to(torch.bfloat16), 1.0 + 0.2 * torch.randn(n, generator=g)
        norm.bind({"w": w.cuda()})
        y = torch.randn(max(sa, 1), rows, n, generator=g)
        delta = NormedDelta(put(y, sa), yw.cuda(), 1.0)
        new = hd.cpu().double() + P.unit_rms(of(y, sa), 1e-5) * yw.double()
        few = norm.forward_add(hd, delta, rows=torch.tensor([rows - 1, 0], dtype=torch.int32, device="cuda"), out_dtype=torch.float32)
        assert torch.allclose(few.cpu().double(), P.centred_norm(new, w.double(), 1e-5)[[rows - 1, 0]], atol=2e-5)
        out = norm.forward_add(hd, delta)
        assert torch.allclose(hd.cpu().double(), new, atol=2e-5)
        assert torch.allclose(out.cpu().double(), P.centred_norm(new, w.double(), 1e-5), **(dict(atol=2e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=1e-2)))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,slices,index,splits", [(24, 3, 1, 1), (7, 5, 4, 2), (256, 2, 0, 4), (130, 1, 0, 1)])
def test_a_tokens_own_vector_behind_its_gate(dtype, dim, slices, index, splits):
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(dim)
    T, V = 37, 50
    table = torch.randn(V, slices * dim, generator=g).to(torch.bfloat16)
    gate = 2.0 * torch.randn(splits, T, dim, generator=g)
    ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    z = gate.double().sum(0) if splits > 1 else gate[0].to(dtype).double()
    want = P.gelu_tanh(z) * table.double()[ids.long()][:, index * dim:(index + 1) * dim]
    out = torch.empty((T, dim), dtype=dtype, device="cuda")
    kernels.token_gate(gate.cuda() if splits > 1 else gate[0].to(dtype).cuda(), table.cuda(), index * dim, ids.cuda(), out)
    assert torch.allclose(out.cpu().double(), want, **(dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)))
    # an id outside the vocabulary is reported and reads nothing
    status = torch.zeros(2, dtype=torch.int32, device="cuda")
    ids[5] = V
    kernels.token_gate(gate.cuda() if splits > 1 else gate[0].to(dtype).cuda(), table.cuda(), index * dim, ids.cuda(), out, status=status)
    assert status.tolist() == [1, 5] and float(out[5].abs().max()) == 0.0


def _paged_setup(lens, page_size, nkv, hd, dtype, seed=0, planes=2):
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
    pages = torch.zeros((len(ids), planes, nkv, page_size, hd), dtype=dtype, device="cuda")
    return table.cuda(), pages


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps,page_size,splits,temp,gate", [
    (4, 2, 16, 24, 3, 8, 1, (0.4, 16), True), (3, 1, 12, 20, 1, 4, 3, None, True), (8, 4, 64, 64, 4, 16, 2, (0.5, 64), True), (20, 1, 7, 5, 5, 8, 1, (1.5, 3), False),
    (2, 1, 160, 192, 16, 16, 4, (0.2, 7), True), (2, 2, 10, 6, 2, 16, 1, None, False), (16, 2, 128, 128, 4, 16, 1, (0.1, 1), True), (6, 3, 32, 8, 9, 8, 2, (-0.3, 2.5), True), (8, 4, 16, 32, 6, 16, 1, (0.5, 16), True),
    (16, 4, 24, 40, 11, 16, 2, None, True), (4, 4, 64, 64, 16, 16, 1, (0.2, 64), True), (12, 4, 32, 32, 3, 8, 3, None, True)])
def test_queries_and_cache_rows_behind_the_convolution(dtype, heads, kv_heads, dim, vdim, taps, page_size, splits, temp, gate):
    """Three requests' runs in one step (a long one, one token, a run shorter than the taps), twice in a row, in slots that are not
    in the batch's order: queries, keys and values equal the plain convolution of the whole sequences, the state carries what the second
    step needs, rows are zero behind their content, nothing else is written."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(heads * 100 + dim + taps)
    hd = (max(dim, vdim) + 7) // 8 * 8
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    C, ld = nq + nk + nv, nq + nk + nv + heads
    lens, runs = [61, 15, 9], [(45, 16), (14, 1), (2, 7)]           # two steps' tokens of every request
    kernel = torch.randn(C, taps, generator=g) / taps ** 0.5
    seqs = [torch.randn(splits, n, ld, generator=g) for n in lens]
    u = [(s.double().sum(0) if splits > 1 else s[0].to(dtype).double()) for s in seqs]
    y = [P.time_conv(x[:, :C], kernel.double()) for x in u]
    slots = torch.tensor([2, 0, 3], dtype=torch.int32).cuda()
    state = torch.zeros((5, (taps - 1) * C), device="cuda") if taps > 1 else None
    other = torch.full_like(state[1], 5.0) if taps > 1 else None
    if taps > 1:
        state[1] = other
    table, pages = _paged_setup(lens, page_size, kv_heads, hd, dtype)
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=4e-2, rtol=1e-2)
    done = [0, 0, 0]
    for step in range(2):
        n_of = [r[step] for r in runs]
        part = torch.cat([s[:, d:d + n] for s, d, n in zip(seqs, done, n_of)], dim=1)
        pos = torch.tensor([d + i for d, n in zip(done, n_of) for i in range(n)], dtype=torch.int32)
        T = pos.shape[0]
        starts = torch.tensor([0] + list(np.cumsum(n_of)), dtype=torch.int32)
        q_out = torch.full((T, heads * hd), 7.0, dtype=dtype, device="cuda")
        gates = torch.empty((T, heads), dtype=torch.float32, device="cuda") if gate else None
        kernels.conv_qkv_store(part.cuda().contiguous() if splits > 1 else part[0].to(dtype).cuda().contiguous(), kernel.t().contiguous().cuda(), state, starts.cuda(),
                               slots, 3, max(n_of), pos.cuda(), q_out, table, pages, heads, kv_heads, dim, vdim, temp=temp, gate_col=C, gate_out=gates)
        rows = torch.cat([x[d:d + n] for x, d, n in zip(y, done, n_of)])
        q = rows[:, :nq].reshape(T, heads, dim)
        if temp is not None:
            q = q * P.query_temperature(pos, {"coef": temp[0], "every": temp[1]})[:, None, None]
        got = q_out.cpu().double().reshape(T, heads, hd)
        assert torch.allclose(got[..., :dim], q, **tol) and float(got[..., dim:].abs().sum()) == 0.0, step
        if gate:
            raw = torch.cat([x[d:d + n, C:] for x, d, n in zip(u, done, n_of)])
            assert torch.allclose(gates.cpu().double(), torch.sigmoid(raw), atol=1e-5)
        done = [d + n for d, n in zip(done, n_of)]
    table_h, pages_h = table.cpu(), pages.cpu().double()
    for s, n in enumerate(lens):
        k, v = y[s][:, nq:nq + nk].reshape(n, kv_heads, dim), y[s][:, nq + nk:].reshape(n, kv_heads, vdim)
        for t in range(n):
            page, slot = int(table_h[s, t // page_size]), t % page_size
            assert torch.allclose(pages_h[page, 0, :, slot, :dim], k[t], **tol) and torch.allclose(pages_h[page, 1, :, slot, :vdim], v[t], **tol), (s, t)
            assert float(pages_h[page, 0, :, slot, dim:].abs().sum()) == 0.0 and float(pages_h[page, 1, :, slot, vdim:].abs().sum()) == 0.0
    assert int((pages_h.abs().sum(dim=(1, 2, 4)) > 0).sum()) == sum(lens)
    if taps > 1:
        assert torch.equal(state[1], other)
        for s, slot in enumerate((2, 0, 3)):
            past = torch.cat([torch.zeros(taps - 1, C, dtype=P.F), u[s][:, :C]])[-(taps - 1):]
            assert torch.allclose(state[slot].cpu().double().reshape(taps - 1, C), past, atol=1e-5)


def _score(q, k, scale, cap, slopes, i, j):
    s = P.capped(torch.einsum("ihd,jhd->hij", q, k) * scale, cap)
    return s if slopes is None else s - slopes[:, None, None] * (i[:, None] - j[None, :]).to(P.F)[None]


@gpu
@pytest.mark.parametrize("path", ["plain32", "plain16", "tensor"])
@pytest.mark.parametrize("heads,kv_heads,hd,window,cap,bias,sinks,scaled,page_size,planes", [
    (4, 2, 24, 20, 12.0, True, True, True, 8, 2), (8, 4, 64, 64, 20.0, True, True, True, 16, 2), (16, 1, 128, 40, 30.0, True, False, True, 16, 2),
    (2, 1, 64, None, 50.0, True, True, False, 16, 2), (4, 4, 32, 7, 0.0, True, True, True, 8, 2), (6, 2, 128, 130, 15.0, False, True, False, 16, 2),
    (16, 1, 96, None, 0.0, False, True, False, 16, 1), (3, 1, 16, None, 0.0, False, False, True, 16, 1), (2, 2, 40, 1, 5.0, True, True, True, 16, 2),
    (5, 1, 64, None, 8.0, True, True, True, 32, 2)])
def test_capped_and_biased_scores_with_sinks_and_a_gate_a_head(path, heads, kv_heads, hd, window, cap, bias, sinks, scaled, page_size, planes):
    """A portion of a long prompt, a whole prompt and two decoded tokens over shuffled pages, on the plain kernel in both formats and on
    the tensor-core kernels for portions and for decoding (pairs whole and split over blocks); a few queries point at one key: the
    window's oldest key and the one before it, a page's first and last place, the first key, the query's own.  Every other sink is large
    enough to take most of a softmax, one is far beyond any score."""
    from spyinfer_b200 import kernels

    dtype = torch.float32 if path == "plain32" else torch.bfloat16
    if path == "tensor" and not kernels.attention_tc_takes(heads, kv_heads, hd, dtype):
        pytest.skip("sizes the tensor-core kernels do not take")
    g = torch.Generator().manual_seed(hd + heads)
    lens = [300, 40, 261, 1200]
    keys = [torch.randn(n, kv_heads, hd, generator=g).to(dtype).double() for n in lens]
    values = [torch.randn(n, kv_heads, hd, generator=g).to(dtype).double() for n in lens] if planes == 2 else keys
    table, pages = _paged_setup(lens, page_size, kv_heads, hd, dtype, seed=3, planes=planes)
    pages_h = pages.cpu()
    for s, n in enumerate(lens):
        for j in range(n):
            page = int(table[s, j // page_size])
            pages_h[page, 0, :, j % page_size] = keys[s][j].to(dtype)
            if planes == 2:
                pages_h[page, 1, :, j % page_size] = values[s][j].to(dtype)
    pages.copy_(pages_h)
    spans = [(2, 260, 261), (3, 1199, 1200), (0, 150, 300), (1, 0, 40)]           # the decoded tokens first, as the step function lays a mixed batch out
    pos = torch.tensor([p for _, a, b in spans for p in range(a, b)], dtype=torch.int32)
    seq = torch.tensor([i for i, (_, a, b) in enumerate(spans) for _ in range(a, b)], dtype=torch.int32)
    T = pos.shape[0]
    q = torch.randn(T, heads, hd, generator=g)
    first, last = 2, heads - 1                                    # the row of request 0's position 150; the head with the gentlest slope
    w = window or 100
    for p, target in ((170, 170 - w + 1), (171, 171 - w), (190, (190 // page_size) * page_size), (191, (190 // page_size) * page_size - 1), (210, 0), (299, 299)):
        if 0 <= target <= p:
            q[first + p - 150, last] = keys[0][target, last // (heads // kv_heads)].float() * (14.0 / hd ** 0.5)
    q = q.to(dtype)
    scale, rep = hd ** -0.5 * 1.5, heads // kv_heads
    slopes = torch.tensor([P.distance_slope(h, heads) for h in range(heads)], dtype=P.F) if bias else None
    sink = torch.tensor([(-1.0, 4.0, 1.0, 300.0)[h % 4] for h in range(heads)], dtype=P.F) if sinks else None
    factor = torch.rand(T, heads, generator=g) if scaled else None
    want, at = [], 0
    for s, a, b in spans:
        seen = P.visibility(b, window)[a:b]
        k, v = keys[s][:b].repeat_interleave(rep, dim=1), values[s][:b].repeat_interleave(rep, dim=1)
        sc = _score(q[at:at + b - a].double(), k, scale, cap, slopes, torch.arange(a, b), torch.arange(b))
        p = torch.stack([P.softmax_with_sink(sc[h], seen, sink[h] if sinks else None) for h in range(heads)])
        want.append(torch.einsum("hij,jhd->ihd", p, v))
        at += b - a
    want = torch.cat(want)
    if scaled:
        want = want * factor.double()[..., None]
    table_d = table[[s for s, _, _ in spans]].contiguous()
    dev = lambda t: t.float().cuda() if t is not None else None
    options = dict(softcap=cap, slopes=dev(slopes), sinks=dev(sink), out_scale=dev(factor))
    qd = q.reshape(T, heads * hd).cuda()

    def check(out, what):
        worst = (out.cpu().double().reshape(T, heads, hd) - want).abs().amax(dim=(1, 2))
        assert float(worst.max()) < (4e-5 if dtype == torch.float32 else 4e-2), f"{what}: token {int(worst.argmax())} (position {int(pos[int(worst.argmax())])}): {float(worst.max()):.3e}"

    if path != "tensor":
        out = torch.empty((T, heads * hd), dtype=dtype, device="cuda")
        kernels.attention_generic(qd, heads, hd, out, pages, table_d, pos.cuda(), seq.cuda(), scale, window=window, **options)
        return check(out, path)
    q_start = torch.tensor([0, 1, 2, 152, 192], dtype=torch.int32).cuda()
    for share in ("auto", "split", "whole"):
        out = torch.full((T, heads * hd), 9.0, dtype=dtype, device="cuda")
        kernels.attention_decode(qd, heads, hd, out, pages, table_d[:2], pos.cuda(), q_start[:3], 2, scale, window=window, share=share, **options)
        kernels.attention_tc(qd, heads, hd, out, pages, table_d[2:], pos.cuda(), q_start[2:], 2, scale, window=window, **options)
        check(out, f"tensor, {share}")
    out = torch.full((T, heads * hd), 9.0, dtype=dtype, device="cuda")
    kernels.attention_tc(qd, heads, hd, out, pages, table_d, pos.cuda(), q_start, 4, scale, window=window, **options)      # the kernel for portions takes single tokens as well
    check(out, "tensor, portions alone")


@gpu
def test_scores_with_options_leave_no_logarithms_and_shapes_are_checked():
    from spyinfer_b200 import kernels

    q, out = (torch.zeros((1, 32), dtype=torch.bfloat16, device="cuda") for _ in range(2))
    pages = torch.zeros((1, 2, 1, 16, 32), dtype=torch.bfloat16, device="cuda")
    table, pos, start = (torch.zeros(s, dtype=torch.int32, device="cuda") for s in ((1, 1), (1,), (2,)))
    one = torch.ones(1, device="cuda")
    for fn in (kernels.attention_tc, kernels.attention_decode):
        with pytest.raises(kernels.KernelError):
            fn(q, 1, 32, out, pages, table, pos, start, 1, 1.0, lse=torch.empty((1, 1), device="cuda"), sinks=one)
        with pytest.raises(kernels.KernelError):
            fn(q, 1, 32, out, pages, table, pos, start, 1, 1.0, slopes=torch.ones(2, device="cuda"))
        with pytest.raises(kernels.KernelError):
            fn(q, 1, 32, out, pages, table, pos, start, 1, 1.0, softcap=-1.0)
        with pytest.raises(kernels.KernelError):
            fn(q, 1, 32, out, pages, table, pos, start, 1, 1.0, out_scale=one)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rot_dim,kv_rank,vdim,yarn", [(4, 12, 8, 24, 20, (3.0, 64, 8.0, 0.5)), (16, 32, 32, 96, 48, (8.0, 512, 32.0, 1.0)), (3, 9, 2, 13, 11, None),
                                                                 (2, 40, 20, 150, 50, (2.0, 30, 6.0, 1.0)), (2, 16, 0, 20, 16, None)])
def test_the_absorbed_query_of_a_projection_left_in_32_bit(dtype, heads, dim, rot_dim, kv_rank, vdim, yarn):
    """Queries without a latent of their own: columns of the fused 32-bit projection go through the key projections head by head, their
    rotated part is turned in halves by stretched frequencies; the values' expansion takes the gate from the same projection."""
    from spyinfer_b200 import kernels
    from spyinfer_b200.config import PartSpec
    from spyinfer_b200.parts import BuildContext, build_part

    g = torch.Generator().manual_seed(heads + dim)
    T, qw, row = 41, heads * (dim + rot_dim), kv_rank + rot_dim
    fused = torch.randn(T, qw + row + heads * vdim, generator=g)
    uk = torch.randn(heads, dim, kv_rank, generator=g).to(torch.bfloat16)
    uv = torch.randn(heads, kv_rank, vdim, generator=g).to(torch.bfloat16)
    pos = torch.randint(0, 300, (T,), generator=g, dtype=torch.int32)
    rot, table = None, None
    if rot_dim:
        rot = {"base": 700.0, "dims": rot_dim}
        params = {"theta": 700.0, "rotary_dim": rot_dim}
        if yarn:
            rot["scaling"] = params["yarn_scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
        table = build_part(PartSpec("rotary_half", params), BuildContext(torch.float32, torch.device("cuda"), 300)).rotation_table()
    q = fused.double()[:, :qw].reshape(T, heads, dim + rot_dim)
    want = torch.cat([torch.einsum("thd,hdr->thr", q[..., :dim], uk.double()), P.rotate_halves(q[..., dim:], pos, rot)], dim=-1)
    out = torch.empty((T, heads * row), dtype=dtype, device="cuda")
    kernels.head_product(fused.cuda(), dim + rot_dim, uk.cuda(), out, row, tail=rot_dim, rope_table=table, positions=pos.cuda())
    tol = dict(atol=1e-4, rtol=1e-4) if dtype == torch.float32 else dict(atol=5e-2, rtol=1e-2)
    assert torch.allclose(out.cpu().double().reshape(T, heads, row), want, **tol)
    mixed = torch.randn(T, heads, row, generator=g).to(dtype)
    gated = torch.einsum("thr,hrv->thv", mixed.double()[..., :kv_rank], uv.double()) * torch.sigmoid(fused.double()[:, qw + row:]).reshape(T, heads, vdim)
    o = torch.empty((T, heads * vdim), dtype=dtype, device="cuda")
    kernels.head_product(mixed.reshape(T, -1).cuda(), row, uv.cuda(), o, vdim, gate=fused.cuda(), gate_offset=qw + row)
    assert torch.allclose(o.cpu().double().reshape(T, heads, vdim), gated, **tol)


@gpu
@pytest.mark.parametrize("gate_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 128, 300])
@pytest.mark.parametrize("heads,dim,rot_dim,kv_rank,vdim,pairing", [(4, 32, 32, 64, 40, "half"), (16, 128, 32, 96, 128, "half"), (3, 8, 8, 24, 12, "interleaved"),
                                                                    (2, 64, 0, 512, 100, "half"), (1, 200, 24, 136, 300, "half"), (5, 16, 16, 40, 7, "interleaved")])
def test_per_head_products_on_the_tensor_cores(heads, dim, rot_dim, kv_rank, vdim, pairing, T, gate_dtype):
    """The same two products by the kernel that the bfloat16 path uses where the sizes allow: one and several tiles of tokens, blocks
    of inputs (also more of them than are held at a time) and outputs, sizes that fill no tile, rows beyond the batch untouched."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(heads + dim + T)
    qw, row = heads * (dim + rot_dim), kv_rank + rot_dim
    bf = lambda *shape: torch.randn(*shape, generator=g).to(torch.bfloat16)
    q, uk, uv, gate = bf(T, qw + 16), bf(heads, kv_rank, dim), bf(heads, vdim, kv_rank), torch.randn(T, 5 + heads * vdim, generator=g).to(gate_dtype)
    assert kernels.head_gemm_takes(dim, qw + 16, dim + rot_dim) and kernels.head_gemm_takes(kv_rank, heads * row, row)
    pos = torch.randint(0, 200, (T,), generator=g, dtype=torch.int32)
    table, x = None, q.double()[:, :qw].reshape(T, heads, dim + rot_dim)
    tail = x[..., dim:]
    if rot_dim:
        rot = {"base": 700.0, "dims": rot_dim}
        ang = torch.arange(200, dtype=P.F)[:, None] * torch.tensor(P.stretched_frequencies(rot)[0], dtype=P.F)[None]
        table = torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).float().cuda()
        order = list(range(rot_dim)) if pairing == "half" else [e for e in range(0, rot_dim, 2)] + [e for e in range(1, rot_dim, 2)]
        tail = P.rotate_halves(tail[..., order], pos, rot)[..., [order.index(e) for e in range(rot_dim)]]
    want = torch.cat([torch.einsum("thd,hrd->thr", x[..., :dim], uk.double()), tail], dim=-1)
    out = torch.full((T + 1, heads * row), 3.0, dtype=torch.bfloat16, device="cuda")
    kernels.head_gemm(q.cuda(), dim + rot_dim, uk.cuda(), out[:T], row, tail=rot_dim, rope_table=table, interleaved=pairing == "interleaved", positions=pos.cuda())
    tol = lambda w: dict(atol=2e-2 * float(w.abs().max()) ** 0.5, rtol=1e-2)
    assert torch.allclose(out[:T].cpu().double().reshape(T, heads, row), want, **tol(want)) and bool((out[T] == 3.0).all())
    mixed = bf(T, heads, row)
    want = torch.einsum("thr,hvr->thv", mixed.double()[..., :kv_rank], uv.double()) * torch.sigmoid(gate.double()[:, 5:]).reshape(T, heads, vdim)
    o = torch.full((T + 1, heads * vdim), 3.0, dtype=torch.bfloat16, device="cuda")
    kernels.head_gemm(mixed.reshape(T, -1).cuda(), row, uv.cuda(), o[:T], vdim, gate=gate.cuda(), gate_offset=5)
    assert torch.allclose(o[:T].cpu().double().reshape(T, heads, vdim), want, **tol(want)) and bool((o[T] == 3.0).all())


@gpu
@pytest.mark.parametrize("cap", [4.0, 25.0])
def test_capped_scores_near_and_far_from_the_cap(cap):
    """Prompt portions whose scores all stay well below the cap, all lie near it, or change from one to the other along the sequence:
    the two ways in which the kernel for portions forms them agree with the plain scores."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(8)
    T, hd = 400, 64
    table, pages = _paged_setup([T], 16, 1, hd, torch.bfloat16)
    k, v, base = (torch.randn(T, 1, hd, generator=g).to(torch.bfloat16) for _ in range(3))
    pages_h = pages.cpu()
    for j in range(T):
        page = int(table[0, j // 16])
        pages_h[page, 0, :, j % 16], pages_h[page, 1, :, j % 16] = k[j], v[j]
    pages.copy_(pages_h)
    pos = torch.arange(T, dtype=torch.int32)
    for size in (torch.full((T, 1, 1), 0.1), torch.full((T, 1, 1), 5.0), torch.linspace(0.01, 4.0, T).reshape(T, 1, 1)):
        q = (base.float() * size * cap / hd ** 0.5).to(torch.bfloat16)
        s = _score(q.double(), k.double(), 1.0, cap, torch.tensor([0.01], dtype=P.F), pos, pos)[0]
        want = P.softmax_with_sink(s, P.visibility(T, None), None) @ v.double()[:, 0]
        out = torch.empty((T, hd), dtype=torch.bfloat16, device="cuda")
        kernels.attention_tc(q.reshape(T, hd).cuda(), 1, hd, out, pages, table, pos.cuda(), torch.tensor([0, T], dtype=torch.int32).cuda(), 1, 1.0, softcap=cap,
                             slopes=torch.tensor([0.01]).cuda())
        assert float((out.cpu().double() - want).abs().max()) < 3e-2


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,shared", [(6, 2, 24, 40), (4, 1, 16, 0), (5, 5, 12, 7), (64, 8, 8, 16), (3, 2, 10, 6)])
def test_experts_by_table_weights_activations_and_pairs(dtype, experts, top, ff, shared):
    """An expert that the table does not name for a token contributes exactly nothing, a named one its activation times 1 / top, the
    shared expert its own; the sorted pairs name every (token, expert) once, padded or not."""
    from spyinfer_b200 import kernels

    g = torch.Generator().manual_seed(experts)
    T, V, cols = 53, 30, experts * ff + shared
    table = torch.rand(V, experts, generator=g).argsort(1)[:, :top].to(torch.int32).contiguous()
    ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    gu = torch.randn(T, 2 * cols, generator=g).to(dtype)
    out = torch.full((T, cols), 3.0, dtype=dtype, device="cuda")
    kernels.moe_activation_table(gu.cuda(), table.cuda(), ids.cuda(), out, experts, ff, shared_ff=shared)
    got, x = out.cpu().double(), gu.double()
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
    for t in range(T):
        chosen = set(table[ids[t]].tolist())
        for e in range(experts):
            part = got[t, e * ff:(e + 1) * ff]
            if e in chosen:
                a = x[t, 2 * e * ff:2 * (e + 1) * ff]
                assert torch.allclose(part, P.silu(a[:ff]) * a[ff:] / top, **tol)
            else:
                assert float(part.abs().sum()) == 0.0
        if shared:
            a = x[t, 2 * experts * ff:]
            assert torch.allclose(got[t, experts * ff:], P.silu(a[:shared]) * a[shared:], **tol)
    for pad in (1, 16):
        offsets, slot, row_token, row_w, *_ = kernels.moe_route_table(table.cuda(), ids.cuda(), experts, pad=pad)
        offsets, slot, row_token, row_w = offsets.tolist(), slot.tolist(), row_token.tolist(), row_w.tolist()
        rows = {}
        for t in range(T):
            for k in range(top):
                e, r = int(table[ids[t], k]), slot[t][k]
                assert offsets[e] <= r < offsets[e + 1] and row_token[r] == t and abs(row_w[r] - 1.0 / top) < 1e-7
                rows[r] = (t, e)
        assert len(rows) == T * top and all(o % pad == 0 for o in offsets)


# ---- whole models through the step function -----------------------------------------------------------------

@gpu
@pytest.mark.parametrize("name", sorted(BX))
def test_the_stream_after_every_layer(models, name):
    from spyinfer_b200.engine.batch import StepEntry

    runner = make_runner(models[name][0], "float32", graphs=False)
    toks = tokens_of(name, 45)
    got = []

    def watch(block):
        inner = block.forward

        def forward(hidden, delta, batch, cache):
            hidden, delta = inner(hidden, delta, batch, cache)
            got.append(block.settle(hidden.clone(), delta).cpu().double())
            return hidden, delta
        block.forward = forward

    for layer in runner.model.layers:
        watch(layer.block)
    runner.step([StepEntry("r", toks, [44])])
    streams = []
    P.forward(models[name][1], models[name][2], toks, streams=streams)
    assert len(got) == len(streams) == len(models[name][1]["layers"])
    for i, (a, b) in enumerate(zip(got, streams)):
        assert float((a - b).abs().max() / b.abs().max()) < 1e-4, f"layer {i}"


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(BX))
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
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(BX))
def test_long_decoding_passes_windows_and_pages(models, name, dtype):
    """260 tokens, all but the first three one by one (through the decode graphs): every window passes over decoded tokens,
    every page border is crossed by a decoded token, and the windowed groups give their pages back."""
    runner = make_runner(models[name][0], dtype, page_size=8, num_pages=40)
    toks = tokens_of(name, 260, salt=1)
    got = run_cuts(runner, "long", toks, [3] + [1] * 257)
    agrees(got, plain_logits(name, models, toks), dtype, "decoded")
    assert runner.graph_steps > 200


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(BX))
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


def _pointing_model(tmp_path, kind, window):
    """A one-layer model without experts and token input whose weights are made so that the token ``A`` as a query points at the token
    ``B`` as a key with a score near its cap on one head: the key projection takes B's input (its latent) to the direction of A's query.
    The convolutions hardly mix neighbours, the rotated elements of that head take no part, and in the window layer it is the head with the gentlest
    slope, so the two may stand anywhere.  The other heads' queries are so small that they weigh all visible keys by their distance and the sink
    alone, so their results move when one key too many or too few is seen."""
    if kind == "attention":
        mixer, head = _attn(2, 1, 32, 12, 1.0, 3, cap=25.0, temp=(0.1, 100), window=window), 1
    else:
        mixer, head = _latent(2, 32, 8, 12, 24, 1.0, 1000.0, (4.0, 64, 8.0, 1.0)), 0
    cfg = _config(60, 64, 1e-5, 1.0, 0, [_layer(mixer, None)])
    w = P.as_float64(P.random_weights(cfg, 77))
    p, A, B = "l0.mix.", 58, 59
    h = P.centred_norm(w["embed"], w["l0.norm1"], 1e-5)
    w[p + "sink"].fill_(2.0)
    if kind == "attention":
        for n in "qkv":
            w[f"{p}{n}.conv"] *= 0.05
            w[f"{p}{n}.conv"][:, -1] = 1.0
        w[p + "q"][:32] *= 1e-3
        q, src, key = w[p + "q"][32:] @ h[A], h, p + "k"
        rows = slice(0, 32)
    else:
        w[p + "q"][40:] *= 1e-3
        w[p + "q"][32:40] = 0.0
        q, src, key = w[p + "q"][:32] @ h[A], P.unit_rms(h @ w[p + "dkv"][:24].T, 1e-5) * w[p + "dkv.norm"], p + "uk"
        rows = slice(0, 32)
    w[key] *= 0.05
    b = src[B] - src.mean(0)                                         # what sets B apart from the others
    w[key][rows] += 25.0 / float(q @ q) * torch.outer(q, b / (b @ src[B]))
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    d_ = tmp_path / f"point_{kind}_{window}"
    d_.mkdir()
    return write_model(d_, cfg, w), cfg, P.as_float64(w), A, B, head


def _pointing_case(tmp_path, kind, window):
    model_dir, cfg, w, A, B, head = _pointing_model(tmp_path, kind, window)
    rng = random.Random(5)
    n = 400
    toks = [rng.randrange(50) for _ in range(n)]
    if window:
        # queries: the key is the window's oldest place, one before it, at a page's last and first place, among the first tokens
        keys = [1, 200, 303, 304]
        asks = [200 + window - 1, 200 + window, 150, 390, 305, 304 + window, 10]
        sees = [[200], [], [], [], [303, 304], [], [1]]
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
    on = probs[0][head]                                              # [query, key]
    for a, seen in zip(asks, sees):
        unseen = [k for k in keys if k not in seen and k <= a]
        assert (not seen or float(on[a, seen].sum()) > 0.8) and float(on[a, unseen].sum() if unseen else 0.0) < 1e-9, (a, float(on[a, seen].sum()))
    return model_dir, toks, want, asks


POINTING = [("latent_attention", None), ("attention", None), ("attention", 40), ("attention", 24)]


def test_the_plain_model_points_where_the_test_wants_it_to(tmp_path):
    for case in POINTING:
        _pointing_case(tmp_path, *case)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,window", POINTING)
def test_a_query_that_points_at_one_key_finds_it_far_back_and_at_every_edge(tmp_path, dtype, kind, window):
    """The key token stands a few times in a sequence of 400 others; the query token is asked at places where the key is far
    back, at a page's first or last place, at the window's oldest place and one beyond it, and among the first tokens.  The
    engine's logits equal the plain model's, whole, in portions that cut windows and pages anywhere, and decoded one by one."""
    model_dir, toks, want, asks = _pointing_case(tmp_path, kind, window)
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
        check(run_cuts(runner, "e", toks, [200, window - 1, 1, 1, n - 200 - window - 1]), "portions at the edges")


@gpu
@pytest.mark.parametrize("what", ["sink", "slopes", "cap", "temperature", "gate", "conv", "side", "table", "shared", "scale", "yarn"])
def test_every_mechanism_shows_in_the_logits(models, what):
    """The plain model with one mechanism altered is farther from the engine than the tolerance: the agreement above is no accident of
    weights that hide it."""
    model_dir, cfg, w = models["a"]
    cfg, w = json.loads(json.dumps(cfg)), {k: v.clone() for k, v in w.items()}
    toks = tokens_of("a", 120)
    for i, L in enumerate(cfg["layers"]):
        p, m, latent = f"l{i}.", L["mixer"], L["type"] == "latent_attention"
        if what == "sink":
            w[p + "mix.sink"].fill_(-math.inf)
        elif what == "cap" and not latent:
            m["softcap"] *= 1e6
        elif what == "temperature" and not latent:
            m["q_temp"]["every"] += 1
        elif what == "gate":
            w[p + "mix.g"] *= 0.0
        elif what == "conv" and not latent:
            w[p + "mix.v.conv"][:, 0] = 0.0
        elif what == "side":
            w[p + "side.gate"] *= 0.9
        elif what == "table":
            w[p + "mlp.table"] = (w[p + "mlp.table"] + 1) % int(L["mlp"]["router"]["experts"])
        elif what == "shared":
            w[p + "mlp.shared.down"] *= 0.9
        elif what == "yarn" and latent:
            m["rot"].pop("scaling")
    if what == "scale":
        cfg["embedding"]["scale"] *= 1.05
    slope = P.distance_slope
    try:
        if what == "slopes":
            P.distance_slope = lambda h, H: slope(h, H) * 1.1
        want = P.forward(cfg, w, toks).numpy()
    finally:
        P.distance_slope = slope
    got = run_cuts(make_runner(model_dir, "float32"), "r", toks, [120])
    assert (np.abs(got - want).max(axis=-1) / np.abs(want).max()).max() > 10 * TOL["float32"], what


@gpu
def test_the_replay_program_runs_the_model(models, tmp_path):
    name = "a"
    rng = random.Random(2)
    reqs = {f"r{n}": tokens_of(name, n, salt=3) for n in (40, 3, 77, 25)}
    b = TraceBuilder()
    b.whole("whole", reqs["r77"])
    mixed_trace(b, reqs, {r: max(1, len(t) - 10) for r, t in reqs.items()}, rng, max_live=4, portion_sizes=(5, 2, 16))
    for dtype in ("float32", "bfloat16"):
        out = run_trace(models[name][0], dtype, b, str(tmp_path / dtype), peak_tokens(b), BX[name]["config"]["vocab"])
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
@pytest.mark.parametrize("name", ["a", "b", "c", "f"])
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

    def attention():
        heads, dim = rng.choice([1, 2, 4, 8, 16, 3, 6, 20, 32]), rng.choice([8, 16, 32, 64, 128, 24, 48, 192, 10])
        return _attn(heads, divisor(heads), dim, rng.choice([8, 16, 32, 64, 128, 40, dim, dim]), rng.choice([dim ** -0.5, 0.13, 0.2]), rng.choice([1, 2, 3, 4, 4, 6, 11]),
                     cap=rng.choice([None, 5.0, 15.0, 20.0, 30.0, 50.0]), temp=rng.choice([None, (0.5, 64), (0.1, 16), (1.0, 7)]),
                     window=rng.choice([None, 1, 5, 16, 17, 33, 64, 100, 200, 1000]))

    def latent():
        heads, dim, rot = rng.choice([1, 2, 4, 8, 16, 3, 20]), rng.choice([8, 16, 32, 64, 24, 10]), rng.choice([4, 8, 16, 32, 64, 6])
        yarn = (rng.choice([1.0, 2.0, 4.0, 16.0]), rng.choice([32, 128, 512]), rng.choice([32.0, 8.0, 2.0]), rng.choice([1.0, 0.5])) if rng.random() < 0.8 else None
        return _latent(heads, dim, rot, rng.choice([8, 16, 32, 64, 40]), rng.choice([16, 32, 64, 96, 200, 36]), rng.choice([(dim + rot) ** -0.5, 0.15]),
                       rng.choice([10000.0, 500000.0, 100.0]), yarn)

    def mlp():
        if rng.random() < 0.12:
            return None
        experts = rng.randrange(1, 17)
        return _moe(experts, rng.randrange(1, min(experts, 5) + 1), rng.choice([16, 32, 64, 24, 12]), rng.choice([None, 32, 48, 20]))

    layers = [_layer(rng.choice([attention, latent])(), mlp()) for _ in range(rng.randrange(2, 7))]
    return _config(rng.randrange(50, 600), rng.choice([64, 96, 128, 160, 200, 256, 320]), rng.choice([1e-5, 1e-6]), rng.choice([1.0, 2.0, 4.0, 0.5, 7.5]),
                   rng.choice([0, 8, 16, 24, 40, 10]), layers)


@gpu
@pytest.mark.parametrize("seed", [3, 11, 19, 27, 42, 58, 77, 91, 1009, 1011, 1020, 1036])
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
