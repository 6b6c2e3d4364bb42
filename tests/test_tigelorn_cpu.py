"""Tigelorn on a machine without a GPU: configuration, plan, loader, cache entries and the engine's host side (step
function, state slots, pages, scheduler) over the plain kernel statements of tests/kernel_refs.py, against the plain
implementation of tests/plain_tigelorn.py.  The CUDA kernels themselves are the business of test_tigelorn_gpu.py."""
import copy
import math

import pytest
import torch

import plain_tigelorn as P
import tiny
import tiny_tigelorn as TT
from kernel_refs import ReferenceKernels
from infurnace_b200.cache import CacheLayout, CacheManager
from infurnace_b200.config.specs import (
    EMBEDDING_CACHE, BigramEmbeddingSpec, DeltaRuleSpec, LatentAttentionSpec, ParallelMixerSpec, PreNormBlockSpec,
)
from infurnace_b200.engine import Engine, EngineOptions, SamplingParams
from infurnace_b200.errors import ModelConfigError, WeightError
from infurnace_b200.models import config_from_dict, plan_for

TOL = 2e-5      # float32 stream and buffers against the float64 oracle
F64 = torch.float64


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("tigelorn"))
    return {n: TT.make_model_dir(n, root) for n in ("T1", "T2")}


def engine(model_dir, page_size, pool=320, **kw):
    opts = dict(dtype="float32", device="cpu", page_size=page_size, num_pages=pool // page_size, max_num_seqs=4,
                max_num_batched_tokens=pool)
    opts.update(kw)
    return Engine.from_model_dir(model_dir, EngineOptions(**opts), kernels=ReferenceKernels(torch.float64))


def tolerance(ref):
    return TOL * max(1.0, float(ref.abs().max()))


# ------------------------------------------------------------------------------ each mechanism of the oracle alone
def test_the_oracles_mechanisms_alone():
    g = torch.Generator().manual_seed(0)
    # the pair table's rows: the first token's own row; then previous and current, each with its multiplier
    assert P.bigram_rows([3, 4, 3], 10, 7, 2) == [10, (21 + 8) % 10, (28 + 6) % 10]
    # a norm whose stored weight is zero leaves a unit root mean square
    x = torch.randn(4, 8, generator=g, dtype=F64)
    assert torch.allclose(P.layer_norm(x, torch.zeros(8, dtype=F64), 0.0).pow(2).mean(-1), torch.ones(4, dtype=F64))
    # rotation in both pairings: pair i turns by position * frequency_i
    v = torch.randn(5, 2, 6, generator=g, dtype=F64)
    rot = {"base": 10.0, "dims": 4}
    a = torch.tensor(3 * 10.0 ** (-2 / 4), dtype=F64)                 # pair 1 at position 3
    for neighbours, (i, j) in ((True, (2, 3)), (False, (1, 3))):
        t = P.rotate(v, rot, neighbours)
        assert torch.equal(t[0], v[0]) and torch.equal(t[..., 4:], v[..., 4:])
        assert torch.allclose(t[3, 0, i], v[3, 0, i] * torch.cos(a) - v[3, 0, j] * torch.sin(a))
        assert torch.allclose(t[3, 0, j], v[3, 0, j] * torch.cos(a) + v[3, 0, i] * torch.sin(a))
    # stretched frequencies: fast pairs keep theirs, slow ones are divided
    plain, one = P.rotary_frequencies({"base": 100.0, "dims": 8})
    freq, gain = P.rotary_frequencies({"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}})
    assert one == 1.0 and abs(gain - (0.1 * math.log(4.0) + 1)) < 1e-12
    assert torch.allclose(freq[0], plain[0]) and torch.allclose(freq[-1], plain[-1] / 4.0)
    # the window
    z = torch.zeros(4, 1, 2, dtype=F64)
    val = torch.arange(4, dtype=F64).view(4, 1, 1)
    assert torch.allclose(P.softmax_attention(z, z, val, 1.0, 2)[:, 0, 0], torch.tensor([0.0, 0.5, 1.5, 2.5], dtype=F64))
    # the convolution: the last column is the current token's
    u = P.short_convolution(torch.tensor([[1.0], [10.0], [100.0]], dtype=F64), torch.tensor([[3.0, 2.0]], dtype=F64))
    assert u[:, 0].tolist() == [2.0, 23.0, 230.0]
    # the delta rule: with beta 1, no decay and unit keys, what a key holds is replaced, and the read-out sees this write
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]], dtype=F64).view(3, 1, 2)
    val = torch.tensor([5.0, 7.0, 2.0], dtype=F64).view(3, 1, 1)
    ones = torch.ones(3, 1, 2, dtype=F64)
    o = P.delta_rule(ones, k, val, ones, torch.ones(3, 1, dtype=F64))
    assert o[:, 0, 0].tolist() == [5.0, 12.0, 9.0]
    # decays act on the rows before the value under the key is compared
    g2 = ones.clone()
    g2[2, 0, 0] = 0.5
    o = P.delta_rule(k, k, val, g2, torch.full((3, 1), 0.5, dtype=F64))
    assert abs(float(o[2, 0, 0]) - (1.25 + 0.5 * (2.0 - 1.25))) < 1e-12           # S = 2.5 -> 1.25, halfway towards 2


# ------------------------------------------------------------------------------ configuration, plan, weights
def test_configuration_round_trip_and_plan():
    for name, spec in TT.TINY.items():
        conf = spec["config"]
        cfg = config_from_dict(conf)
        assert cfg.to_dict() == conf, name
        plan = plan_for(cfg)
        made = TT.make_weights(conf, 0)
        assert set(n for n, t in plan.tensors().items() if not t.optional) == set(made), name
        for tname, t in made.items():
            assert tuple(plan.tensors()[tname].shape) == tuple(t.shape), tname
        b = conf["embedding"]["bigram"]
        assert isinstance(plan.embedding, BigramEmbeddingSpec)
        assert (plan.embedding.buckets, plan.embedding.mul_prev, plan.embedding.mul_cur) == (b["buckets"], b["mul_prev"], b["mul_cur"])
        assert plan.lm_head.tied and plan.lm_head.weight == plan.embedding.weight and plan.final_norm.offset == 1.0
        roots = [TT.root(conf["layers"], i) for i in range(len(conf["layers"]))]
        assert len(plan.layers) == len(set(roots)) and len(plan.schedule) == len(roots)
        assert len({c.cache for c in plan.schedule}) == len(roots)                 # cache entries of their own
        for call, entry, r in zip(plan.schedule, conf["layers"], roots):
            layer = plan.layers[call.layer]
            assert isinstance(layer, PreNormBlockSpec) and layer.mixer_norm.weight == f"l{r}.norm1" and layer.mixer_norm.offset == 1.0
            m, mixer = entry["mixer"], layer.mixer
            assert (layer.ffn is None) == (entry["mlp"] is None) == (layer.ffn_norm is None)
            if layer.ffn is not None:
                assert (layer.ffn.intermediate_size, layer.ffn.activation) == (entry["mlp"]["ff"], "gelu_tanh")
            if entry["type"] == "channel_delta":
                assert isinstance(mixer, DeltaRuleSpec) and mixer.unit_eps == 1e-6 and mixer.eps == conf["norm"]["eps"]
                assert (mixer.num_heads, mixer.num_kv_heads, mixer.head_dim, mixer.value_head_dim, mixer.taps) == \
                    (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            elif entry["type"] == "latent_attention":
                assert isinstance(mixer, LatentAttentionSpec) and mixer.sink is None and mixer.gate is None and mixer.window is None
                assert (mixer.num_heads, mixer.head_dim, mixer.rot_dim, mixer.value_head_dim, mixer.kv_rank, mixer.q_rank, mixer.scale) == \
                    (m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["scale"])
                sc = m["rot"].get("scaling")
                assert mixer.position.interleaved
                assert mixer.position.scaling == ((sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None)
            else:
                assert isinstance(mixer, ParallelMixerSpec) and mixer.scales == (m["left_scale"], m["right_scale"])
                att, lin = mixer.mixers
                assert (att.num_heads, att.num_kv_heads, att.head_dim, att.value_head_dim, att.scale, att.window) == \
                    tuple(m["left"][k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")) + (m["left"]["mask"]["size"],)
                assert att.unit_qk and att.gate and att.q_bias and not att.position.interleaved
                assert lin.decay == tuple(m["right"]["decay"]) and lin.key_scale == 1.0 and lin.input_activation == "silu"
                assert lin.joint_norm and lin.gate_activation == "sigmoid"


def test_cache_entries_pages_and_states():
    conf = TT.TINY["T1"]["config"]
    plan = plan_for(config_from_dict(conf))
    layout = CacheLayout(plan)
    kinds = sorted((type(need).__name__, need.window, len(ids)) for need, ids in layout.kv.values())
    assert kinds == [("KVCacheNeed", 7, 2), ("PagedCacheNeed", None, 1)]           # the parallel layer runs twice
    states = {need.shape: len(ids) for need, ids in layout.state.values()}
    # the previous token; the delta rule's states and inputs, of the layer that runs three times and of the other; linear attention
    assert states == {(1,): 1, (4, 8, 10): 3, (2, 72): 3, (2, 12, 6): 1, (4, 60): 1, (3, 6, 10): 2}
    cache = CacheManager(plan, page_size=8, num_pages=6, max_requests=2, dtype=torch.float32, device="cpu")
    assert cache.state_groups[cache.state_group_of(EMBEDDING_CACHE)].need.shape == (1,)
    cache.add_request("a")
    slot = cache.slot_of("a")
    for g in cache.state_groups:
        for t in g.tensors.values():
            t[slot].fill_(2.0)
    cache.free_request("a")
    cache.add_request("b")
    assert cache.slot_of("b") == slot
    assert all(float(t[slot].abs().max()) == 0.0 for g in cache.state_groups for t in g.tensors.values())


def test_configuration_faults_are_named():
    base = TT.TINY["T1"]["config"]

    def broken(edit):
        c = copy.deepcopy(base)
        edit(c)
        with pytest.raises(ModelConfigError) as e:
            config_from_dict(c)
        return str(e.value)

    assert "type" in broken(lambda c: c["layers"][0].update(type="lstm"))
    assert "kv_heads" in broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=3))
    assert "conv" in broken(lambda c: c["layers"][1]["mixer"].pop("conv"))
    assert "q_rank" in broken(lambda c: c["layers"][2]["mixer"].pop("q_rank"))
    assert "rot.dims" in broken(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=8))
    assert "scaling.factor" in broken(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("factor"))
    assert "left.heads" in broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    assert "mask.size" in broken(lambda c: c["layers"][0]["mixer"]["left"].update(mask={}))
    assert "right.decay" in broken(lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]))
    assert "right_scale" in broken(lambda c: c["layers"][0]["mixer"].pop("right_scale"))
    assert "dense" in broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    assert "weights_of" in broken(lambda c: c["layers"][4].update(weights_of=9))
    assert "weights_of" in broken(lambda c: c["layers"][1].update(weights_of=4))           # a circle
    assert "weights_of" in broken(lambda c: c["layers"][4].update(weights_of=3))           # another layer's sizes
    assert "buckets" in broken(lambda c: c["embedding"]["bigram"].update(buckets=0))
    assert "eps" in broken(lambda c: c.update(norm={}))
    assert "layers" in broken(lambda c: c.update(layers=[]))


def test_loader_lists_what_is_wrong(models, tmp_path):
    import os
    import shutil
    from safetensors.torch import load_file, save_file
    d = str(tmp_path / "bad")
    shutil.copytree(models["T1"], d)
    t = load_file(os.path.join(d, "model.safetensors"))
    del t["l1.mix.A_log"]
    t["l4.mix.q"] = torch.zeros(16, 48)             # layer 4 has no tensors of its own
    t["l1.norm2"] = torch.ones(48)                  # layer 1 has no feed-forward
    t["l0.mix.left.q.b"] = torch.ones(31)
    t["bigram"] = torch.ones(37, 48)                # the first token's row is missing
    t["head"] = torch.ones(101, 48)                 # the head is the embedding table
    save_file(t, os.path.join(d, "model.safetensors"))
    with pytest.raises(WeightError) as e:
        engine(d, 16)
    msg = str(e.value)
    assert all(name in msg for name in ("l1.mix.A_log", "l4.mix.q", "l1.norm2", "l0.mix.left.q.b", "bigram", "head"))


def test_bottleneck_widths_come_from_the_tensors(models, tmp_path):
    """Without ``rank`` the stored matrices give the widths, which may differ; matrices that do not fit together are named."""
    import json
    import os
    from safetensors.torch import load_file, save_file
    conf = {**TT.TINY["T1"]["config"], "layers": [TT._delta(2, 1, 4, 6, 2, 3)]}
    d = TT.make_model_dir("_ranks", str(tmp_path), config=conf, seed=1, store="float32")
    del conf["layers"][0]["mixer"]["rank"]
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(conf, f)
    path = os.path.join(d, "model.safetensors")
    t = load_file(path)
    t["l0.mix.g1"], t["l0.mix.g2"] = torch.randn(7, 48), torch.randn(12, 7)
    save_file(t, path)
    cfg, w = TT.load_model_dir(d)
    toks = tiny.random_tokens(101, 20, 1)
    ref = P.forward(cfg, w, toks)
    out = tiny.collect(s := tiny.schedule_whole({"a": toks}), tiny.run_inprocess(engine(d, 16).runner, s), 101)["a"]
    assert (out - ref).abs().max() < tolerance(ref)
    t["l0.mix.g2"] = torch.randn(12, 6)
    save_file(t, path)
    with pytest.raises(WeightError) as e:
        engine(d, 16)
    assert "l0.mix.g2" in str(e.value)


# ------------------------------------------------------------------------------ the engine's host side
LENS = [37, 75, 64, 19, 50, 1, 2, 3]


def _requests(vocab, seed=0):
    return {f"r{i}": tiny.random_tokens(vocab, n, seed + i) for i, n in enumerate(LENS)}


@pytest.mark.parametrize("name", ["T1", "T2"])
@pytest.mark.parametrize("mode", ["whole", "bulk_tail", "portions", "mixed"])
def test_cutting_modes_on_the_host_path(models, name, mode):
    cfg, w = TT.load_model_dir(models[name])
    reqs = _requests(cfg["vocab"])
    steps = {"whole": tiny.schedule_whole, "bulk_tail": lambda r: tiny.schedule_bulk_tail(r, tail=30),
             "portions": lambda r: tiny.schedule_portions(r, seed=3),
             "mixed": lambda r: tiny.schedule_mixed(r, max_tokens=320, seed=4)}[mode](reqs)
    eng = engine(models[name], TT.TINY[name]["page_size"])
    out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), cfg["vocab"])
    for rid, toks in reqs.items():
        ref = P.forward(cfg, w, toks)
        assert (out[rid] - ref).abs().max() < tolerance(ref), (rid, mode)
    eng.runner.cache.check()
    assert eng.runner.cache.num_free_slots == 4
    assert eng.runner.cache.free_pages() == [g.pool.num_pages for g in eng.runner.cache.kv_groups]


@pytest.mark.parametrize("fold", [True, False])
def test_the_stream_after_every_layer(models, fold):
    """The residual stream after each layer run, not only the logits, is the plain implementation's; with norms folded into
    the products around them and without."""
    cfg, w = TT.load_model_dir(models["T1"])
    toks = tiny.random_tokens(cfg["vocab"], 30, 5)
    _, layers = P.forward(cfg, w, toks, return_layers=True)
    eng = Engine.from_model_dir(models["T1"], EngineOptions(dtype="float32", device="cpu", page_size=16, num_pages=20, max_num_seqs=4,
                                                            max_num_batched_tokens=320), kernels=ReferenceKernels(torch.float64, fold=fold))
    seen = []
    for layer in eng.runner.model.layers:
        inner = layer.forward

        def spy(x, pending, ctx, call, next_layer=None, inner=inner):
            out = inner(x, pending, ctx, call, next_layer=next_layer)
            seen.append(x.clone() if not isinstance(out, torch.Tensor) else x + out)      # the last delta is added by what follows
            return out
        layer.forward = spy
    tiny.run_inprocess(eng.runner, tiny.schedule_whole({"a": toks}))
    assert len(seen) == len(cfg["layers"])
    for i, got in enumerate(seen):
        assert (got.double() - layers[i]).abs().max() < tolerance(layers[i]), i


def test_the_oracle_would_show_a_lost_mechanism(models):
    """The tiny models are made so that these faults move the logits by far more than the tolerance."""
    cfg, w = TT.load_model_dir(models["T1"])
    toks = tiny.random_tokens(cfg["vocab"], 40, 9)
    ref = P.forward(cfg, w, toks)

    def moved(cfg2=None, **tensors):
        w2 = dict(w)
        w2.update(tensors)
        return float((P.forward(cfg2 or cfg, w2, toks) - ref).abs().max()) > 1000 * tolerance(ref)

    def edited(edit):
        other = copy.deepcopy(cfg)
        edit(other)
        return other

    def left(c):
        return c["layers"][0]["mixer"]["left"], c["layers"][5]["mixer"]["left"]

    assert moved(edited(lambda c: [m["mask"].update(size=8) for m in left(c)]))              # a window one token off
    assert moved(edited(lambda c: [m["mask"].update(size=6) for m in left(c)]))
    assert moved(edited(lambda c: [m["rot"].update(base=90.0) for m in left(c)]))
    assert moved(edited(lambda c: [m["rot"].update(dims=8) for m in left(c)]))
    assert moved(edited(lambda c: [m.update(scale=1.0) for m in left(c)]))
    assert moved(edited(lambda c: [c["layers"][i]["mixer"].update(left_scale=1.0) for i in (0, 5)]))
    assert moved(edited(lambda c: [c["layers"][i]["mixer"].update(right_scale=1.0) for i in (0, 5)]))
    assert moved(edited(lambda c: [c["layers"][i]["mixer"]["right"].update(decay=[0.6, 0.95, 0.98]) for i in (0, 5)]))
    assert moved(edited(lambda c: c["layers"][2]["mixer"]["rot"].pop("scaling")))
    assert moved(edited(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=2.0)))
    assert moved(edited(lambda c: c["layers"][2]["mixer"].update(scale=0.6)))
    assert moved(edited(lambda c: c["norm"].update(eps=1e-2)))
    assert moved(edited(lambda c: c["embedding"]["bigram"].update(mul_prev=12)))
    assert moved(edited(lambda c: c["embedding"]["bigram"].update(mul_cur=4)))
    for name in ("q.b", "k.b", "v.b", "g"):
        assert moved(**{"l0.mix.left." + name: torch.zeros_like(w["l0.mix.left." + name])}), name
    assert moved(**{"l0.mix.right.g": torch.zeros_like(w["l0.mix.right.g"])})
    assert moved(**{"l0.mix.right.norm": torch.ones_like(w["l0.mix.right.norm"])})
    for name in ("q", "k", "v"):
        assert moved(**{f"l1.mix.{name}.conv": torch.roll(w[f"l1.mix.{name}.conv"], 1, dims=1)}), name    # the taps in another order
    for name in ("b", "a1", "g1"):
        assert moved(**{"l1.mix." + name: torch.zeros_like(w["l1.mix." + name])}), name
    assert moved(**{"l1.mix.A_log": w["l1.mix.A_log"] + 0.5})
    assert moved(**{"l1.mix.dt_bias": torch.roll(w["l1.mix.dt_bias"], 1)})                     # decays of other channels
    assert moved(**{"l1.mix.norm": torch.ones_like(w["l1.mix.norm"])})
    assert moved(**{"l2.mix.dq.norm": torch.ones_like(w["l2.mix.dq.norm"])})
    for name in ("l0.norm1", "l0.norm2", "final.norm"):
        assert moved(**{name: torch.zeros_like(w[name])}), name
    first = w["bigram"].clone()
    first[-1] = 0.0
    assert moved(bigram=first)                                                                # the first token's row

    def planted(**swap):
        kept = {k: getattr(P, k) for k in swap}
        try:
            for k, f in swap.items():
                setattr(P, k, f)
            return float((P.forward(cfg, w, toks) - ref).abs().max()) > 1000 * tolerance(ref)
        finally:
            for k, f in kept.items():
                setattr(P, k, f)

    def read_before_write(q, k, v, g, beta):
        o = P_delta(q, k, v, g, beta)
        return torch.cat((torch.zeros_like(o[:1]), o[:-1]))
    P_delta, P_rotate = P.delta_rule, P.rotate
    assert planted(delta_rule=read_before_write)
    assert planted(delta_rule=lambda q, k, v, g, beta: P_delta(q, k, v, torch.ones_like(g), beta))
    assert planted(rotate=lambda v, rot, neighbours: P_rotate(v, rot, not neighbours))
    assert planted(gelu_tanh=P.silu)
    assert planted(unit_vector=lambda x: x)


def test_prefill_equals_token_by_token_decoding(models):
    for name in ("T1", "T2"):
        cfg, w = TT.load_model_dir(models[name])
        toks = tiny.random_tokens(cfg["vocab"], 50, 21)
        ref = P.forward(cfg, w, toks)
        steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
        eng = engine(models[name], TT.TINY[name]["page_size"])
        out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), cfg["vocab"])["x"]
        assert (out - ref).abs().max() < tolerance(ref), name


@pytest.mark.parametrize("pattern", [[2] * 25, [3, 2, 5, 2, 2, 7, 1, 1, 2, 25], [1, 49], [48, 2]])
def test_portions_down_to_two_tokens(models, pattern):
    """Portions shorter than the convolutions' reach and than the window; the window's and pages' edges fall inside them."""
    cfg, w = TT.load_model_dir(models["T1"])
    toks = tiny.random_tokens(cfg["vocab"], sum(pattern), 31)
    ref = P.forward(cfg, w, toks)
    steps, at = [], 0
    for i, n in enumerate(pattern):
        steps.append({"step": i, "entries": [{"id": "x", "tokens": toks[at:at + n], "want": list(range(n))}], "end": []})
        at += n
    out = tiny.collect(steps, tiny.run_inprocess(engine(models["T1"], 16).runner, steps), cfg["vocab"])["x"]
    assert (out - ref).abs().max() < tolerance(ref)


def test_pages_and_slots_are_used_again(models):
    """A request longer than its window holds few of that group's pages; another then takes them, and its slot: the new
    request's first token has no predecessor, its convolutions see zeros, its states start at zero."""
    cfg, w = TT.load_model_dir(models["T1"])
    long_toks, short, third = (tiny.random_tokens(cfg["vocab"], n, n) for n in (100, 30, 31))
    eng = engine(models["T1"], 16, pool=144, max_num_seqs=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": long_toks[:70], "want": list(range(70))}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": long_toks[70:], "want": list(range(30))},
                                     {"id": "b", "tokens": short, "want": list(range(30))}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": third, "want": list(range(31))}], "end": ["b", "c"]}]
    outs = tiny.run_inprocess(eng.runner, steps[:1])
    held = {g.need.window: g.pool.num_pages - g.pool.num_free for g in eng.runner.cache.kv_groups}
    assert held[7] <= 2 and held[None] == 5
    outs.update(tiny.run_inprocess(eng.runner, steps[1:]))
    out = tiny.collect(steps, outs, cfg["vocab"])
    for rid, toks in (("a", long_toks), ("b", short), ("c", third)):
        ref = P.forward(cfg, w, toks)
        assert (out[rid] - ref).abs().max() < tolerance(ref), rid


VARIANTS = {
    # one layer of each kind alone; one head, two taps, a window of two; no pair table
    "delta_only": {k: v for k, v in TT._config(30, 16, 1e-5, [TT._delta(1, 1, 4, 4, 2, 1, TT._dense(8))], (5, 1, 1)).items() if k != "embedding"},
    "latent_only": TT._config(41, 24, 1e-6, [TT._lat(1, 4, 2, 4, 4, 3, 0.5, 50.0, None)], (100, 1, 100)),
    "parallel_only": TT._config(33, 16, 1e-5, [TT._par((1, 1, 6, 4, 0.8, 2, 2.0, 6), (2, 3, (0.5,)), (2.0, 0.5), TT._dense(4))], (9, 10, 20)),
    # no feed-forward anywhere, seven taps (longer than most portions), every layer the first one's weights
    "shared": TT._config(50, 24, 1e-6, [_l := TT._delta(6, 3, 4, 2, 7, 2), TT._again([_l], 0), TT._again([_l], 0)], (64, 3, 7)),
}


@pytest.mark.parametrize("name", list(VARIANTS))
def test_other_arrangements_of_the_layers(tmp_path, name):
    """Values that make mechanisms coincide or vanish, other sizes and orders, in a mixed schedule over a small pool, and
    greedy generation through the scheduler."""
    conf = VARIANTS[name]
    d = TT.make_model_dir("_" + name, str(tmp_path), config=conf, seed=3, store="float32")
    cfg, w = TT.load_model_dir(d)
    V = conf["vocab"]
    reqs = {f"r{i}": tiny.random_tokens(V, n, i) for i, n in enumerate([20, 1, 33, 7, 2, 15])}
    steps = tiny.schedule_mixed(reqs, max_tokens=192, seed=1)
    eng = Engine.from_model_dir(d, EngineOptions(dtype="float32", device="cpu", page_size=4, num_pages=48, max_num_seqs=4,
                                                 max_num_batched_tokens=192), kernels=ReferenceKernels(torch.float64))
    out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), V)
    for rid, toks in reqs.items():
        ref = P.forward(cfg, w, toks)
        assert (out[rid] - ref).abs().max() < tolerance(ref), rid
    prompt = tiny.random_tokens(V, 5, 9)
    assert eng.generate([prompt], SamplingParams(max_tokens=6)) == [P.greedy(cfg, w, prompt, 6)]


def test_mixers_side_by_side_with_and_without_shared_products():
    """Two recurrences of one kind beside each other: with their products shared, and each with its own (whose results go
    through one buffer), the sum is the same."""
    from infurnace_b200.config.specs import LayerCall, RetentionSpec
    from infurnace_b200.parts import Runtime, build_part
    g = torch.Generator().manual_seed(5)
    specs, weights = [], {}
    for name, dim in (("a.", 3), ("b.", 5)):
        s = RetentionSpec(16, 2, dim, 4, (0.5, 0.9), 1.0, 1e-5, *(name + x for x in "qkvgo"))
        specs.append(s)
        weights.update({n: torch.randn(t.shape, generator=g) for n, t in s.tensors().items()})
    k = ReferenceKernels(torch.float64)

    class Ctx:
        cu_q, seq_lens, state_slots = torch.tensor([0, 6], dtype=torch.int32), torch.tensor([6], dtype=torch.int32), torch.tensor([0], dtype=torch.int32)
        max_q_len, held = 6, {}

        def __init__(self):
            self.states = {(0, i): torch.zeros(1, 2, d, 4) for i, d in enumerate((3, 5))}

        def buffer(self, name, shape, dtype, rows=None):
            return self.held.setdefault((name, tuple(shape), dtype), torch.zeros(shape, dtype=dtype))

        def state(self, cid):
            return self.states[cid]
    rt = Runtime(device=torch.device("cpu"), act_dtype=torch.float32, kernels=k)
    h = torch.randn(6, 16, generator=g)
    mixer = build_part(ParallelMixerSpec(tuple(specs), (0.7, -1.5)), weights, rt)
    assert mixer.joint and not mixer.can_return_weighted
    got = mixer.forward(h, Ctx(), LayerCall(0, 0)).clone()
    alone = [build_part(s, weights, rt).forward(h, Ctx(), LayerCall(0, (0, i))).clone() for i, s in enumerate(specs)]
    assert torch.allclose(got, 0.7 * alone[0] - 1.5 * alone[1], atol=1e-5)
    separate = build_part(ParallelMixerSpec(tuple(specs), (0.7, -1.5)), weights, rt)
    separate.mixers, separate.joint = [build_part(s, weights, rt) for s in specs], False
    assert torch.allclose(separate.forward(h, Ctx(), LayerCall(0, 0)), got, atol=1e-5)


def test_greedy_generation_through_the_scheduler(models):
    cfg, w = TT.load_model_dir(models["T1"])
    eng = engine(models["T1"], 16, max_num_batched_tokens=24)          # prompts go in as portions beside decoded tokens
    prompts = [tiny.random_tokens(cfg["vocab"], n, 40 + n) for n in (1, 9, 33, 50, 5, 18)]      # six requests, four slots
    outs = eng.generate(prompts, SamplingParams(max_tokens=8))
    for p, o in zip(prompts, outs):
        assert o == P.greedy(cfg, w, p, 8)
    eng.runner.cache.check()
    assert eng.runner.cache.num_free_slots == 4
