"""Lovurax through the engine on the CPU (PyTorch math of the ops): the cache, state slots, batching, scheduling and generation
against the plain statement of the design in lovurax_oracle.py."""
import copy
import json
import math

import pytest
import torch

import lovurax_oracle as O
from trainscale_b200.hub import ModelSerializer, load_pretrained
from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, GenerationParams, SchedulerConfig, SOTAInferenceEngine
from trainscale_b200.inference.batch import StepEntry
from trainscale_b200.inference.trace import TraceRunner
from trainscale_b200.models import architecture_of
from trainscale_b200.models.lovurax import LovuraxConfig, LovuraxForCausalLM, build_model, load_model

# unlike layers: every size and constant differs from layer to layer
MIXED = dict(width=40, types=("attention", "retention", "latent_attention", "retention", "attention"), heads=[6, 4, 3, 2, 4], kv_heads=[2, 4, 1, 2, 1],
             dim=[12, 8, 10, 14, 7], vdim=[6, 16, 10, 9, 5], temp=[0.5, 0.2, 0.3], every=[5, 1, 11, 3, 7], rheads=[3, 5, 1, 2], rdim=[12, 10, 8, 16],
             rvdim=[20, 6, 8, 11], rot=[8, 4, 2, 16], base=[500.0, 50.0, 3000.0], decay=[(0.9, 0.99, 0.6), (0.8, 0.97), (0.5,)], lheads=[3, 1, 5, 4],
             ldim=[12, 8, 14, 6], lvdim=[10, 8, 7], rank=[20, 8, 18], mlps=(1, 1, 0, 1), ff=[56, 17, 64], logit_scale=0.6)


def make(seed=0, sharp=1.5, blocks=64, block_size=4, seqs=4, budget=512, prefix=False, **over):
    cfg = O.make_config(**{**MIXED, **over})
    w = O.make_weights(cfg, seed, sharp)
    core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", dtype="float32",
                                   scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                                   cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=256,
                                                     enable_prefix_caching=prefix)),
                      model=load_model(cfg, w, torch.float32))
    return cfg, w, core


def oracle(w, cfg, ids):
    return O.logits({k: v.double() for k, v in w.items()}, cfg, ids)


def tokens(n, seed, vocab=300):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, tol=2e-4):
    assert (got - want).abs().max() <= tol * want.abs().max(), (got - want).abs().max() / want.abs().max()


def run_portions(core, seq, ids, sizes):
    out, at = [], 0
    sizes = list(sizes)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        out.append(core.execute([StepEntry(seq, ids[at:at + n], list(range(n)))]))
        at += n
    return torch.cat(out)


# ---------------------------------------------------------------------------------------------- single mechanisms
def test_xielu_and_leading_columns():
    from trainscale_b200.ops import grouped
    p, q = torch.tensor([0.4, -1.1], dtype=torch.float64)
    a, b = torch.log1p(torch.exp(p)).item(), 0.5 + torch.log1p(torch.exp(q)).item()
    z = torch.linspace(-30, 30, 4 * 96).view(4, 96)
    want = O.xielu(z.double(), p, q)
    assert torch.allclose(grouped.activate(z, grouped.ACT_XIELU, a, b).double(), want, rtol=1e-5, atol=1e-7)
    part = grouped.activate(z, grouped.ACT_XIELU, a, b, 32)
    assert torch.equal(part[:, 32:], z[:, 32:]) and torch.allclose(part[:, :32].double(), want[:, :32], rtol=1e-5, atol=1e-7)
    small = torch.tensor([-1e-6, -1e-3, 1e-6, -0.2])
    want = O.xielu(small.double(), p, q)
    assert torch.allclose(grouped.activate(small, grouped.ACT_XIELU, a, b).double(), want, rtol=1e-6, atol=0)
    assert torch.equal(grouped.activate(z, grouped.ACT_SCALE, -0.5), -0.5 * z)


def test_boundary_with_a_gate_per_element():
    from trainscale_b200.ops import stream
    g = torch.Generator().manual_seed(1)
    x, y, z, b, w = (torch.randn(*s, generator=g) for s in ((5, 24), (5, 24), (5, 40), (24,), (24,)))
    gate = stream.ElementGate(z[:, 8:32], b)
    want = x + y * torch.sigmoid(z[:, 8:32] + b)
    for base in (0.0, 1.0):
        h = O.rms(want, 1e-4) * (base + w)
        xo, ho = stream.prenorm(x, y, gate, None, w, 1e-4, torch.float32, base)
        assert torch.allclose(xo, want, atol=1e-6) and torch.allclose(ho, h, atol=1e-5)
        assert torch.allclose(stream.prenorm_final(x, y, gate, None, w, 1e-4, torch.tensor([3, 0]), torch.float32, base), h[[3, 0]], atol=1e-5)


def test_slopes_and_temperature():
    from trainscale_b200.ops import window_attention as wa
    for H in (1, 2, 3, 8, 20):
        assert torch.allclose(wa.distance_slopes(H).double(), O.distance_slopes(H))
    s = wa.WindowShape(2, 1, 4, 4, 0, 99, 1.0, sigmoid=True, temperature=(0.3, 5))
    n = 40
    proj = torch.randn(n, s.q_width + s.kv_width, generator=torch.Generator().manual_seed(2))
    before, cache = proj.clone(), torch.zeros(10, 4, s.row_width)
    wa.prepare(proj, s, None, None, 1e-5, None, torch.arange(n), cache, pos=torch.arange(n, dtype=torch.int32))
    f = O.temperature(n, 0.3, 5)[:, None]
    assert torch.allclose(proj[:, :8].double(), before[:, :8] * f, rtol=1e-6) and torch.equal(proj[:, 8:], before[:, 8:])
    assert f[3] == 1 and f[4] > 1 and f[8] == f[4] and f[9] > f[8]


def test_powers_of_the_decays():
    from trainscale_b200.ops.recurrent import RETENTION_CHUNK, RetentionShape
    s = RetentionShape(3, 4, 6, 2, (0.984375, 0.3, 1.0))
    p = s.powers()
    assert p.shape == (3, RETENTION_CHUNK + 1) and (p[:, 0] == 1).all() and (p[2] == 1).all()
    assert torch.allclose(p[0, 1:].double(), 0.984375 ** torch.arange(1, RETENTION_CHUNK + 1, dtype=torch.float64), rtol=1e-7)
    assert s.state_width == 3 * 4 * 6 and s.proj_width == 2 * (12 + 18)


# ---------------------------------------------------------------------------------------------- the model in the engine
def test_whole_prompt_matches_oracle_with_unlike_layers():
    cfg, w, core = make()
    ids = tokens(41, 1)
    got = core.execute([StepEntry(0, ids, list(range(41)))])
    close(got, oracle(w, cfg, ids))
    close(core.model(torch.tensor([ids]))[0], oracle(w, cfg, ids))


def test_stream_after_every_layer():
    from trainscale_b200.inference.batch import HostBatch
    cfg, w, core = make()
    ids, seen = tokens(19, 2), {}
    batch = HostBatch(core.cache, [StepEntry(0, ids)]).to_device("cpu")
    core.model.serve(batch, core.cache, lambda n, x: seen.update({n: x.clone()}))
    trail = O.forward({k: v.double() for k, v in w.items()}, cfg, ids)[1]
    assert sorted(seen) == list(range(len(cfg["layers"]) - 1))
    for n, x in seen.items():
        close(x, trail[n], 1e-5)


@pytest.mark.parametrize("over", [
    dict(types=("attention",)), dict(types=("retention",)), dict(types=("latent_attention",)), dict(mlps=(0,)), dict(mlps=(1,)),
    dict(every=1, temp=0.0), dict(every=1000), dict(width=33, vocab=301), dict(heads=1, kv_heads=1, lheads=1, rheads=1), dict(types=("retention",), rdim=7, rot=6),
    dict(types=("retention",), rot=2), dict(types=("retention",), rdim=12, rot=12), dict(decay=((1.0,),)), dict(decay=((0.01, 0.999),)),
    dict(scale=[0.3, 1.0, 0.05]), dict(logit_scale=1.0), dict(logit_scale=-3.0), dict(ff=1), dict(ff=32), dict(eps=0.01), dict(rank=1, types=("latent_attention",))])
def test_other_sizes(over):
    cfg, w, core = make(**over)
    ids = tokens(23, 2)
    close(core.execute([StepEntry(0, ids, list(range(23)))]), oracle(w, cfg, ids))
    close(run_portions(core, 1, ids, [2, 2, 3, 5]), oracle(w, cfg, ids))


@pytest.mark.parametrize("sizes", [[1], [2] * 30, [3, 2, 7, 1, 4, 16], [40], [4] * 20, [5, 1, 1, 30]])
def test_portions_and_decoding_match_whole_prompt(sizes):
    cfg, w, core = make()
    ids = tokens(41, 3)
    close(run_portions(core, 0, ids, sizes), oracle(w, cfg, ids))


def test_long_decoding():
    cfg, w, core = make(types=("retention", "attention", "latent_attention"), decay=((0.999, 0.95),))
    ids = tokens(150, 4)
    close(run_portions(core, 0, ids, [2]), oracle(w, cfg, ids))


def test_batch_of_unequal_requests_and_reuse_of_pages_and_slots():
    """Requests of different lengths advance by different amounts in one batch; finished ones give pages and state slots to new
    ones (the pool holds only a few at a time)."""
    cfg, w, core = make(blocks=40, seqs=3)
    reqs = {f"r{i}": tokens(n, 10 + i) for i, n in enumerate([37, 5, 22, 1, 48, 13, 29, 2])}
    waiting, live, at = list(reqs), [], {}
    runner, got, step = TraceRunner(core), {r: [] for r in reqs}, 0
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
        entries, end = [], []
        for j, r in enumerate(live):
            lo = at.get(r, 0)
            n = min([1, 9, 2, 5, 1, 3][(step + j) % 6], len(reqs[r]) - lo)
            if (step + j) % 5 == 4:
                continue                      # left out of this step
            entries.append({"id": r, "tokens": reqs[r][lo:lo + n], "want": list(range(n))})
            at[r] = lo + n
            if at[r] == len(reqs[r]):
                end.append(r)
        logits = runner.run({"step": step, "entries": entries, "end": end})
        row = 0
        for e in entries:
            got[e["id"]].append(logits[row:row + len(e["want"])])
            row += len(e["want"])
        live = [r for r in live if r not in end]
        step += 1
    assert core.cache.alloc.num_free == 40 and sorted(core.cache.free_slots) == [0, 1, 2]
    for r, ids in reqs.items():
        close(torch.cat(got[r]), oracle(w, cfg, ids))


def test_want_nothing_still_advances():
    cfg, w, core = make()
    ids = tokens(12, 5)
    assert core.execute([StepEntry(0, ids[:7], [])]) is None
    close(core.execute([StepEntry(0, ids[7:], [4, 0])]), oracle(w, cfg, ids)[[11, 7]])


@pytest.mark.parametrize("kind", ["attention", "retention", "latent_attention"])
def test_every_earlier_token_matters_and_no_later_one(kind):
    """With one layer: a changed token moves its own logits and those of every later position, however the tokens are cut (slow
    decays and gentle slopes, so that none of it is lost), and none before it."""
    cfg, w, core = make(types=(kind,), mlps=(1,), heads=4, kv_heads=2, decay=((0.9, 0.99),))
    n, base = 33, tokens(33, 6)
    for sizes in ([n], [n - 1, 1], [n - 2, 2], [5, 3, n - 8], [1]):
        def logits(ids):
            y = run_portions(core, 0, ids, sizes)
            core.release(0)
            return y
        ref = logits(base)
        for at in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32):
            ids = list(base)
            ids[at] = (base[at] + 1) % 300
            d = (logits(ids) - ref).abs().max(-1).values
            assert (d[:at] == 0).all() and (d[at:] > 1e-6).all(), (sizes, at)


@pytest.mark.parametrize("kind", ["attention", "latent_attention", "retention"])
@pytest.mark.parametrize("place", [0, 4, 11, 60])
def test_far_key_is_found(kind, place):
    """The last token's query is made to point at the key of one earlier token, which takes most of the weight (or more than
    its share of the state's answer): missing it, or its place, is far above the tolerance."""
    n, H = 64, 1
    ids = tokens(n, 7)
    ids[place], ids[n - 1] = 298, 299
    others = ids[:place] + ids[place + 1:n - 1]
    ids = [t if t not in (298, 299) or i in (place, n - 1) else 5 for i, t in enumerate(ids)]
    assert len(others) == n - 2
    moved = {}
    for point in (True, False):
        cfg = O.make_config(types=(kind,), mlps=(1,), heads=H, kv_heads=1, lheads=1, rheads=1, rot=2, base=1e30, decay=((0.98,),), temp=0.2, every=16)
        w = O.make_weights(cfg, 0, 2.0)
        eps, p, m = cfg["norm"]["eps"], "l0.mix.", cfg["layers"][0]["mixer"]
        x = O.norm(w["embed"][[298, 299]], w["l0.norm1"], eps)
        if kind == "attention":
            w[p + "pb"] = torch.full((H,), -4.0)
            w[p + "q.norm"] = torch.full((m["dim"],), 3.0)
            w[p + "k.norm"] = torch.full((m["dim"],), 3.0)
        if point:
            if kind == "latent_attention":
                key = w[p + "uk"] @ O.norm(x[0] @ w[p + "dkv"].t(), w[p + "dkv.norm"], eps)
            else:
                key = w[p + "k"] @ x[0]
            q = w[p + "q"]
            w[p + "q"] = (q + torch.outer(6 * key - q @ x[1], x[1]) / (x[1] @ x[1])).to(torch.bfloat16).float()
        core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", cache=CacheConfig(block_size=4, num_gpu_blocks=64)),
                          model=load_model(cfg, w, torch.float32))
        want = oracle(w, cfg, ids)
        for i, sizes in enumerate(([64], [50, 2, 5, 7], [40], [61, 2, 1])):
            close(run_portions(core, i, ids, sizes), want)
            core.release(i)
        swapped = list(ids)
        swapped[place] = 17
        moved[point] = (oracle(w, cfg, swapped)[-1] - want[-1]).abs().max() / want[-1].abs().max()
    assert moved[True] > 0.01 and (kind == "retention" or moved[True] > 2 * moved[False]), moved     # a state's answer is normed


def test_first_tokens_alone_and_after_pages_were_used():
    cfg, w, core = make(seqs=1)
    for i, ids in enumerate([[17], [0], [299, 3], tokens(30, 1), [17], [5, 5]]):
        close(core.execute([StepEntry(i, ids, list(range(len(ids))))]), oracle(w, cfg, ids))
        core.release(i)


def test_planted_mistakes_show():
    """The test weights are sharp enough: each constant or tensor, altered in the oracle, moves the logits far beyond `close`."""
    cfg, w, _ = make()
    ids = tokens(40, 8)
    want = oracle(w, cfg, ids)

    def moved(w2, c):
        return (oracle(w2, c, ids) - want).abs().max() > 2e-3 * want.abs().max()

    def mixer(c, i):
        return c["layers"][i]["mixer"]

    changes = {
        "scale": lambda c: mixer(c, 0).update(scale=mixer(c, 0)["scale"] * 1.05),
        "latent scale": lambda c: mixer(c, 2).update(scale=mixer(c, 2)["scale"] * 1.05),
        "temperature": lambda c: mixer(c, 0)["q_temp"].update(coef=0.45),
        "steps of the temperature": lambda c: mixer(c, 0)["q_temp"].update(every=6),
        "base": lambda c: mixer(c, 1)["rot"].update(base=mixer(c, 1)["rot"]["base"] * 1.5),
        "rotated dimensions": lambda c: mixer(c, 3)["rot"].update(dims=mixer(c, 3)["rot"]["dims"] - 2),
        "decay": lambda c: mixer(c, 1).update(decay=[d * 0.99 for d in mixer(c, 1)["decay"]]),
        "order of the decays": lambda c: mixer(c, 3).update(decay=mixer(c, 3)["decay"][::-1]),
        "logit scale": lambda c: c.update(logit_scale=0.59),
        "eps": lambda c: c["norm"].update(eps=0.1)}
    for name, change in changes.items():
        c = copy.deepcopy(cfg)
        change(c)
        assert moved(w, c), name
    for name in w:
        assert moved({**w, name: w[name] * 1.05 + 0.01}, cfg) or moved({**w, name: w[name] * 1.5 + 0.3}, cfg), name


def test_greedy_generation_with_chunked_prefill_and_preemption():
    """Greedy tokens through `generate` equal the oracle's: ample cache, prompts cut into portions by a small token budget,
    and a pool so small that requests are preempted and computed again."""
    cfg, w, core = make()
    prompts = [tokens(n, 30 + n) for n in (19, 3, 33, 8, 26)]
    want = [O.greedy(w, cfg, p, 9) for p in prompts]
    for kw in (dict(), dict(budget=7), dict(seqs=2), dict(blocks=14), dict(blocks=14, budget=5)):
        _, _, core = make(**kw)
        eng = SOTAInferenceEngine.__new__(SOTAInferenceEngine)
        eng.config, eng.core, eng.draft_model = core.config, core, None
        res = eng.generate(prompts, GenerationParams(max_tokens=9, temperature=0.0, ignore_eos=True)).unwrap()
        assert [r.token_ids for r in res] == want, kw
        assert core.cache.alloc.num_free == core.cache.alloc.num_blocks


def test_prefixes_are_shared_only_without_state():
    """Layers with a state cannot start in the middle of a shared prefix; a model of attending layers alone takes it over."""
    common = tokens(24, 3)
    for types, shared in ((("retention", "attention"), 0), (("latent_attention", "attention"), 24)):
        cfg, w, core = make(prefix=True, types=types)
        for tail in ([], tokens(9, 4), tokens(13, 5)):
            before = core.cache.prefix_hits
            r = core.add_request(common + tail, GenerationParams(max_tokens=4, temperature=0.0, ignore_eos=True))
            while core.has_unfinished():
                core.step()
            assert r.output_ids == O.greedy(w, cfg, common + tail, 4)
            assert core.cache.prefix_hits - before == (shared if tail else 0)


def test_checkpoint_directory_round_trip(tmp_path):
    """config.json picks the class; weights written by `to_checkpoint` load again; a wrong checkpoint is refused."""
    cfg = O.make_config(**MIXED)
    w = O.make_weights(cfg, 3)
    m = load_model(cfg, w, torch.float32)
    (tmp_path / "config.json").write_text(json.dumps(m.config.to_dict()))
    ModelSerializer().save(m.to_checkpoint(), tmp_path)
    m2 = load_pretrained(tmp_path, dtype=torch.float32)
    assert isinstance(m2, LovuraxForCausalLM) and m2.config == m.config == LovuraxConfig.from_dict(cfg)
    ids = torch.tensor([tokens(9, 4)])
    assert torch.equal(m(ids), m2(ids))
    sd = m.to_checkpoint()
    assert sd.keys() == w.keys() and all(torch.equal(sd[k].float(), w[k]) for k in w)
    with pytest.raises(KeyError):
        load_model(cfg, {k: v for k, v in w.items() if k != "l0.rg1.b"}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l1.mix.o": w["l1.mix.o"][:-1]}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l0.mlp.up": w["l0.mlp.up"][:-1]}, torch.float32)
    core = EngineCore(EngineConfig(model=str(tmp_path), device="cpu"))      # no tokenizer files: bytes
    assert core.tokenizer.encode_raw("ab", add_special_tokens=False) == [97, 98]


def test_configurations_the_class_cannot_run_are_refused():
    cases = [(0, ("type",), "other"), (2, ("mixer", "kv_heads"), 3), (2, ("mixer", "q_temp", "every"), 0), (2, ("mixer", "q_temp", "every"), 2.5),
             (1, ("mixer", "rot", "dims"), 3), (1, ("mixer", "rot", "dims"), 400), (1, ("mixer", "decay"), [0.5]), (1, ("mixer", "dim"), 300),
             (1, ("mixer", "vdim"), 600), (0, ("mlp", "kind"), "moe")]
    for layer, path, value in cases:
        cfg = O.make_config()
        d = cfg["layers"][layer]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            LovuraxConfig.from_dict(cfg)
    with pytest.raises(ValueError):
        LovuraxConfig.from_dict({**O.make_config(), "layers": []})
    assert architecture_of({"architecture": "Lovurax"}).name == "Lovurax"


def test_features_of_the_llama_path_are_refused_with_a_reason():
    _, _, core = make()
    with pytest.raises(ValueError, match="LoRA"):
        core.load_adapters({"a": {}})
    cfg = EngineConfig(model="custom", tokenizer="byte", device="cpu")
    cfg.parallel.tensor_parallel_size = 2
    with pytest.raises(ValueError, match="one GPU"):
        EngineCore(cfg, model=core.model)


def test_cache_spec_presets_and_registry():
    from trainscale_b200.models import is_preset
    from trainscale_b200.registry import MODEL_REGISTRY
    assert is_preset("lovurax-tiny") and is_preset("lovurax-2b")
    assert MODEL_REGISTRY["lovurax"].architecture == "LovuraxForCausalLM"
    a, b = build_model("lovurax-tiny", torch.float32, seed=5), build_model("lovurax-tiny", torch.float32, seed=5)
    assert all(torch.equal(x, y) for x, y in zip(a.parameters(), b.parameters()))
    assert torch.isfinite(a(torch.tensor([tokens(20, 1)]))).all()
    spec = a.cache_spec()
    assert spec.has_state and spec.bytes_per_token(2) == 2 * (2 * 128 + 96) and spec.bytes_per_sequence() == 2 * 4 * 2 * 2 * 64 * 128
    assert math.isclose(a.config.layers[0].mixer.shape.decay[0], 1 - 2.0 ** -5)


def test_cli_batch(capsys):
    from trainscale_b200.inference import main
    assert main(["batch", "--model", "lovurax-tiny", "--prompt", "hi", "--max-tokens", "3", "--temperature", "0"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["finish_reason"] in ("length", "stop")
