"""Vibepel through the engine on the CPU (PyTorch math of the ops): the cache, the state slots, batching, scheduling and
generation against the plain statement of the design in vibepel_oracle.py."""
import copy
import json

import pytest
import torch

import vibepel_oracle as O
from trainscale_b200.hub import ModelSerializer, load_pretrained
from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, GenerationParams, SchedulerConfig, SOTAInferenceEngine
from trainscale_b200.inference.batch import StepEntry
from trainscale_b200.inference.trace import TraceRunner
from trainscale_b200.models import architecture_of
from trainscale_b200.models.vibepel import VibepelConfig, VibepelForCausalLM, build_model, load_model

# unlike layers: every size and constant differs from layer to layer
MIXED = dict(width=40, types=("wkv", "parallel", "parallel", "wkv"), heads=[6, 4, 3], kv_heads=[2, 4, 1], dim=[12, 8, 10],
             vdim=[6, 16, 10], window=[19, 5, 7], rot=[8, 8, 4], base=[500.0, 50.0, 3000.0], dheads=[4, 2, 3], dkv=[2, 1, 3],
             ddim=[8, 12, 6], dvdim=[10, 12, 4], taps=[4, 1, 3], wheads=[3, 2], wdim=[8, 12], ff=[40, 17, 64], decay_rank=[5, 12],
             left_scale=[0.7, 1.4], right_scale=[1.1, 0.4], scaling=[O.SCALING, None, {"factor": 2.0, "low": 1.0, "high": 2.0, "original": 20}])


def make(seed=0, sharp=1.5, blocks=64, block_size=4, seqs=4, budget=512, slow=False, **over):
    cfg = O.make_config(**{**MIXED, **over})
    w = O.make_weights(cfg, seed, sharp, slow)
    core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", dtype="float32",
                                   scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                                   cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=256)),
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


def test_whole_prompt_matches_oracle_with_unlike_layers():
    cfg, w, core = make()
    ids = tokens(41, 1)
    got = core.execute([StepEntry(0, ids, list(range(41)))])
    close(got, oracle(w, cfg, ids))
    close(core.model(torch.tensor([ids]))[0], oracle(w, cfg, ids))


@pytest.mark.parametrize("over", [dict(mlp_every=2), dict(types=("parallel",)), dict(types=("wkv",)), dict(window=1), dict(window=1000),
                                  dict(width=33, vocab=301), dict(taps=6), dict(heads=1, kv_heads=1, dheads=1, dkv=1, wheads=1),
                                  dict(rot=2, dim=7, vdim=3, ddim=5, dvdim=3, wdim=3, types=("parallel", "wkv")),
                                  dict(types=("parallel", "wkv"), mlp_every=3, left_scale=1.0, right_scale=1.0)])
def test_other_sizes(over):
    cfg, w, core = make(**over)
    ids = tokens(23, 2)
    close(core.execute([StepEntry(0, ids, list(range(23)))]), oracle(w, cfg, ids))
    close(run_portions(core, 1, ids, [2, 2, 3, 5]), oracle(w, cfg, ids))


@pytest.mark.parametrize("sizes", [[1], [2] * 30, [3, 2, 7, 1, 4, 16], [40], [4] * 20, [5, 1, 1, 30]])
def test_portions_and_decoding_match_whole_prompt(sizes):
    cfg, w, core = make(slow=True)
    ids = tokens(41, 3)
    close(run_portions(core, 0, ids, sizes), oracle(w, cfg, ids))


def test_batch_of_unequal_requests_and_reuse_of_pages_and_slots():
    """Requests of different lengths advance by different amounts in one batch; finished ones give their pages and state
    slots to new ones (the pool holds only a few at a time)."""
    cfg, w, core = make(blocks=40, seqs=3, slow=True)
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
    assert core.cache.alloc.num_free == 40 and len(core.cache.free_slots) == 3
    for r, ids in reqs.items():
        close(torch.cat(got[r]), oracle(w, cfg, ids))


def test_want_nothing_still_advances():
    cfg, w, core = make()
    ids = tokens(12, 5)
    assert core.execute([StepEntry(0, ids[:7], [])]) is None
    close(core.execute([StepEntry(0, ids[7:], [4, 0])]), oracle(w, cfg, ids)[[11, 7]])


@pytest.mark.parametrize("window", [1, 4, 5, 8, 9])
def test_window_edge_in_prompts_and_decoding(window):
    """With one attention layer and the delta rule's share set to zero, the token `window - 1` back matters and the one
    `window` back does not."""
    cfg, w, core = make(types=("parallel",), window=window, right_scale=0.0)
    n, base = 21, tokens(21, 6)
    for k, sizes in enumerate(([n], [n - 1, 1], [n - 2, 2], [5, 3, n - 8])):
        ref = run_portions(core, 3 * k, base, sizes)[-1]
        inside, outside = list(base), list(base)
        inside[n - window] = (base[n - window] + 1) % 300
        outside[n - 1 - window] = (base[n - 1 - window] + 1) % 300
        assert torch.equal(run_portions(core, 3 * k + 1, outside, sizes)[-1], ref)
        assert (run_portions(core, 3 * k + 2, inside, sizes)[-1] - ref).abs().max() > 1e-3
        for s in (3 * k, 3 * k + 1, 3 * k + 2):
            core.release(s)


def test_far_key_inside_the_window_is_found():
    """The last token's query is made to point at the key of one token near the window's far end, which then takes most of the
    weight: missing it shows at once, and so does seeing it when it has just left the window."""
    ids = tokens(64, 7)
    ids[4], ids[63] = 298, 299
    assert 298 not in ids[5:] + ids[:4] and 299 not in ids[:63]
    results = {}
    for window in (60, 59):
        slow = {"factor": 1e6, "low": 1.0, "high": 2.0, "original": 1}      # hardly any rotation between the two
        cfg = O.make_config(types=("parallel",), window=window, heads=1, kv_heads=1, rot=2, scaling=slow, right_scale=0.0)
        w = O.make_weights(cfg, 0, 3.0)
        x = w["embed"][299] * cfg["embedding"]["scale"]
        key = w["l0.mix.left.k"] @ (w["embed"][298] * cfg["embedding"]["scale"])
        q = w["l0.mix.left.q"]
        w["l0.mix.left.q"] = (q + torch.outer(4 * key - q @ x, x) / (x @ x)).to(torch.bfloat16).float()
        core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", cache=CacheConfig(block_size=4, num_gpu_blocks=64)),
                          model=load_model(cfg, w, torch.float32))
        want = oracle(w, cfg, ids)
        for i, sizes in enumerate(([64], [50, 2, 5, 7], [40], [61, 2, 1])):
            close(run_portions(core, i, ids, sizes), want)
            core.release(i)
        results[window] = want[-1]
    assert (results[60] - results[59]).abs().max() > 0.3


@pytest.mark.parametrize("types", [("wkv",), ("parallel",)])
def test_recurrent_state_remembers_the_first_token(types):
    """The very first token still moves the logits fifty tokens later, also when everything between is decoded singly."""
    cfg, w, core = make(types=types, slow=True, left_scale=0.0, taps=2)
    a, b = tokens(50, 8), tokens(50, 8)
    b[0] = (a[0] + 3) % 300
    want = oracle(w, cfg, a)[-1], oracle(w, cfg, b)[-1]
    assert (want[0] - want[1]).abs().max() > 5e-3
    for i, sizes in enumerate(([50], [1], [2, 3, 1, 20])):
        close(run_portions(core, 2 * i, a, sizes)[-1], want[0])
        close(run_portions(core, 2 * i + 1, b, sizes)[-1], want[1])
        core.release(2 * i), core.release(2 * i + 1)


def test_first_tokens_alone_and_after_a_slot_was_used():
    cfg, w, core = make(seqs=1)
    for i, ids in enumerate([[17], [0], [299, 3], tokens(30, 1), [17], [5, 5]]):
        close(core.execute([StepEntry(i, ids, list(range(len(ids))))]), oracle(w, cfg, ids))
        core.release(i)


def test_planted_mistakes_show():
    """The test weights are sharp enough: each constant or tensor, altered in the oracle, moves the logits far beyond `close`."""
    cfg, w, _ = make(slow=True)
    ids = tokens(30, 8)
    want = oracle(w, cfg, ids)

    def moved(w2, c):
        return (oracle(w2, c, ids) - want).abs().max() > 2e-3 * want.abs().max()

    def left(c):
        return c["layers"][1]["mixer"]["left"]

    changes = {
        "window": lambda c: left(c)["mask"].update(size=left(c)["mask"]["size"] + 1),
        "scale": lambda c: left(c).update(scale=left(c)["scale"] * 1.05),
        "base": lambda c: left(c)["rot"].update(base=left(c)["rot"]["base"] * 1.5),
        "rotated dimensions": lambda c: left(c)["rot"].update(dims=left(c)["rot"]["dims"] - 2),
        "scaling": lambda c: c["layers"][2]["mixer"]["left"]["rot"]["scaling"].update(factor=3.0),
        "left scale": lambda c: c["layers"][1]["mixer"].update(left_scale=1.5),
        "right scale": lambda c: c["layers"][1]["mixer"].update(right_scale=0.5),
        "embedding scale": lambda c: c["embedding"].update(scale=2.6),
        "soft cap": lambda c: c.update(logit_softcap=19.0)}
    for name, change in changes.items():
        c = copy.deepcopy(cfg)
        change(c)
        assert moved(w, c), name
    for name in w:
        if name == "l2.mix.right.b":           # (checked with a larger change below)
            continue
        w2 = {**w, name: w[name] * 1.05 + 0.01}
        if not moved(w2, cfg):
            assert moved({**w, name: w[name] * 1.5 + 0.3}, cfg), name


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
        assert len(core.cache.free_slots) == core.cache.state_slots


def test_checkpoint_directory_round_trip(tmp_path):
    """config.json picks the class; weights written by `to_checkpoint` load again; a wrong checkpoint is refused.  The inner
    size of the WKV decay comes from the tensor when config.json does not name it."""
    cfg = O.make_config(**MIXED, mlp_every=2)
    w = O.make_weights(cfg, 3)
    m = load_model(cfg, w, torch.float32)
    (tmp_path / "config.json").write_text(json.dumps(m.config.to_dict()))
    ModelSerializer().save(m.to_checkpoint(), tmp_path)
    m2 = load_pretrained(tmp_path, dtype=torch.float32)
    assert isinstance(m2, VibepelForCausalLM) and m2.config == m.config == VibepelConfig.from_dict(cfg)
    ids = torch.tensor([tokens(9, 4)])
    assert torch.equal(m(ids), m2(ids))
    sd = m.to_checkpoint()
    assert sd.keys() == w.keys() and all(torch.equal(sd[k].float(), w[k]) for k in w)
    silent = copy.deepcopy(cfg)
    for l in silent["layers"]:
        l["mixer"].pop("decay_rank", None)
    assert load_model(silent, w, torch.float32).config == m.config
    with pytest.raises(KeyError):
        load_model(cfg, {k: v for k, v in w.items() if k != "l0.mix.u"}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l1.mix.left.o": w["l1.mix.left.o"][:-1]}, torch.float32)
    core = EngineCore(EngineConfig(model=str(tmp_path), device="cpu"))      # no tokenizer files: bytes
    assert core.tokenizer.encode_raw("ab", add_special_tokens=False) == [97, 98]


def test_configurations_the_class_cannot_run_are_refused():
    for path, value in ((("type",), "other"), (("mixer", "left", "rot", "dims"), 3), (("mixer", "left", "rot", "dims"), 400),
                        (("mlp", "kind"), "moe"), (("mixer", "left", "kv_heads"), 3), (("mixer", "right", "kv_heads"), 3),
                        (("mixer", "right", "dim"), 300), (("mixer", "left", "mask", "size"), 0)):
        cfg = O.make_config(types=("parallel",))
        d = cfg["layers"][0]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            VibepelConfig.from_dict(cfg)
    assert architecture_of({"architecture": "Vibepel"}).name == "Vibepel"


def test_features_of_the_llama_path_are_refused_with_a_reason():
    _, _, core = make()
    with pytest.raises(ValueError, match="LoRA"):
        core.load_adapters({"a": {}})
    cfg = EngineConfig(model="custom", tokenizer="byte", device="cpu")
    cfg.parallel.tensor_parallel_size = 2
    with pytest.raises(ValueError, match="one GPU"):
        EngineCore(cfg, model=core.model)


def test_prefix_sharing_is_off_for_models_with_state():
    cfg, w, core = make()
    ids = tokens(24, 3)
    outs = []
    for _ in range(2):
        r = core.add_request(ids, GenerationParams(max_tokens=4, temperature=0.0, ignore_eos=True))
        while core.has_unfinished():
            core.step()
        outs.append(r.output_ids)
    assert outs[0] == outs[1] == O.greedy(w, cfg, ids, 4) and core.cache.prefix_hits == 0


def test_cache_spec_presets_and_registry():
    from trainscale_b200.models import is_preset
    from trainscale_b200.registry import MODEL_REGISTRY
    assert is_preset("vibepel-tiny") and is_preset("vibepel-2b")
    assert MODEL_REGISTRY["vibepel"].architecture == "VibepelForCausalLM"
    a, b = build_model("vibepel-tiny", torch.float32, seed=5), build_model("vibepel-tiny", torch.float32, seed=5)
    assert all(torch.equal(x, y) for x, y in zip(a.parameters(), b.parameters()))
    assert torch.isfinite(a(torch.tensor([tokens(20, 1)]))).all()
    spec = a.cache_spec()
    assert spec.has_state and spec.bytes_per_token(2) == 3 * 2 * 2 * 128 and spec.paged[3] == {}
    only = O.make_config(types=("wkv",))                   # a model without any paged entry
    core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu"), model=load_model(only, O.make_weights(only), torch.float32))
    assert core.execute([StepEntry(0, [1, 2, 3])]).shape == (1, 300)


def test_block_scan_algebra():
    """The identities behind the scans in blocks: (I + L)^-1 form of the delta rule, decayed Gram form of WKV."""
    g = torch.Generator().manual_seed(1)
    n, D, V = 8, 6, 5
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)   # noqa: E731
    q, k, v, S0 = rnd(n, 1, D), O.unit(rnd(n, 1, D)), rnd(n, 1, V), rnd(1, D, V)
    lg, beta = -torch.rand(n, 1, generator=g, dtype=torch.float64), torch.rand(n, 1, generator=g, dtype=torch.float64)
    o, S = O.delta_recurrence(q, k, v, lg.exp(), beta, S0)
    c = lg[:, 0].cumsum(0)
    ratio = (c[:, None] - c[None]).exp().tril()
    L = (beta * ratio * (k[:, 0] @ k[:, 0].t())).tril(-1)
    U = torch.linalg.solve(torch.eye(n, dtype=torch.float64) + L, beta * (v[:, 0] - c.exp()[:, None] * (k[:, 0] @ S0[0])))
    assert torch.allclose(c.exp()[:, None] * (q[:, 0] @ S0[0]) + (ratio * (q[:, 0] @ k[:, 0].t())) @ U, o[:, 0])
    assert torch.allclose(c[-1].exp() * S0[0] + (k[:, 0] * (c[-1] - c).exp()[:, None]).t() @ U, S[0])
    w, u = torch.rand(n, 1, D, generator=g, dtype=torch.float64), rnd(1, D)
    o, S = O.wkv_recurrence(q, k, v, w, u, S0)
    cw = w[:, 0].log().cumsum(0)
    before = torch.cat([torch.zeros(1, D, dtype=torch.float64), cw[:-1]])
    A = torch.zeros(n, n, dtype=torch.float64)
    for i in range(n):
        A[i, i] = (q[i, 0] * u[0] * k[i, 0]).sum()
        for j in range(i):
            A[i, j] = (q[i, 0] * k[j, 0] * (before[i] - cw[j]).exp()).sum()
    assert torch.allclose((q[:, 0] * before.exp()) @ S0[0] + A @ v[:, 0], o[:, 0])
    assert torch.allclose(cw[-1].exp()[:, None] * S0[0] + (k[:, 0] * (cw[-1] - cw).exp()).t() @ v[:, 0], S[0])


def test_cli_batch(capsys):
    from trainscale_b200.inference import main
    assert main(["batch", "--model", "vibepel-tiny", "--prompt", "hi", "--max-tokens", "3", "--temperature", "0"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["finish_reason"] in ("length", "stop")
