"""Mezilix through the engine on the CPU (PyTorch math of the ops): the cache, the state slots, batching, scheduling and
generation against the plain statement of the design in mezilix_oracle.py."""
import json

import pytest
import torch

import mezilix_oracle as O
from trainscale_b200.hub import ModelSerializer, load_pretrained
from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, GenerationParams, SchedulerConfig, SOTAInferenceEngine
from trainscale_b200.inference.batch import StepEntry
from trainscale_b200.inference.trace import TraceRunner
from trainscale_b200.models import architecture_of
from trainscale_b200.models.llama import LlamaForCausalLM
from trainscale_b200.models.mezilix import MezilixConfig, MezilixForCausalLM, build_model, load_model

MIXED = dict(layers=3, heads=[2, 3, 1], dim=[24, 12, 40], rot_dim=[8, 4, 16], vdim=[16, 20, 8], kv_rank=[40, 24, 33],
             window=[7, 19, 3], experts=[5, 3, 4], top=[2, 1, 4], ff=[24, 10, 17], base=[500.0, 10000.0, 50.0])


def make(seed=0, sharp=2.0, blocks=64, block_size=4, seqs=4, budget=512, **over):
    cfg = O.make_config(**{**MIXED, **over})
    w = O.make_weights(cfg, seed, sharp)
    core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", dtype="float32",
                                   scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                                   cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=256)),
                      model=load_model(cfg, w, torch.float32))
    return cfg, w, core


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
    close(got, O.logits(w, cfg, ids))
    close(core.model(torch.tensor([ids]))[0], O.logits(w, cfg, ids))


@pytest.mark.parametrize("over", [dict(mlp_every=2), dict(layers=1), dict(heads=1, top=1, experts=1), dict(window=1),
                                  dict(window=1000), dict(width=50, kv_rank=7, dim=3, rot_dim=2, vdim=5, ff=9)])
def test_other_sizes(over):
    cfg, w, core = make(**over)
    ids = tokens(23, 2)
    close(core.execute([StepEntry(0, ids, list(range(23)))]), O.logits(w, cfg, ids))
    close(run_portions(core, 1, ids, [2, 2, 3, 5]), O.logits(w, cfg, ids))


@pytest.mark.parametrize("sizes", [[1], [2] * 30, [3, 2, 7, 1, 4, 16], [40], [4] * 20, [5, 1, 1, 30]])
def test_portions_and_decoding_match_whole_prompt(sizes):
    cfg, w, core = make()
    ids = tokens(41, 3)
    close(run_portions(core, 0, ids, sizes), O.logits(w, cfg, ids))


def test_batch_of_unequal_requests_and_reuse_of_pages_and_slots():
    """Requests of different lengths advance by different amounts in one batch; finished ones give their pages and state
    slots to new ones (the pool holds only a few at a time)."""
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
    assert core.cache.alloc.num_free == 40 and len(core.cache.free_slots) == 3
    for r, ids in reqs.items():
        close(torch.cat(got[r]), O.logits(w, cfg, ids))


def test_want_nothing_still_advances():
    cfg, w, core = make()
    ids = tokens(12, 5)
    assert core.execute([StepEntry(0, ids[:7], [])]) is None
    close(core.execute([StepEntry(0, ids[7:], [4, 0])]), O.logits(w, cfg, ids)[[11, 7]])


@pytest.mark.parametrize("window", [1, 4, 5, 8, 9])
def test_window_edge_in_prompts_and_decoding(window):
    """Changing the token that is `window - 1` back changes a single-layer model's attention, the one `window` back does
    not: with one layer nothing else carries information that far (the bigram and the shift reach one token)."""
    cfg, w, core = make(layers=1, window=window, heads=2, dim=24, rot_dim=8, vdim=16, kv_rank=40)
    n = 21
    base = tokens(n, 6)

    def last(ids, sizes, seq):
        return run_portions(core, seq, ids, sizes)[-1]

    for k, sizes in enumerate(([n], [n - 1, 1], [n - 2, 2], [5, 3, n - 8])):
        ref = last(base, sizes, 3 * k)
        # a key is h of its own and of the previous token, embedding pairs reach one further: position p depends on
        # tokens p, p - 1 (shift) and p - 2 (bigram of the shifted one)
        inside, outside = list(base), list(base)
        inside[n - window] = (base[n - window] + 1) % 300
        far = n - 1 - window - 2
        if far >= 0:
            outside[far] = (base[far] + 1) % 300
            assert torch.equal(last(outside, sizes, 3 * k + 1), ref)
        assert (last(inside, sizes, 3 * k + 2) - ref).abs().max() > 1e-3
        for s in (3 * k, 3 * k + 1, 3 * k + 2):
            core.release(s)


def test_far_key_inside_the_window_is_found():
    """One key far back is made to dominate: its query/key pair gets a large score, so missing it shows at once."""
    cfg, w, core = make(layers=1, window=60, heads=1, dim=16, rot_dim=4, vdim=16, kv_rank=32, sharp=6.0)
    ids = tokens(64, 7)
    want = O.logits(w, cfg, ids)
    close(run_portions(core, 0, ids, [50, 2, 5, 1]), want)
    changed = list(ids)
    changed[4:9] = [(t + 7) % 300 for t in ids[4:9]]
    assert (O.logits(w, cfg, changed)[63] - want[63]).abs().max() > 1e-3
    close(run_portions(core, 1, changed, [50, 2, 5, 1]), O.logits(w, cfg, changed))


def test_first_token_uses_the_extra_bigram_row_and_zero_shift():
    cfg, w, core = make()
    for t in (0, 17, 299):
        close(core.execute([StepEntry(t, [t], [0])]), O.logits(w, cfg, [t]))
        core.release(t)
    other = {**w, "bigram": w["bigram"].clone()}
    other["bigram"][-1] += 1.0
    assert (O.logits(other, cfg, [17]) - O.logits(w, cfg, [17])).abs().max() > 1e-3


def test_planted_mistakes_show():
    """The test weights are sharp enough: each mechanism, altered in the oracle, moves the logits far beyond `close`."""
    cfg, w, _ = make()
    ids = tokens(30, 8)
    want = O.logits(w, cfg, ids)
    import copy
    for change in ("window", "mul_prev", "scale", "base", "top"):
        c = copy.deepcopy(cfg)
        if change == "window":
            c["layers"][1]["mixer"]["mask"]["size"] += 1
        elif change == "mul_prev":
            c["embedding"]["bigram"]["mul_prev"] += 1
        elif change == "scale":
            c["layers"][0]["mixer"]["scale"] *= 1.05
        elif change == "base":
            c["layers"][0]["mixer"]["rot"]["base"] *= 1.5
        else:
            c["layers"][0]["mlp"]["router"]["top"] = 1
        assert (O.logits(w, c, ids) - want).abs().max() > 2e-3 * want.abs().max(), change
    for name in ("l1.shift", "l0.dwa", "l2.mix.dkv.norm", "l1.norm1"):
        w2 = {**w, name: w[name] * 1.05 + 0.01}
        assert (O.logits(w2, cfg, ids) - want).abs().max() > 2e-3 * want.abs().max(), name


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


def test_request_larger_than_the_cache_is_an_error():
    _, _, core = make(blocks=3)
    core.add_request(tokens(30, 1), GenerationParams(max_tokens=2))
    with pytest.raises(MemoryError):
        while core.has_unfinished():
            core.step()


def test_invalid_steps_are_refused_on_the_host():
    _, _, core = make(blocks=4)
    with pytest.raises(ValueError):
        core.execute([StepEntry(0, [1, 300], [0])])
    with pytest.raises(ValueError):
        core.execute([StepEntry(0, [1, 2], [2])])
    with pytest.raises(ValueError):
        core.execute([StepEntry(0, [1], [0]), StepEntry(0, [2], [0])])
    with pytest.raises(MemoryError):
        core.execute([StepEntry(0, tokens(17, 1), [0])])
    with pytest.raises(ValueError):
        core.add_request([5, -1])
    assert core.cache.alloc.num_free == 4


def test_checkpoint_directory_round_trip(tmp_path):
    """config.json picks the class; weights written by `to_checkpoint` load again; a wrong checkpoint is refused."""
    cfg = O.make_config(**MIXED, mlp_every=2)
    w = O.make_weights(cfg, 3)
    m = load_model(cfg, w, torch.float32)
    (tmp_path / "config.json").write_text(json.dumps(m.config.to_dict()))
    ModelSerializer().save(m.to_checkpoint(), tmp_path)
    m2 = load_pretrained(tmp_path, dtype=torch.float32)
    assert isinstance(m2, MezilixForCausalLM) and m2.config == m.config == MezilixConfig.from_dict(cfg)
    ids = torch.tensor([tokens(9, 4)])
    assert torch.equal(m(ids), m2(ids))
    assert m.to_checkpoint().keys() == w.keys()
    with pytest.raises(KeyError):
        load_model(cfg, {k: v for k, v in w.items() if k != "l0.dwa"}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l0.shift": w["l0.shift"][:-1]}, torch.float32)
    core = EngineCore(EngineConfig(model=str(tmp_path), device="cpu"))      # no tokenizer files: bytes
    assert core.tokenizer.encode_raw("ab", add_special_tokens=False) == [97, 98]


def test_configurations_the_class_cannot_run_are_refused():
    for path, value in ((("type",), "other"), (("mixer", "rot", "dims"), 2), (("mlp", "kind"), "dense"),
                        (("mlp", "router", "top"), 9)):
        cfg = O.make_config(layers=1)
        d = cfg["layers"][0]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            MezilixConfig.from_dict(cfg)
    with pytest.raises(ValueError):
        architecture_of({"architecture": "Unknown"})
    assert architecture_of({"model_type": "llama"}).name == "Llama"


def test_features_of_the_llama_path_are_refused_with_a_reason():
    _, _, core = make()
    with pytest.raises(ValueError, match="LoRA"):
        core.load_adapters({"a": {}})
    cfg = EngineConfig(model="custom", tokenizer="byte", device="cpu")
    cfg.speculative.enabled = True
    eng = SOTAInferenceEngine(cfg, model=core.model, draft_model=core.model)
    assert eng.generate("ab", GenerationParams(max_tokens=2)).is_err()
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


def test_presets_and_registry():
    from trainscale_b200.models import is_preset
    from trainscale_b200.registry import MODEL_REGISTRY
    assert is_preset("mezilix-tiny") and is_preset("tiny") and not is_preset("nothing")
    assert MODEL_REGISTRY["mezilix"].architecture == "MezilixForCausalLM"
    a, b = build_model("mezilix-tiny", torch.float32, seed=5), build_model("mezilix-tiny", torch.float32, seed=5)
    assert torch.equal(a.head, b.head) and not isinstance(a, LlamaForCausalLM)
    spec = a.cache_spec()
    assert spec.has_state and spec.bytes_per_token(2) == 4 * 2 * 128


def test_cli_batch(capsys):
    from trainscale_b200.inference import main
    assert main(["batch", "--model", "mezilix-tiny", "--prompt", "hi", "--max-tokens", "3", "--temperature", "0"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["finish_reason"] in ("length", "stop")
