"""Kabulix through the engine on the CPU (PyTorch math of the ops): the cache, batching, scheduling and generation against the
plain statement of the design in kabulix_oracle.py."""
import copy
import json

import pytest
import torch

import kabulix_oracle as O
from trainscale_b200.hub import ModelSerializer, load_pretrained
from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, GenerationParams, SchedulerConfig, SOTAInferenceEngine
from trainscale_b200.inference.batch import HostBatch, StepEntry
from trainscale_b200.inference.trace import TraceRunner
from trainscale_b200.models import architecture_of
from trainscale_b200.models.kabulix import KabulixConfig, KabulixForCausalLM, build_model, load_model
from trainscale_b200.ops.masks import KeyMask

# unlike layers: every size and constant differs from layer to layer
MIXED = dict(width=40, types=("latent_attention", "attention", "attention_2", "attention", "latent_attention"), heads=[6, 4, 3, 2],
             kv_heads=[2, 4, 1, 2], dim=[12, 8, 10, 14], vdim=[6, 16, 10], window=[19, 5, 7, 11], keep=[2, 0, 5, 1], chunk=[7, 13, 6],
             rot=[8, 8, 4, 6], base=[500.0, 50.0, 3000.0], lheads=[3, 1, 2, 4, 5], ldim=[12, 8, 8, 6, 7], lrot=[6, 4, 4, 4, 8], lvdim=[10, 8, 8, 8, 5],
             rank=[20, 8, 8, 8, 13], lwindow=[13, 1, 1, 1, 6], mlps=("moe", "dense", "moe", None, "moe"), ff=[40, 17, 64],
             experts=[6, 8, 12, 4, 8], top=[2, 1, 3, 1, 4], groups=[3, 4, 3, 2, 8], keep_groups=[2, 2, 1, 1, 5], expert_ff=[20, 7, 33],
             shared_ff=[28, 16, 5])


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
def test_masks():
    for size, keep, chunked in ((1, 0, False), (5, 3, False), (5, 9, False), (4, 0, True), (1, 0, True), (100, 2, False)):
        m, n = KeyMask(size, keep, chunked), 23
        want = O.chunk_mask(n, size) if chunked else O.window_mask(n, size, keep)
        for p in range(n):
            assert m.positions(p) == want[p].nonzero().flatten().tolist()
            assert len(m.positions(p)) <= m.most(p + 1)


def test_prompt_context_lists_each_portions_keys_once():
    """Key rows of portions: the kept first positions and the window or chunk of the first query, in key order."""
    _, _, core = make(blocks=60)
    core.execute([StepEntry(0, tokens(21, 1), []), StepEntry(1, tokens(3, 2), [])])
    b = HostBatch(core.cache, [StepEntry(0, tokens(6, 3)), StepEntry(1, tokens(9, 4)), StepEntry(2, [5])]).to_device("cpu")
    pages = {s: core.cache.seqs[s].blocks for s in (0, 1)}
    for mask in (KeyMask(5), KeyMask(5, 2), KeyMask(5, 30), KeyMask(8, 0, True), KeyMask(100, 3)):
        keys = b.prompt_context(mask)
        want = []
        for seq, start, n in ((0, 21, 6), (1, 3, 9)):
            pos = sorted(set().union(*(mask.positions(start + i) for i in range(n))))
            want.append([pages[seq][j // 4] * 4 + j % 4 for j in pos])
        assert keys.slots.tolist() == want[0] + want[1]
        assert keys.cu_k.tolist() == [0, len(want[0]), len(want[0]) + len(want[1])] and keys.cu_q.tolist() == [0, 6, 15]


def test_yarn_frequencies():
    from trainscale_b200.models.kabulix import Rotation
    for dims, base, s in ((16, 500.0, O.SCALING), (8, 50.0, {"factor": 2.5, "original": 4000, "fast": 32.0, "slow": 1.0}),
                          (6, 10.0, {"factor": 4.0, "original": 9, "fast": 2.0, "slow": 0.01}), (4, 1e4, None)):
        r = {"dims": dims, "base": base} | ({"scaling": s} if s else {})
        rot = Rotation.from_dict(r)
        assert torch.allclose(rot.inv_freq().double(), O.frequencies(r), rtol=1e-6)
        assert rot.magnitude == O.magnitude(r)


def test_router_in_groups():
    from trainscale_b200.ops.moe import Router
    for E, top, count, keep in ((12, 3, 4, 2), (8, 4, 8, 5), (6, 2, 1, 1), (9, 1, 3, 3), (16, 8, 4, 2)):
        z = torch.randn(40, E + 3, generator=torch.Generator().manual_seed(E))
        w, idx = Router(E, top, True, count, keep).choose(z)
        want_idx, want_w = O.group_routing(z[:, :E].double(), top, count, keep)
        assert torch.equal(idx, want_idx) and torch.allclose(w.double(), want_w, atol=1e-6)
        assert all(len({int(e) // (E // count) for e in row}) <= keep for row in idx)


@pytest.mark.parametrize("ff", [1, 15, 16, 17, 48])
def test_packed_gate_and_up_rows(ff):
    from trainscale_b200.ops import grouped
    g = torch.Generator().manual_seed(ff)
    gate, up, x = torch.randn(ff, 6, generator=g), torch.randn(ff, 6, generator=g), torch.randn(5, 6, generator=g)
    packed = torch.zeros(2 * grouped.glu_width(ff), 6)
    parts = [grouped.GluRows(packed, ff, i) for i in range(2)]
    parts[0].copy_(gate), parts[1].copy_(up)
    assert torch.equal(parts[0].detach(), gate) and torch.equal(parts[1].detach(), up)
    for act, fn in ((grouped.ACT_SILU_GLU, torch.nn.functional.silu), (grouped.ACT_GELU_GLU, O.gelu_tanh)):
        y = grouped.activate(x @ packed.t(), act)
        assert torch.allclose(y[:, :ff], fn(x @ gate.t()) * (x @ up.t()), atol=1e-5) and (y[:, ff:] == 0).all()


# ---------------------------------------------------------------------------------------------- the model in the engine
def test_whole_prompt_matches_oracle_with_unlike_layers():
    cfg, w, core = make()
    ids = tokens(41, 1)
    got = core.execute([StepEntry(0, ids, list(range(41)))])
    close(got, oracle(w, cfg, ids))
    close(core.model(torch.tensor([ids]))[0], oracle(w, cfg, ids))


@pytest.mark.parametrize("over", [
    dict(types=("attention",)), dict(types=("attention_2",)), dict(types=("latent_attention",)), dict(mlps=(None,)), dict(mlps=("dense",)),
    dict(window=1, chunk=1, lwindow=1), dict(window=1000, chunk=1000, lwindow=1000), dict(keep=0), dict(keep=40), dict(keep=1, window=1),
    dict(width=33, vocab=301), dict(heads=1, kv_heads=1, lheads=1), dict(types=("attention",), rot=2, dim=7),
    dict(types=("attention",), rot=[12, 4], dim=[12, 4]), dict(scaling=None), dict(experts=4, groups=1, keep_groups=1, top=4),
    dict(experts=6, groups=6, keep_groups=6, top=1), dict(scale=[0.3, 1.0, 0.05])])
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


def test_batch_of_unequal_requests_and_reuse_of_pages():
    """Requests of different lengths advance by different amounts in one batch; finished ones give their pages to new ones
    (the pool holds only a few at a time)."""
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
    assert core.cache.alloc.num_free == 40
    for r, ids in reqs.items():
        close(torch.cat(got[r]), oracle(w, cfg, ids))


def test_want_nothing_still_advances():
    cfg, w, core = make()
    ids = tokens(12, 5)
    assert core.execute([StepEntry(0, ids[:7], [])]) is None
    close(core.execute([StepEntry(0, ids[7:], [4, 0])]), oracle(w, cfg, ids)[[11, 7]])


EDGES = [("attention", dict(window=w, keep=0), [w - 1], [w]) for w in (1, 4, 5, 8, 9)] + \
        [("latent_attention", dict(lwindow=w), [w - 1], [w]) for w in (1, 4, 5, 9)] + \
        [("attention_2", dict(chunk=c), [20 % c], [20 % c + 1]) for c in (1, 4, 7, 10, 20)] + \
        [("attention", dict(window=4, keep=k), [20, 21 - k], [20 - k]) for k in (1, 3, 8)]


@pytest.mark.parametrize("kind,over,seen,unseen", EDGES)
def test_edges_of_what_a_token_sees(kind, over, seen, unseen):
    """With one layer, tokens `seen` back from the last one (position 20) matter, those `unseen` back do not."""
    cfg, w, core = make(types=(kind,), mlps=("dense",), **over)
    n, base = 21, tokens(21, 6)
    for sizes in ([n], [n - 1, 1], [n - 2, 2], [5, 3, n - 8], [1]):
        def last(ids):
            y = run_portions(core, 0, ids, sizes)[-1]
            core.release(0)
            return y
        ref = last(base)
        for back in seen + unseen:
            ids = list(base)
            ids[20 - back] = (base[20 - back] + 1) % 300
            d = (last(ids) - ref).abs().max()
            assert d > 1e-3 if back in seen else d == 0, (sizes, back)


@pytest.mark.parametrize("kind,over", [("attention", dict(window=60, keep=0)), ("attention", dict(window=59, keep=0)), ("attention", dict(window=5, keep=5)),
                                       ("attention", dict(window=5, keep=4)), ("attention_2", dict(chunk=64)), ("attention_2", dict(chunk=60)),
                                       ("latent_attention", dict(lwindow=60)), ("latent_attention", dict(lwindow=59))])
def test_far_key_is_found_or_not(kind, over):
    """The last token's query is made to point at the key of the token at position 4, which takes most of the weight where it
    is seen: missing it shows at once, and so does seeing it when it is out of sight."""
    ids = tokens(64, 7)
    ids[4], ids[63] = 298, 299
    assert 298 not in ids[5:] + ids[:4] and 299 not in ids[:63]
    results = {}
    for point in (True, False):
        still = dict(base=1e30)                                    # all pairs but the first hardly turn
        cfg = O.make_config(types=(kind,), mlps=("dense",), heads=1, kv_heads=1, lheads=1, lrot=2, rot=2, scaling=None, **still, **over)
        w = O.make_weights(cfg, 0, 2.0)
        eps, p = cfg["norm"]["eps"], "l0.mix."
        x = O.norm1p(w["embed"][[298, 299]], w["l0.norm1"], eps)
        if point:
            if kind == "latent_attention":
                K, D = 20, 12
                c = O.rms(x[0] @ w[p + "dkv"][:K].t(), eps) * w[p + "dkv.norm"]
                key, rows = w[p + "uk"] @ c, slice(0, D)
            else:
                key, rows = w[p + "k"] @ x[0], slice(None)
            q = w[p + "q"][rows]
            w[p + "q"][rows] = (q + torch.outer(6 * key - q @ x[1], x[1]) / (x[1] @ x[1])).to(torch.bfloat16).float()
        core = EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cpu", cache=CacheConfig(block_size=4, num_gpu_blocks=64)),
                          model=load_model(cfg, w, torch.float32))
        want = oracle(w, cfg, ids)
        for i, sizes in enumerate(([64], [50, 2, 5, 7], [40], [61, 2, 1])):
            close(run_portions(core, i, ids, sizes), want)
            core.release(i)
        swapped = list(ids)
        swapped[4] = 17
        results[point] = (oracle(w, cfg, swapped)[-1] - want[-1]).abs().max()
    visible = 4 in {"attention": KeyMask(over.get("window", 1), over.get("keep", 0)), "attention_2": KeyMask(over.get("chunk", 1), 0, True),
                    "latent_attention": KeyMask(over.get("lwindow", 1))}[kind].positions(63)
    assert results[True] > 0.3 if visible else results[True] == 0


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
        "window": lambda c: mixer(c, 1)["mask"].update(size=mixer(c, 1)["mask"]["size"] + 1),
        "kept tokens": lambda c: mixer(c, 3)["mask"].update(keep_first=2),
        "chunk": lambda c: mixer(c, 2)["mask"].update(size=mixer(c, 2)["mask"]["size"] + 1),
        "latent window": lambda c: mixer(c, 0)["mask"].update(size=mixer(c, 0)["mask"]["size"] - 1),
        "scale": lambda c: mixer(c, 1).update(scale=mixer(c, 1)["scale"] * 1.05),
        "chunk scale": lambda c: mixer(c, 2).update(scale=mixer(c, 2)["scale"] * 1.05),
        "latent scale": lambda c: mixer(c, 0).update(scale=mixer(c, 0)["scale"] * 1.05),
        "base": lambda c: mixer(c, 1)["rot"].update(base=mixer(c, 1)["rot"]["base"] * 1.5),
        "rotated dimensions": lambda c: mixer(c, 1)["rot"].update(dims=mixer(c, 1)["rot"]["dims"] - 2),
        "stretch": lambda c: mixer(c, 0)["rot"]["scaling"].update(factor=3.5),
        "ramp": lambda c: mixer(c, 0)["rot"]["scaling"].update(original=600),
        "top": lambda c: c["layers"][0]["mlp"]["router"].update(top=3),
        "groups": lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3),
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


def test_prompts_share_prefixes():
    """A sequence has no state besides its pages, so a second prompt takes over the pages of a common beginning."""
    cfg, w, core = make(prefix=True)
    common = tokens(24, 3)
    for tail in ([], tokens(9, 4), tokens(13, 5)):
        before = core.cache.prefix_hits
        r = core.add_request(common + tail, GenerationParams(max_tokens=4, temperature=0.0, ignore_eos=True))
        while core.has_unfinished():
            core.step()
        assert r.output_ids == O.greedy(w, cfg, common + tail, 4)
        assert core.cache.prefix_hits - before == (24 if tail else 0)


def test_checkpoint_directory_round_trip(tmp_path):
    """config.json picks the class; weights written by `to_checkpoint` load again; a wrong checkpoint is refused."""
    cfg = O.make_config(**MIXED)
    w = O.make_weights(cfg, 3)
    m = load_model(cfg, w, torch.float32)
    (tmp_path / "config.json").write_text(json.dumps(m.config.to_dict()))
    ModelSerializer().save(m.to_checkpoint(), tmp_path)
    m2 = load_pretrained(tmp_path, dtype=torch.float32)
    assert isinstance(m2, KabulixForCausalLM) and m2.config == m.config == KabulixConfig.from_dict(cfg)
    ids = torch.tensor([tokens(9, 4)])
    assert torch.equal(m(ids), m2(ids))
    sd = m.to_checkpoint()
    assert sd.keys() == w.keys() and all(torch.equal(sd[k].float(), w[k]) for k in w)
    with pytest.raises(KeyError):
        load_model(cfg, {k: v for k, v in w.items() if k != "l0.mix.g"}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l1.mix.o": w["l1.mix.o"][:-1]}, torch.float32)
    with pytest.raises(ValueError):
        load_model(cfg, {**w, "l0.mlp.e1.up": w["l0.mlp.e1.up"][:-1]}, torch.float32)
    core = EngineCore(EngineConfig(model=str(tmp_path), device="cpu"))      # no tokenizer files: bytes
    assert core.tokenizer.encode_raw("ab", add_special_tokens=False) == [97, 98]


def test_configurations_the_class_cannot_run_are_refused():
    cases = [(0, ("type",), "other"), (0, ("mixer", "rot", "dims"), 3), (0, ("mixer", "rot", "dims"), 400), (0, ("mixer", "kv_heads"), 3),
             (0, ("mixer", "mask", "size"), 0), (0, ("mixer", "vdim"), 5), (0, ("mlp", "kind"), "other"), (1, ("mixer", "kv_heads"), 3),
             (1, ("mlp", "router", "top"), 5), (1, ("mlp", "router", "groups", "count"), 4), (1, ("mlp", "router", "groups", "keep"), 4),
             (2, ("mixer", "rot", "dims"), 6)]
    for layer, path, value in cases:
        cfg = O.make_config()
        d = cfg["layers"][layer]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            KabulixConfig.from_dict(cfg)
    assert architecture_of({"architecture": "Kabulix"}).name == "Kabulix"


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
    assert is_preset("kabulix-tiny") and is_preset("kabulix-3b")
    assert MODEL_REGISTRY["kabulix"].architecture == "KabulixForCausalLM"
    a, b = build_model("kabulix-tiny", torch.float32, seed=5), build_model("kabulix-tiny", torch.float32, seed=5)
    assert all(torch.equal(x, y) for x, y in zip(a.parameters(), b.parameters()))
    assert torch.isfinite(a(torch.tensor([tokens(20, 1)]))).all()
    spec = a.cache_spec()
    assert not spec.has_state and spec.bytes_per_token(2) == 2 * (3 * 2 * 128 + 128)


def test_cli_batch(capsys):
    from trainscale_b200.inference import main
    assert main(["batch", "--model", "kabulix-tiny", "--prompt", "hi", "--max-tokens", "3", "--temperature", "0"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["finish_reason"] in ("length", "stop")
