"""The Nesisun decoder through the engine's host side, without a GPU: configuration, registry, weight names, shared
weights, the state of the pair embedding, and -- with the plain PyTorch operator set of tests/torch_ops.py in place of
the CUDA kernels -- every way of cutting requests into steps against the whole-sequence plain implementation of
tests/plain_nesisun.py."""
import copy
import json

import pytest
import torch

import plain_nesisun as plain
import traces
from conftest import random_tokens
from torch_ops import TorchOps
from pytriton_llama_b200.config import ConfigError, EngineConfig, NesisunConfig, resolve_architecture
from pytriton_llama_b200.engine.engine import Engine, StepEntry
from pytriton_llama_b200.models.decoder import DecoderModel
from pytriton_llama_b200.parts.base import Runtime

TOL = 2e-4      # float32 operators against float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, cfg=None, seed=5, weights=None):
        if name not in made:
            folder = tmp_path_factory.mktemp(f"nesisun_{name}")
            plain.write_model(folder, cfg or plain.TINY[name], seed, weights=weights)
            made[name] = folder
        return made[name]
    return get


def _engine(folder, page, pages, max_seq_len=256, slots=4):
    cfg = EngineConfig(dtype="float32", page_size=page, max_gpu_num_blocks=pages, max_seq_len=max_seq_len, max_num_seqs=slots)
    return Engine(folder, cfg, device="cpu", ops=TorchOps())


def _reference(folder, seqs):
    from pytriton_llama_b200.weights import read_folder
    cfg = json.loads((folder / "config.json").read_text())
    W = read_folder(folder)
    return {r: plain.forward(cfg, W, s) for r, s in seqs.items()}


def _seqs(lengths, vocab, seed):
    return {f"r{i}": random_tokens(n, vocab, seed * 100 + i) for i, n in enumerate(lengths)}


def _close(got, want, tol=TOL):
    err = (got.double() - want).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), err


def _model(cfg):
    arch = resolve_architecture(cfg)
    return DecoderModel(arch.spec_from_config(arch.config_from_dict(cfg)), Runtime(torch.device("cpu"), torch.float32, None))


# ---------------------------------------------------------------------------- configuration and names
def test_config_reads_every_key_and_round_trips():
    cfg = NesisunConfig.from_dict(plain.TINY_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale) == (97, 48, 1e-5, 0.6)
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (61, 13, 5)
    assert [L.weights_of for L in cfg.layers] == [None, None, 1, None, 0]
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.window, a.keep_first, a.rot.dims, a.rot.base) == (4, 2, 16, 0.3, 11, 6, 8, 1000.0)
    assert cfg.layers[0].mlp.ff == 40 and cfg.layers[3].mlp is None
    m = cfg.layers[1].mlp
    assert (m.ff, m.limit, m.experts, m.identity, m.top, m.scale) == (24, 0.8, 5, 2, 3, 1.7)
    for other in plain.TINY.values():
        c = NesisunConfig.from_dict(other)
        assert NesisunConfig.from_dict(c.to_dict()) == c
    c = NesisunConfig.from_dict(plain.TINY_C)
    assert c.layers[0].mixer.window == 0 and c.layers[0].mixer.rot is None and c.layers[1].mlp.identity == 1
    assert resolve_architecture(plain.TINY_A).name == "Nesisun"


@pytest.mark.parametrize("change", [
    lambda c: c.pop("vocab"), lambda c: c["layers"][0].update(type="conv"), lambda c: c["layers"][0]["mixer"].update(heads=5),
    lambda c: c["layers"][0]["mixer"].update(vdim=24), lambda c: c["layers"][0]["mlp"].update(kind="gated"), lambda c: c["norm"].update(eps=0),
    lambda c: c.update(layers=[]), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=8), lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0),
    lambda c: c["layers"][2].update(weights_of=2), lambda c: c["layers"][2].update(weights_of=9), lambda c: c["layers"][2].update(weights_of=0),
    lambda c: c["embedding"]["bigram"].update(buckets=0), lambda c: c["embedding"]["bigram"].pop("mul_cur"),
    lambda c: c["layers"][4].update(weights_of=2),
])
def test_config_names_what_is_wrong(change):
    bad = copy.deepcopy(plain.TINY_A)
    change(bad)
    with pytest.raises(ConfigError):
        NesisunConfig.from_dict(bad)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_model_expects_the_checkpoint_names_and_shapes(name):
    assert {k: tuple(v.shape) for k, v in _model(plain.TINY[name]).expected_tensors().items()} == plain.tensor_shapes(plain.TINY[name])


def test_layers_with_shared_weights_are_runs_of_one_block_with_caches_of_their_own():
    model = _model(plain.TINY_A)
    assert len(model.blocks) == 3 and [(e.layer, e.cache) for e in model.spec.run_order] == [(0, 0), (1, 1), (1, 2), (2, 3), (0, 4)]
    needs = model.cache_entries()
    assert sorted(needs) == [model.EMBEDDING_ENTRY, 0, 1, 2, 3, 4]
    assert (needs[1].kind, needs[1].window, needs[1].keep_first, needs[1].kv_heads, needs[1].head_dim) == ("window", 7, 3, 2, 24)
    assert needs[1] == needs[2] and needs[0] == needs[4] and needs[0] != needs[1]
    assert needs[model.EMBEDDING_ENTRY].kind == "none" and needs[model.EMBEDDING_ENTRY].states[0][2] == torch.int32
    assert _model(plain.TINY_C).cache_entries()[0].kind == "full"


def test_random_weights_mode_writes_a_model_that_runs(tmp_path):
    from pytriton_llama_b200.weights import read_folder, write_random_model
    folder = write_random_model(tmp_path / "m", plain.TINY_A, seed=3, dtype=torch.float32, std=0.2)
    cfg = json.loads((folder / "config.json").read_text())
    W = read_folder(folder)
    toks = random_tokens(30, 97, 2)
    got = traces.replay(_engine(folder, 8, 24), traces.portions({"x": toks}))["x"]
    _close(got, plain.forward(cfg, W, toks))


# ---------------------------------------------------------------------------- every cut equals the whole sequence
@pytest.mark.parametrize("name,page", [("A", 4), ("A", 16), ("B", 8), ("C", 4)])
def test_every_cut_of_the_requests_matches_the_plain_implementation(folders, name, page):
    folder = folders(name)
    vocab = plain.TINY[name]["vocab"]
    seqs = _seqs([41, 1, 23, 58, 9], vocab, 21)
    want = _reference(folder, seqs)
    for steps in (traces.whole(seqs), traces.prefill_then_decode(seqs, 12), traces.portions(seqs), traces.mixed(seqs)):
        eng = _engine(folder, page, max(40, traces.max_live_tokens(steps, page) // page + 8))
        got = traces.replay(eng, steps)
        for rid in seqs:
            _close(got[rid], want[rid][traces.wanted_positions(steps, rid)])


def test_six_requests_through_three_slots_and_few_pages_reuse_what_was_freed(folders):
    folder = folders("A")
    seqs = _seqs([30, 17, 44, 5, 26, 38], 97, 4)
    want = _reference(folder, seqs)
    steps = traces.mixed(seqs, live=3)
    pages = traces.max_live_tokens(steps, 4) // 4 + 2
    eng = _engine(folder, 4, pages, slots=3)
    got = traces.replay(eng, steps)
    for rid in seqs:
        _close(got[rid], want[rid][traces.wanted_positions(steps, rid)])
    assert eng.cache.free_slots() == 3
    assert all(eng.cache.free_pages(g) == grp.pool.num_pages for g, grp in enumerate(eng.cache.groups) if grp.paged)


def test_an_unequal_batch_equals_each_request_alone(folders):
    folder = folders("B")
    seqs = _seqs([33, 2, 14], 70, 8)
    eng = _engine(folder, 8, 40)
    together = eng.step([StepEntry(r, s, list(range(len(s)))) for r, s in seqs.items()]).logits
    eng.finish_all()
    at = 0
    for r, s in seqs.items():
        alone = eng.step([StepEntry(r, s, list(range(len(s))))]).logits
        eng.finish(r)
        assert torch.allclose(together[at:at + len(s)], alone, atol=1e-5, rtol=1e-5)
        at += len(s)


def test_long_decoding_token_by_token_with_pages_that_come_back(folders):
    folder = folders("A")
    toks = random_tokens(150, 97, 13)
    want = _reference(folder, {"x": toks})["x"]
    eng = _engine(folder, 4, 8)           # 8 pages of 4 for 150 tokens: the kept positions' pages and the window's, no more
    rows = [eng.step([StepEntry("x", [t], [0])]).logits[0] for t in toks]
    _close(torch.stack(rows), want)
    eng.cache.check_invariants()


# ---------------------------------------------------------------------------- the pair embedding and its state
def test_rows_of_the_pair_table():
    assert plain.bigram_rows([4], 7, 3, 2) == [7] and plain.bigram_rows([], 7, 3, 2) == []
    assert plain.bigram_rows([4, 5, 0], 7, 3, 2) == [7, (4 * 3 + 5 * 2) % 7, (5 * 3) % 7]


def test_the_token_before_a_portion_comes_from_the_requests_own_state(folders):
    """A pair table with one outstanding row: the pair (8, 9).  Its token pairs straddle a cut, another request's tokens run
    between the two steps, and a slot's next owner starts with token 9 after an owner that ended in 8."""
    cfg = plain.config(41, 32, [plain.layer(plain.attention(2, 1, 8, 0.3, size=6, keep=2), plain.dense(16))], buckets=1681, mul_prev=41, mul_cur=1)
    W = plain.random_weights(cfg, 4)
    W["bigram"] *= 0.1
    W["bigram"][8 * 41 + 9] = 5.0
    folder = folders("pairs", cfg, weights=W)
    a, b, c = [3, 7, 8, 9, 9], [20, 8, 21], [9, 8, 9]
    want = {k: plain.forward(cfg, W, s) for k, s in (("a", a), ("b", b), ("c", c))}
    eng = _engine(folder, 4, 20, slots=2)
    _close(eng.step([StepEntry("a", a[:3], [2]), StepEntry("b", b[:1], [0])]).logits, torch.stack([want["a"][2], want["b"][0]]))
    _close(eng.step([StepEntry("b", b[1:2], [0])]).logits, want["b"][1:2])
    out = eng.step([StepEntry("b", b[2:], [0]), StepEntry("a", a[3:], [0, 1])]).logits
    _close(out, torch.cat([want["b"][2:], want["a"][3:]]))
    eng.finish("a")
    eng.finish("b")
    eng.step([StepEntry("d", [5, 8], [])])
    eng.finish("d")
    _close(eng.step([StepEntry("c", c, [0, 1, 2])]).logits, want["c"])           # in the slot whose last token was 8
    swapped = dict(W)
    swapped["bigram"] = W["bigram"].clone()
    swapped["bigram"][8 * 41 + 9] = 0.0
    assert (plain.forward(cfg, swapped, a)[3] - want["a"][3]).abs().max() > 0.1


# ---------------------------------------------------------------------------- each mechanism alone
def _one_layer(mixer, mlp=None, width=32, **kw):
    return plain.config(41, width, [plain.layer(mixer, mlp)], **kw)


_ATT = plain.attention(2, 1, 8, 0.4, size=6, keep=2, dims=4)
ALONE = {
    "window_and_kept": _one_layer(plain.attention(4, 2, 8, 0.4, size=6, keep=3, dims=8, base=20.0)),
    "kept_beyond_the_window": _one_layer(plain.attention(3, 3, 12, 0.3, size=4, keep=13, dims=6)),
    "window_alone": _one_layer(plain.attention(2, 2, 8, 0.4, size=5, keep=0, dims=8)),
    "window_one": _one_layer(plain.attention(2, 1, 8, 0.4, size=1, keep=1, dims=2)),
    "everything_seen_part_turned": _one_layer(plain.attention(6, 2, 16, 0.2, dims=10, base=300.0)),
    "nothing_turned": _one_layer(plain.attention(2, 1, 8, 0.4, size=6, keep=2)),
    "odd_head": _one_layer(plain.attention(3, 1, 7, 0.4, size=6, keep=2, dims=4)),
    "dense": _one_layer(_ATT, plain.dense(24)),
    "dense_odd": _one_layer(_ATT, plain.dense(13), width=27),
    "experts_top1": _one_layer(_ATT, plain.moe(12, 6, 1, limit=0.5)),
    "experts_and_identity": _one_layer(_ATT, plain.moe(12, 4, 3, identity=3, scale=2.2, limit=0.7)),
    "one_expert_many_identity": _one_layer(_ATT, plain.moe(8, 1, 2, identity=5, scale=0.5)),
    "all_chosen": _one_layer(_ATT, plain.moe(8, 3, 5, identity=2, scale=1.0, limit=3.0)),
    "no_pairs": _one_layer(_ATT, plain.dense(16), buckets=0),
    "no_pairs_no_scale": _one_layer(_ATT, plain.dense(16), buckets=0, scale=1.0),
    "run_three_times": plain.config(41, 32, [plain.layer(_ATT, plain.moe(12, 4, 2, identity=1)), plain.layer(_ATT, plain.moe(12, 4, 2, identity=1), 0),
                                             plain.layer(_ATT, plain.moe(12, 4, 2, identity=1), 0)]),
    "used_before_it_runs": plain.config(41, 32, [plain.layer(_ATT, plain.dense(12), 1), plain.layer(_ATT, plain.dense(12))]),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(folders, name):
    folder = folders("alone_" + name, ALONE[name], seed=3)
    seqs = _seqs([27, 12], 41, 6)
    want = _reference(folder, seqs)
    for steps in (traces.whole(seqs), traces.portions(seqs, sizes=(3, 2, 9, 2))):
        got = traces.replay(_engine(folder, 4, 30), steps)
        for rid in seqs:
            _close(got[rid], want[rid][traces.wanted_positions(steps, rid)])


@pytest.mark.parametrize("what,change", [
    ("sink", lambda W: W["l0.mix.sink"].fill_(-30.0)), ("sink's share", lambda W: W["l0.mix.sink"].add_(0.5)),
    ("key bias", lambda W: W["l0.mix.k.b"].zero_()), ("query bias", lambda W: W["l0.mix.q.b"].zero_()),
    ("correction", lambda W: W["l0.mlp.correction"].zero_()), ("pair table", lambda W: W["bigram"].zero_()),
    ("last row of the pair table", lambda W: W["bigram"][-1].zero_()),
])
def test_leaving_a_mechanism_out_shows_in_the_plain_implementation(what, change):
    """(so that agreement with it says something about the mechanism)"""
    cfg = _one_layer(_ATT, plain.moe(12, 4, 3, identity=3, scale=2.2, limit=0.7))
    W = plain.random_weights(cfg, 3)
    toks = random_tokens(27, 41, 600)
    want = plain.forward(cfg, W, toks)
    other = {k: v.clone() for k, v in W.items()}
    change(other)
    assert (plain.forward(cfg, other, toks) - want).abs().max() > 100 * TOL


def test_limits_identity_and_weight_scale_show_in_the_plain_implementation():
    base = plain.moe(12, 4, 3, identity=3, scale=2.2, limit=0.7)
    cfg = _one_layer(_ATT, base)
    W = plain.random_weights(cfg, 3)
    toks = random_tokens(27, 41, 600)
    want = plain.forward(cfg, W, toks)
    for part, key, value in (("expert", "limit", 5.0), ("router", "scale", 1.0), ("router", "top", 4)):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mlp"][part][key] = value
        assert (plain.forward(other, W, toks) - want).abs().max() > 0.05, (part, key)
    chosen, w = plain.route(torch.tensor([0.5, 0.3, 0.2], dtype=torch.float64), torch.tensor([-0.4, 0.0, 0.05], dtype=torch.float64), 2, 3.0)
    assert sorted(chosen.tolist()) == [1, 2] and float(w.sum()) == pytest.approx(3.0)
    assert dict(zip(chosen.tolist(), w.tolist()))[1] == pytest.approx(3.0 * 0.6)


# ---------------------------------------------------------------------------- edges that random weights would hide
def _spiked(cfg, seed):
    """Weights such that the key of token 1 dominates the scores of every query that sees it: its embedding lies along
    stream entry 0, queries and keys read entry 0 into entry 6 of every head (which the tests do not turn) and nothing
    else, and the pair table is nought."""
    W = plain.random_weights(cfg, seed)
    m = cfg["layers"][0]["mixer"]
    d = m["dim"]
    W["embed"][:, 0] = 0.8
    W["embed"][1] = 0.0
    W["embed"][1, 0] = 6.0
    W["bigram"].zero_()
    W["l0.norm1"] = torch.ones_like(W["l0.norm1"])
    for name, heads in (("q", m["heads"]), ("k", m["kv_heads"])):
        w = torch.zeros_like(W["l0.mix." + name])
        for h in range(heads):
            w[h * d + 6, 0] = 2.0
        W["l0.mix." + name] = w
        W["l0.mix." + name + ".b"].zero_()
    return W


def _edge_tokens(n, spike):
    toks = [2 + (7 * i) % 30 for i in range(n)]
    toks[spike] = 1
    return toks


@pytest.mark.parametrize("window,keep,page", [(5, 3, 4), (8, 0, 4), (7, 5, 16), (16, 4, 4)])
def test_a_key_just_inside_and_just_outside_the_window_in_prompt_and_decoding(folders, window, keep, page):
    cfg = _one_layer(plain.attention(2, 1, 8, 1.0, size=window, keep=keep, dims=4), None)
    spike = 9
    W = _spiked(cfg, 4)
    n = spike + window + 14
    toks = _edge_tokens(n, spike)
    want = plain.forward(cfg, W, toks)
    for delta in (-1, 1):           # a window that is one off shows at the edge by far more than the tolerance
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = window + delta
        edge = spike + window - 1 + (1 if delta > 0 else 0)
        assert (plain.forward(other, W, toks)[edge] - want[edge]).abs().max() > 50 * TOL * want.abs().max(), delta
    folder = folders(f"edge_{window}_{keep}", cfg, weights=W)
    for steps in (traces.whole({"x": toks}), traces.prefill_then_decode({"x": toks}, n - spike - 2),
                  traces.portions({"x": toks}, sizes=(2, 3, 2, 5))):
        got = traces.replay(_engine(folder, page, 20), steps)["x"]
        _close(got, want[traces.wanted_positions(steps, "x")])


@pytest.mark.parametrize("window,keep,page", [(4, 6, 4), (3, 8, 4), (6, 5, 16), (12, 2, 4)])
@pytest.mark.parametrize("inside", [True, False])
def test_the_last_kept_position_is_seen_for_ever_and_the_next_is_not(folders, window, keep, page, inside):
    cfg = _one_layer(plain.attention(2, 1, 8, 1.0, size=window, keep=keep, dims=4), None)
    spike = keep - 1 if inside else keep
    W = _spiked(cfg, 4)
    n = keep + window + 22
    toks = _edge_tokens(n, spike)
    want = plain.forward(cfg, W, toks)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"]["keep_first"] = keep + (-1 if inside else 1)
    assert (plain.forward(other, W, toks)[-1] - want[-1]).abs().max() > 50 * TOL * want.abs().max()
    folder = folders(f"kept_{window}_{keep}_{inside}", cfg, weights=W)
    for steps in (traces.whole({"x": toks}), traces.prefill_then_decode({"x": toks}, 20),
                  traces.portions({"x": toks}, sizes=(2, 3, 2, 5))):
        got = traces.replay(_engine(folder, page, 14), steps)["x"]
        _close(got, want[traces.wanted_positions(steps, "x")])


def test_a_kept_key_and_its_own_rotation_hundreds_of_tokens_later(folders):
    """The kept positions' keys carry the rotation of where they are; a decoded token far out meets them at that distance."""
    cfg = _one_layer(plain.attention(2, 1, 8, 1.0, size=10, keep=4, dims=8, base=200.0), None)
    W = plain.random_weights(cfg, 8)
    toks = random_tokens(400, 41, 5)
    want = plain.forward(cfg, W, toks)
    swapped = [toks[1], toks[0]] + toks[2:]
    assert (plain.forward(cfg, W, swapped)[-1] - want[-1]).abs().max() > 20 * TOL
    folder = folders("far", cfg, weights=W)
    steps = traces.portions({"x": toks[:370]}, sizes=(32, 17, 64, 2))
    steps[-1]["end"] = []
    steps += [{"step": len(steps) + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks[370:])]
    eng = _engine(folder, 4, 24, max_seq_len=512)          # 24 pages of 4: what the window has passed must come back
    got = traces.replay(eng, steps)["x"]
    _close(got, want[traces.wanted_positions(steps, "x")])


# ---------------------------------------------------------------------------- generation through the public entry point
@pytest.mark.parametrize("overlap", [False, True])
def test_greedy_generation_through_the_scheduler_matches_the_plain_argmax(folders, overlap):
    from pytriton_llama_b200 import LLM, SamplingParams
    from pytriton_llama_b200.weights import read_folder
    folder = folders("A")
    W = read_folder(folder)
    prompts = list(_seqs([9, 21, 3, 1], 97, 17).values())
    llm = LLM(folder, EngineConfig(dtype="float32", page_size=4, max_gpu_num_blocks=40, max_seq_len=64, max_num_seqs=2,
                                   max_batched_tokens=8, compiled_model=False, overlap_steps=overlap), device="cpu", ops=TorchOps())
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_gen_len=7))
    for p, out in zip(prompts, got):
        logits = plain.forward(plain.TINY_A, W, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert row[tok] >= row.max() - 1e-4, (i, tok, int(row.argmax()))


def test_generation_that_runs_out_of_pages_starts_a_request_over(folders):
    """Requests that are set back begin again at position 0, with the last row of the pair table and no token before it."""
    from pytriton_llama_b200 import LLM, SamplingParams
    from pytriton_llama_b200.weights import read_folder
    cfg = _one_layer(plain.attention(2, 1, 8, 0.4, dims=4), plain.dense(16))
    folder = folders("preempt", cfg, seed=11)
    W = read_folder(folder)
    prompts = list(_seqs([12, 11, 13], 41, 31).values())
    llm = LLM(folder, EngineConfig(dtype="float32", page_size=4, max_gpu_num_blocks=11, max_seq_len=40, max_num_seqs=3,
                                   max_batched_tokens=16, compiled_model=False), device="cpu", ops=TorchOps())
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_gen_len=10))
    for p, out in zip(prompts, got):
        assert len(out) == 10
        logits = plain.forward(cfg, W, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert row[tok] >= row.max() - 1e-4, (i, tok, int(row.argmax()))
