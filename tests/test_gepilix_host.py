"""The Gepilix decoder through the engine's host side, without a GPU: configuration, registry, weight names, cache needs,
and -- with the plain PyTorch operator set of tests/torch_ops.py in place of the CUDA kernels -- every way of cutting
requests into steps against the whole-sequence plain implementation of tests/plain_gepilix.py."""
import copy
import json
import math

import pytest
import torch

import plain_gepilix as plain
import traces
from conftest import random_tokens
from torch_ops import TorchOps
from pytriton_llama_b200.config import ConfigError, EngineConfig, GepilixConfig, resolve_architecture
from pytriton_llama_b200.engine.engine import Engine, StepEntry
from pytriton_llama_b200.models.decoder import DecoderModel
from pytriton_llama_b200.parts.base import PartSpec, Runtime, build_part

TOL = 2e-4      # float32 operators against float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, cfg=None, seed=5, weights=None):
        if name not in made:
            folder = tmp_path_factory.mktemp(f"gepilix_{name}")
            plain.write_model(folder, cfg or plain.TINY[name], seed, weights=weights)
            made[name] = folder
        return made[name]
    return get


def _engine(folder, page, pages, max_seq_len=256, slots=4):
    cfg = EngineConfig(dtype="float32", page_size=page, max_gpu_num_blocks=pages, max_seq_len=max_seq_len, max_num_seqs=slots)
    return Engine(folder, cfg, device="cpu", ops=TorchOps())


def _model(cfg):
    arch = resolve_architecture(cfg)
    return DecoderModel(arch.spec_from_config(arch.config_from_dict(cfg)), Runtime(torch.device("cpu"), torch.float32, None))


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


# ---------------------------------------------------------------------------- configuration and names
def test_config_reads_every_key_and_round_trips():
    cfg = GepilixConfig.from_dict(plain.TINY_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (97, 48, 1e-5)
    assert [L.type for L in cfg.layers] == ["parallel", "wkv", "parallel_2", "parallel"] and cfg.layers[3].mlp is None
    a = cfg.layers[0].mixer.left
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.size, a.rot) == (4, 2, 16, 24, 0.3, 12.0, 11, None)
    u = cfg.layers[0].mixer.right
    assert (u.width, u.blocks, u.conv) == (36, 3, 3)
    assert (cfg.layers[1].mixer.heads, cfg.layers[1].mixer.dim, cfg.layers[1].mlp.ff) == (3, 12, 40)
    m = cfg.layers[2].mixer
    assert (m.left_scale, m.right_scale) == (0.8, 1.3)
    r = m.left.rot
    assert (r.dims, r.base, r.factor, r.low, r.high, r.original) == (12, 100.0, 3.0, 0.5, 2.0, 40.0)
    s = m.right
    assert (s.heads, s.vdim, s.state, s.groups, s.norm_groups, s.conv) == (6, 8, 12, 3, 2, 5)
    e = cfg.layers[0].mlp
    assert (e.ff, e.experts, e.top, e.shared_ff, cfg.layers[2].mlp.shared_ff) == (24, 6, 2, 16, 0)
    for other in plain.TINY.values():
        c = GepilixConfig.from_dict(other)
        assert GepilixConfig.from_dict(c.to_dict()) == c
    assert resolve_architecture(plain.TINY_A).name == "Gepilix"


@pytest.mark.parametrize("change", [
    lambda c: c.pop("vocab"), lambda c: c["layers"][0].update(type="conv"), lambda c: c["norm"].update(eps=0), lambda c: c.update(layers=[]),
    lambda c: c["layers"][0]["mixer"]["left"].update(heads=5), lambda c: c["layers"][0]["mixer"]["left"].pop("softcap"),
    lambda c: c["layers"][0]["mixer"]["left"].update(softcap=0), lambda c: c["layers"][0]["mixer"]["left"].pop("mask"),
    lambda c: c["layers"][0]["mixer"]["left"].update(rot={"dims": 8, "base": 10.0}), lambda c: c["layers"][0]["mixer"]["right"].update(blocks=5),
    lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=7), lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=18),
    lambda c: c["layers"][2]["mixer"]["left"]["rot"]["scaling"].pop("high"), lambda c: c["layers"][2]["mixer"]["right"].update(groups=4),
    lambda c: c["layers"][2]["mixer"]["right"].update(norm_groups=5), lambda c: c["layers"][2]["mixer"].pop("right_scale"),
    lambda c: c["layers"][1]["mixer"].pop("dim"), lambda c: c["layers"][1]["mlp"].update(kind="glu"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7), lambda c: c["layers"][0]["mlp"].pop("expert"),
])
def test_config_names_what_is_wrong(change):
    bad = copy.deepcopy(plain.TINY_A)
    change(bad)
    with pytest.raises(ConfigError):
        GepilixConfig.from_dict(bad)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_model_expects_the_checkpoint_names_and_shapes(name):
    got = {k: tuple(abs(n) for n in v.shape) for k, v in _model(plain.TINY[name]).expected_tensors().items()}
    assert got == plain.tensor_shapes(plain.TINY[name], rank=16)


def test_a_checkpoint_brings_its_own_inner_size_of_the_decay(tmp_path):
    cfg = plain.TINY_C
    W = plain.write_model(tmp_path, cfg, 3, weights=plain.random_weights(cfg, 3, rank=5))
    toks = random_tokens(21, 50, 1)
    _close(traces.replay(_engine(tmp_path, 8, 24), traces.portions({"x": toks}))["x"], plain.forward(cfg, W, toks))


def test_cache_needs_of_the_layers():
    needs = _model(plain.TINY_A).cache_entries()
    assert (needs[0].kind, needs[0].window, needs[0].kv_heads, needs[0].head_dim, needs[0].v_dim) == ("chunk", 11, 2, 16, 24)
    assert needs[0].states == (("right.conv", (2, 36)), ("right.S", (36,)))
    assert (needs[1].kind, needs[1].states) == ("none", (("last", (48,)), ("S", (3, 12, 12))))
    assert (needs[2].kind, needs[2].window) == ("window", 9)
    assert needs[2].states == (("right.conv", (4, 48 + 2 * 3 * 12)), ("right.S", (6, 12, 8)))
    assert _model(plain.TINY_B).cache_entries()[3].states[0] == ("right.conv", (1, 32 + 2 * 4 * 16))       # one tap keeps nothing, in one row


def test_random_weights_mode_writes_a_model_that_runs(tmp_path):
    from pytriton_llama_b200.weights import read_folder, write_random_model
    folder = write_random_model(tmp_path / "m", plain.TINY_A, seed=3, dtype=torch.float32, std=0.2)
    cfg = json.loads((folder / "config.json").read_text())
    W = read_folder(folder)
    assert W["final.norm.alpha"].shape == ()
    toks = random_tokens(30, 97, 2)
    got = traces.replay(_engine(folder, 8, 24), traces.portions({"x": toks}))["x"]
    _close(got, plain.forward(cfg, W, toks))


def test_a_norm_made_ahead_of_time_is_taken_by_its_own_reader_only():
    from pytriton_llama_b200.parts.base import NormedInput, ScaledOutput
    rt = Runtime(torch.device("cpu"), torch.float32, TorchOps())
    g = torch.Generator().manual_seed(1)
    norms = []
    for _ in range(2):
        n = build_part("norm", PartSpec("tanh_norm", {"width": 6}, {}), rt)
        n.load({"weight": torch.randn(6, generator=g), "bias": torch.randn(6, generator=g), "alpha": torch.tensor(0.7)})
        norms.append(n)
    res, y = torch.randn(4, 6, generator=g), torch.randn(4, 6, generator=g)
    assert torch.equal(norms[0].forward(NormedInput(y, norms[0].weight), res)[0], y)
    other, kept = norms[1].forward(NormedInput(y, norms[0].weight), res.clone())
    assert torch.allclose(other, torch.tanh(0.7 * res) * norms[1].weight + norms[1].bias) and torch.equal(kept, res)
    scale = torch.randn(6, generator=g)
    rows = torch.tensor([3, 1], dtype=torch.int32)
    picked, none = norms[0].forward(ScaledOutput(y, scale), res, rows=rows)
    want = torch.tanh(0.7 * (res + scale * y)) * norms[0].weight + norms[0].bias
    assert none is None and torch.allclose(picked, want[[3, 1]], atol=1e-6)


def test_scaled_frequencies_below_between_and_above_the_bounds():
    from pytriton_llama_b200.parts.rope import rope_frequencies64, rope_inverse_frequencies
    s = {"rope_type": "llama3", "factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 3.0, "original_max_position_embeddings": 100}
    rot = plain.rotation(16, 1000.0, (4.0, 1.0, 3.0, 100))
    f64 = rope_frequencies64(1000.0, s, 16)
    assert torch.allclose(f64, plain.pair_frequencies(rot), rtol=1e-14)
    assert torch.allclose(f64.float(), rope_inverse_frequencies(16, 1000.0, s), rtol=3e-6)
    plainly = 1000.0 ** (-torch.arange(8, dtype=torch.float64) / 8)
    turns = 100 * plainly / (2 * math.pi)
    assert (turns > 3).any() and (turns < 1).any() and ((turns > 1) & (turns < 3)).any()
    assert torch.equal(f64[turns > 3], plainly[turns > 3]) and torch.allclose(f64[turns < 1], plainly[turns < 1] / 4)


# ---------------------------------------------------------------------------- every cut equals the whole sequence
@pytest.mark.parametrize("name,page", [("A", 4), ("A", 16), ("B", 8), ("C", 4)])
def test_every_cut_of_the_requests_matches_the_plain_implementation(folders, name, page):
    folder = folders(name)
    seqs = _seqs([41, 1, 23, 58, 9], plain.TINY[name]["vocab"], 21)
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
    eng.cache.check_invariants()


def test_a_state_slot_that_is_taken_again_starts_from_zero(folders):
    """One slot: a request of one token, then of many, in the slot of a request that left every state full."""
    for name in "ABC":
        folder = folders(name)
        vocab = plain.TINY[name]["vocab"]
        seqs = _seqs([40, 1, 17], vocab, 9)
        want = _reference(folder, seqs)
        eng = _engine(folder, 4, 20, slots=1)
        for rid, toks in seqs.items():
            rows = [eng.step([StepEntry(rid, toks[:1], [0])]).logits]
            if len(toks) > 1:
                rows.append(eng.step([StepEntry(rid, toks[1:], list(range(len(toks) - 1)))]).logits)
            eng.finish(rid)
            _close(torch.cat(rows), want[rid])


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


def test_long_decoding_token_by_token_through_few_pages(folders):
    folder = folders("A")
    toks = random_tokens(150, 97, 13)
    want = _reference(folder, {"x": toks})["x"]
    eng = _engine(folder, 4, 6)                       # 24 tokens of pages for 150: chunks and windows must give theirs back
    rows = [eng.step([StepEntry("x", [t], [0])]).logits[0] for t in toks]
    _close(torch.stack(rows), want)


# ---------------------------------------------------------------------------- each mechanism alone
def _one_layer(kind, mixer, mlp, width=32):
    return plain.config(41, width, [plain.layer(kind, mixer, mlp)])


_LRU, _SSM, _WKV = plain.linear_unit(8, 2, 2), plain.state_space(2, 8, 4, 1, 1, 2), {"heads": 2, "dim": 8}
_CHUNK = plain.attention(2, 1, 8, 8, 0.4, 10.0, 6)
_WINDOW = plain.attention(2, 1, 8, 8, 0.4, 10.0, 6, rot=plain.rotation(4, 20.0))
ALONE = {
    "chunks": _one_layer("parallel", plain.parallel(plain.attention(6, 2, 8, 12, 0.4, 3.0, 7), _LRU), None),
    "chunk_of_one": _one_layer("parallel", plain.parallel(plain.attention(2, 2, 8, 8, 0.4, 5.0, 1), _LRU), None),
    "chunk_longer_than_anything": _one_layer("parallel", plain.parallel(plain.attention(3, 1, 12, 4, 0.4, 40.0, 1000), _LRU), None),
    "lru_blocks": _one_layer("parallel", plain.parallel(_CHUNK, plain.linear_unit(30, 6, 4)), None),
    "lru_one_block_one_tap": _one_layer("parallel", plain.parallel(_CHUNK, plain.linear_unit(13, 1, 1)), None),
    "lru_nine_taps": _one_layer("parallel", plain.parallel(_CHUNK, plain.linear_unit(12, 3, 9)), None),
    "window": _one_layer("parallel_2", plain.parallel_2(plain.attention(4, 2, 8, 12, 0.4, 3.0, 5, rot=plain.rotation(8, 30.0)), _SSM, 1.0, 0.7), None),
    "window_scaled_rotation": _one_layer("parallel_2", plain.parallel_2(
        plain.attention(2, 1, 12, 8, 0.4, 8.0, 9, rot=plain.rotation(6, 50.0, (2.0, 1.0, 4.0, 16))), _SSM, 0.5, 1.5), None),
    "window_not_rotated": _one_layer("parallel_2", plain.parallel_2(plain.attention(2, 1, 8, 8, 0.4, 8.0, 4), _SSM, 2.0, 1.0), None),
    "ssm_groups": _one_layer("parallel_2", plain.parallel_2(_WINDOW, plain.state_space(6, 4, 10, 2, 3, 4), 1.0, 1.0), None),
    "ssm_one_of_each": _one_layer("parallel_2", plain.parallel_2(_WINDOW, plain.state_space(1, 12, 3, 1, 1, 1), 1.0, 1.0), None),
    "ssm_a_part_per_head": _one_layer("parallel_2", plain.parallel_2(_WINDOW, plain.state_space(4, 6, 8, 4, 4, 3), 0.1, -1.0), None),
    "wkv": _one_layer("wkv", {"heads": 3, "dim": 10}, None),
    "wkv_one_head": _one_layer("wkv", {"heads": 1, "dim": 20}, None),
    "relu2": _one_layer("wkv", _WKV, plain.dense(24)),
    "moe": _one_layer("wkv", _WKV, plain.moe(12, 5, 2)),
    "moe_top1_shared": _one_layer("wkv", _WKV, plain.moe(12, 8, 1, shared=20)),
    "moe_all_chosen": _one_layer("wkv", _WKV, plain.moe(12, 4, 4, shared=4)),
    "odd_width": _one_layer("parallel_2", plain.parallel_2(_WINDOW, _SSM, 1.0, 1.0), plain.moe(10, 3, 2), width=27),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone_in_a_one_layer_model(folders, name):
    folder = folders("alone_" + name, ALONE[name], seed=3)
    seqs = _seqs([27, 12], 41, 6)
    want = _reference(folder, seqs)
    for steps in (traces.whole(seqs), traces.portions(seqs, sizes=(3, 2, 9, 2))):
        got = traces.replay(_engine(folder, 4, 30), steps)
        for rid in seqs:
            _close(got[rid], want[rid][traces.wanted_positions(steps, rid)])


LEFT_OUT = {      # (model, tensors, what stands for leaving the mechanism out)
    "norm bias": ("wkv", ["l0.norm1.b"], 0.0), "norm alpha": ("wkv", ["l0.norm1.alpha"], 1.0), "final norm bias": ("wkv", ["final.norm.b"], 0.0),
    "layer scale": ("wkv", ["l0.ls1"], 1.0), "feed-forward scale": ("relu2", ["l0.ls2"], 1.0),
    "query bias": ("chunks", ["l0.mix.left.q.b"], 0.0), "value bias": ("chunks", ["l0.mix.left.v.b"], 0.0), "head gate": ("chunks", ["l0.mix.left.g"], 0.0),
    "member weight": ("chunks", ["l0.mix.left.out"], 1.0), "gelu branch bias": ("lru_blocks", ["l0.mix.right.y.b"], 0.0),
    "conv input bias": ("lru_blocks", ["l0.mix.right.x.b"], 0.0), "conv bias": ("lru_blocks", ["l0.mix.right.conv.b"], 0.0),
    "recurrence gate": ("lru_blocks", ["l0.mix.right.ra", "l0.mix.right.ra.b"], 0.0), "input gate": ("lru_blocks", ["l0.mix.right.ri", "l0.mix.right.ri.b"], 0.0),
    "skip": ("ssm_groups", ["l0.mix.right.D"], 0.0), "step bias": ("ssm_groups", ["l0.mix.right.dt_bias"], 0.0), "part weight": ("ssm_groups", ["l0.mix.right.norm"], 1.0),
    "token shift": ("wkv", [f"l0.mix.mu.{a}" for a in "rkvgw"], 0.0), "bonus": ("wkv", ["l0.mix.u"], 1.0), "decay bias": ("wkv", ["l0.mix.w0"], 0.0),
    "decay projection": ("wkv", ["l0.mix.w2"], 0.0), "router bias": ("moe", ["l0.mlp.router.b"], 0.0), "shared expert": ("moe_top1_shared", ["l0.mlp.shared.down"], 0.0),
}


@pytest.mark.parametrize("what", sorted(LEFT_OUT))
def test_leaving_a_mechanism_out_shows_in_the_logits(what):
    """The models of the tests are made so that every tensor matters far above the tolerance."""
    name, tensors, value = LEFT_OUT[what]
    W = plain.random_weights(ALONE[name], 3)
    toks = random_tokens(27, 41, 6)
    want = plain.forward(ALONE[name], W, toks)
    for t in tensors:
        assert t in W
        W[t] = torch.full_like(W[t], value)
    assert (plain.forward(ALONE[name], W, toks) - want).abs().max() > 20 * TOL * want.abs().max()


# ---------------------------------------------------------------------------- edges that random weights would hide
def _spiked(cfg, seed):
    """Weights such that the key of token 1 dominates the scores of every query that sees it, in the layer's attention.
    Token 1's embedding lies along stream entry 0, every other token has little there; queries read entry 1, which all have alike,
    into entry 4 of every head (outside what the tests rotate), keys read entry 0 into it, so token 1's score is large and every other
    one small, short of the cap."""
    W = plain.random_weights(cfg, seed)
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    W["embed"][:, 0] = 0.0
    W["embed"][:, 1] = 3.0
    W["embed"][1] = 0.0
    W["embed"][1, 0] = 4.0
    W["embed"][1, 1] = 3.0
    W["l0.norm1"] = torch.ones_like(W["l0.norm1"])
    W["l0.norm1.b"] = torch.zeros_like(W["l0.norm1.b"])
    W["l0.norm1.alpha"] = torch.tensor(1.0)
    for name, heads, column in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        w = torch.zeros_like(W[p + name])
        for h in range(heads):
            w[h * m["dim"] + 4, column] = 3.0
        W[p + name] = w
        if p + name + ".b" in W:
            W[p + name + ".b"] = torch.zeros_like(W[p + name + ".b"])
    return W


def _edge_tokens(n, spike):
    toks = [2 + (7 * i) % 30 for i in range(n)]
    toks[spike] = 1
    return toks


def _differs_at(cfg, changed, W, toks, rows):
    want, moved = plain.forward(cfg, W, toks), plain.forward(changed, W, toks)
    return (moved[rows] - want[rows]).abs().max() > 50 * TOL * want.abs().max()


@pytest.mark.parametrize("window", [5, 8])
def test_a_key_just_inside_and_just_outside_the_window_in_prompt_and_decoding(folders, window):
    cfg = _one_layer("parallel_2", plain.parallel_2(plain.attention(2, 1, 8, 8, 1.0, 30.0, window, rot=plain.rotation(4, 20.0)), _SSM, 1.0, 0.3), None)
    spike = 9
    W = _spiked(cfg, 4)
    toks = _edge_tokens(30, spike)
    for delta in (-1, 1):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["left"]["mask"]["size"] = window + delta
        edge = spike + window - 1 + (1 if delta > 0 else 0)          # the last position that sees the key, the first that does not
        assert _differs_at(cfg, other, W, toks, [edge]), delta
    want = plain.forward(cfg, W, toks)
    folder = folders(f"edge_window_{window}", cfg, weights=W)
    for page in (4, 16):
        for steps in (traces.whole({"x": toks}), traces.prefill_then_decode({"x": toks}, 30 - spike - 2),
                      traces.portions({"x": toks}, sizes=(2, 3, 2, 5))):
            got = traces.replay(_engine(folder, page, 20), steps)["x"]
            _close(got, want[traces.wanted_positions(steps, "x")])


@pytest.mark.parametrize("size,spike", [(6, 11), (6, 12), (8, 15), (8, 16), (5, 10), (5, 14)])
def test_a_key_at_the_end_and_at_the_start_of_a_chunk_in_prompt_and_decoding(folders, size, spike):
    """A key in a chunk's last place is seen by itself alone, one in a chunk's first place by the whole chunk; chunks are
    counted from position 0 wherever a portion starts."""
    cfg = _one_layer("parallel", plain.parallel(plain.attention(2, 1, 8, 8, 1.0, 30.0, size), _LRU), None)
    W = _spiked(cfg, 6)
    toks = _edge_tokens(31, spike)
    for delta in (-1, 1):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["left"]["mask"]["size"] = size + delta
        assert _differs_at(cfg, other, W, toks, slice(spike, 31)), delta
    want = plain.forward(cfg, W, toks)
    folder = folders(f"edge_chunk_{size}_{spike}", cfg, weights=W)
    for page in (4, 16):
        for steps in (traces.whole({"x": toks}), traces.prefill_then_decode({"x": toks}, 31 - spike + 1),
                      traces.portions({"x": toks}, sizes=(2, 3, 2, 5)), traces.portions({"x": toks}, sizes=(size, size - 1, size + 1))):
            got = traces.replay(_engine(folder, page, 20), steps)["x"]
            _close(got, want[traces.wanted_positions(steps, "x")])


def test_the_cap_flattens_large_scores(folders):
    """A spiked key whose score is ten times the cap: without the cap its weight is one, with it another key still counts."""
    cfg = _one_layer("parallel_2", plain.parallel_2(plain.attention(2, 1, 8, 8, 4.0, 2.0, 12), _SSM, 1.0, 0.3), None)
    W = _spiked(cfg, 7)
    toks = _edge_tokens(24, 5)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["left"]["softcap"] = 200.0
    assert _differs_at(cfg, other, W, toks, slice(5, 17))
    folder = folders("cap", cfg, weights=W)
    steps = traces.portions({"x": toks}, sizes=(4, 2, 6))
    _close(traces.replay(_engine(folder, 4, 20), steps)["x"], plain.forward(cfg, W, toks))


def test_a_far_token_reaches_the_end_through_every_recurrence(folders):
    """Decays of almost one: the first token still shows 360 tokens later, through the gated linear recurrence, the state
    space and the matrix state alone (chunks and windows have left it long ago)."""
    kinds = {"lru": ("parallel", plain.parallel(_CHUNK, plain.linear_unit(16, 2, 3))), "ssm": ("parallel_2", plain.parallel_2(_WINDOW, _SSM, 1.0, 1.0)),
             "wkv": ("wkv", _WKV)}
    for name, (kind, mixer) in kinds.items():
        cfg = _one_layer(kind, mixer, None)
        W = plain.random_weights(cfg, 8)
        if name == "lru":
            W["l0.mix.right.lam"] = torch.full_like(W["l0.mix.right.lam"], -9.0)
        elif name == "ssm":
            W["l0.mix.right.A_log"] = torch.full_like(W["l0.mix.right.A_log"], -7.0)
        else:
            W["l0.mix.w0"] = torch.full_like(W["l0.mix.w0"], -9.0)
            W["l0.mix.w2"] *= 0.1
        toks = random_tokens(360, 41, 5)
        want = plain.forward(cfg, W, toks)
        other = plain.forward(cfg, W, [(toks[0] + 1) % 41] + toks[1:])
        assert (other[-1] - want[-1]).abs().max() > 5 * TOL * want.abs().max(), name
        folder = folders("far_" + name, cfg, weights=W)
        steps = traces.portions({"x": toks[:330]}, sizes=(32, 17, 64, 2))
        steps[-1]["end"] = []
        steps += [{"step": len(steps) + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks[330:])]
        got = traces.replay(_engine(folder, 16, 8, max_seq_len=512), steps)["x"]
        _close(got, want[traces.wanted_positions(steps, "x")])


def test_the_token_before_is_met_across_cuts_and_never_across_requests(folders):
    """wkv alone: a portion's first token reads the last one of the portion before, wherever the cut is, and a request's
    first token reads zeros, whatever its slot holds and whoever stands before it in the batch."""
    folder = folders("alone_wkv", ALONE["wkv"], seed=3)
    seqs = _seqs([10, 9], 41, 12)
    want = _reference(folder, seqs)
    a, b = seqs.values()
    for cut in range(1, 9):
        eng = _engine(folder, 4, 20, slots=2)
        one = eng.step([StepEntry("a", a[:cut], list(range(cut))), StepEntry("b", b[:1], [0])]).logits
        two = eng.step([StepEntry("b", b[1:cut + 1], list(range(cut))), StepEntry("a", a[cut:], list(range(10 - cut)))]).logits
        _close(torch.cat([one[:cut], two[cut:]]), want["r0"])
        _close(torch.cat([one[cut:], two[:cut]]), want["r1"][:cut + 1])


def test_the_plain_router_weighs_the_chosen_logits_alone():
    z = torch.tensor([0.5, 3.0, -1.0, 2.0], dtype=torch.float64)
    chosen, w = plain.route(z, 2)
    assert sorted(chosen.tolist()) == [1, 3] and torch.allclose(w, torch.softmax(torch.tensor([3.0, 2.0], dtype=torch.float64), 0))


# ---------------------------------------------------------------------------- generation through the public entry point
@pytest.mark.parametrize("name,slots,budget", [("A", 2, 8), ("B", 3, 16), ("C", 2, 8)])
def test_greedy_generation_through_the_scheduler_matches_the_plain_argmax(folders, name, slots, budget):
    """``C`` without pages for the wkv layers; fewer slots than requests, prompts cut by the token budget."""
    from pytriton_llama_b200 import LLM, SamplingParams
    from pytriton_llama_b200.weights import read_folder
    folder = folders(name)
    W = read_folder(folder)
    prompts = list(_seqs([9, 21, 3, 14], plain.TINY[name]["vocab"], 17).values())
    llm = LLM(folder, EngineConfig(dtype="float32", page_size=4, max_gpu_num_blocks=40, max_seq_len=64, max_num_seqs=slots,
                                   max_batched_tokens=budget, compiled_model=False), device="cpu", ops=TorchOps())
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_gen_len=7))
    for p, out in zip(prompts, got):
        logits = plain.forward(plain.TINY[name], W, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert row[tok] >= row.max() - 1e-4, (i, tok, int(row.argmax()))
