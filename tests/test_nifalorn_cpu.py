"""Nifalorn through the library's own cache, step function and generation loop on a CPU (the kernels' meaning restated
in torch, tests/emulated_ops.py), against the plain implementation: what is tested here is the host side, i.e. the
configuration, the order of the passes with a cache entry per layer run, a layer's chain of cache entries (the state, the
convolution's record), rings of pages under chunks, and the cutting of work into steps."""

import copy
import json
import math

import pytest
import torch

import nifalorn_cases as cases
from conftest import random_tokens
from emulated_ops import EmulatedOps
from helpers import assert_close, run_ragged_batches, run_tail_by_one, run_whole
from plain import nifalorn_plain as plain
from starter_b200.cache import KVGroup, StateGroup
from starter_b200.config import ConfigError, MoESpec, GatedMLPSpec, PairRopeSpec, config_from_dict, load_config
from starter_b200.engine import Engine
from starter_b200.engine.context import Runtime
from starter_b200.engine.session import Session
from starter_b200.parts import build_part


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: cases.write_folder(name, tmp_path_factory.mktemp(f"nifalorn_{name}"), dtype=torch.float32) for name in cases.CASES}


def session(folder, **kw):
    args = dict(dtype="float32", device="cpu", ops=EmulatedOps(), max_tokens=64 * 12, max_seqs=4)
    args.update(kw)
    return Session(folder, **args)


def test_configuration_round_trip_and_parts(folders):
    cfg = load_config(folders["A"])
    assert cfg.architecture == "Nifalorn" and config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    assert spec.residual_float32 and not spec.tie_embeddings and spec.embedding_scale == 0.7 and spec.logit_scale == 1.5
    assert spec.execution_order() == (0, 1, 2, 3, 1, 2, 3, 4) and spec.loop is None and spec.pass_starts() == {}
    assert [b.kind for b in spec.layers] == ["prenorm"] * 5
    assert [b.mixer.kind for b in spec.layers] == ["lightning", "mamba2", "diff_attention", "lightning", "mamba2"]
    assert [b.ff.kind if b.ff is not None else None for b in spec.layers] == ["moe", "act_mlp", "moe", None, "moe"]
    assert spec.layers[0].mixer_norm.offset == 1.0 and spec.final_norm.offset == 1.0
    light = spec.layers[0].mixer
    assert (light.num_heads, light.head_dim, light.v_dim, light.decay) == (3, 16, 24, (0.9, 0.5, 0.99))
    mamba = spec.layers[1].mixer
    assert (mamba.num_heads, mamba.v_dim, mamba.state, mamba.groups, mamba.taps, mamba.norm_groups) == (6, 16, 24, 3, 3, 2)
    attn = spec.layers[2].mixer
    assert (attn.chunk, attn.window, attn.gate, attn.scale, attn.diff) == (24, None, False, 0.4, 0.7)
    assert (attn.position.kind, attn.position.rotary_dim, attn.position.factor, attn.position.low, attn.position.high,
            attn.position.original) == ("rope_pairs", 12, 8.0, 1.0, 4.0, 512.0)
    moe = spec.layers[0].ff
    assert (moe.scores, moe.groups, moe.keep_groups, moe.top, moe.route_scale, moe.shared_gate, moe.n_experts) == ("sigmoid", 3, 2, 3, 1.7, True, 12)
    assert moe.expert.activation == "silu" and moe.expert.intermediate_size == 40 and moe.shared.intermediate_size == 56
    names = cfg.tensor_names()
    assert names.layers[1]["mixer"]["conv_bias"] == "l1.mix.conv.b" and names.layers[0]["ff"]["shared_sg"] == "l0.mlp.shared.sg"
    assert names.layers[2]["ff"]["e9_up"] == "l2.mlp.e9.up" and "ff" not in names.layers[3] and names.lm_head == "head"
    bare = cases.config("C").model_spec()
    assert bare.execution_order() == (0, 1, 0, 1, 0, 1, 2, 3)
    assert bare.layers[2].mixer.position is None and bare.layers[2].mixer.chunk is None and bare.layers[0].ff.shared is None
    assert not bare.layers[0].ff.shared_gate and bare.layers[0].ff.groups == 4
    assert cases.config("B").model_spec().execution_order() == (0, 1, 2, 3)


@pytest.mark.parametrize("change, what", [
    (lambda r: r["layers"][0].update(type="conv"), "unknown"),
    (lambda r: r["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][0]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"].update(groups=4), "evenly"),
    (lambda r: r["layers"][1]["mixer"].update(norm_groups=5), "equal parts"),
    (lambda r: r["layers"][1]["mixer"].pop("state"), "state"),
    (lambda r: r["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][2]["mixer"].update(kv_heads=4), "evenly"),
    (lambda r: r["layers"][2]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=18), "at most dim"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda r: r["layers"][0]["mlp"].update(kind="gated"), "not built"),
    (lambda r: r["layers"][0]["mlp"]["router"]["groups"].update(count=5), "equal groups"),
    (lambda r: r["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "are kept"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=9), "chooses"),
    (lambda r: r["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda r: r["loop"].update(stop=6), "loop runs"),
    (lambda r: r["loop"].update(times=0), "times"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_bad_configurations_are_refused(change, what):
    raw = copy.deepcopy(cases.CASES["A"])
    change(raw)
    with pytest.raises(ConfigError, match=what):
        config_from_dict(raw)


def test_stretched_frequencies_in_all_three_ranges():
    rot = {"base": 1000.0, "dims": 16, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}}
    want = torch.tensor(plain.rotary_frequencies(rot), dtype=torch.float64)
    spec = PairRopeSpec(theta=1000.0, rotary_dim=16, factor=8.0, low=1.0, high=4.0, original=512.0)
    part = build_part("position", spec, {}, Runtime(torch.float32, torch.device("cpu"), EmulatedOps()))
    assert part.magnitude == 1.0 and not part.halves
    assert float((part.frequencies.double() / want - 1).abs().max()) < 1e-6
    plain_f = torch.tensor([1000.0 ** (-2.0 * i / 16) for i in range(8)], dtype=torch.float64)
    ratio = want / plain_f
    assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 1.0 / 8.0) < 1e-12                       # kept, and slowed down
    assert any(1.0 / 8.0 + 1e-3 < float(r) < 1.0 - 1e-3 for r in ratio)                               # and a blend between
    assert 512.0 / (2.0 * math.pi / float(plain_f[-1])) < 1.0


def test_a_cache_entry_per_layer_run(folders):
    layers = session(folders["A"], max_step_tokens=50).cache.layers
    assert len(layers) == 8
    runs_of_mamba = [layers[1], layers[4]]
    assert len({(id(l.group), l.index) for l in runs_of_mamba}) == 2            # every pass keeps a state of its own
    for l in runs_of_mamba:
        assert isinstance(l.group, StateGroup) and l.state.shape[1:] == (6 * 24 * 16,)
        assert isinstance(l.aux.group, StateGroup) and l.aux.state.shape[1:] == (2, 6 * 16 + 2 * 3 * 24)
    runs_of_attention = [layers[2], layers[5]]
    assert all(isinstance(l.group, KVGroup) and l.group.ring_pages for l in runs_of_attention)     # a chunk bounds what is kept
    assert runs_of_attention[0].index != runs_of_attention[1].index
    assert runs_of_attention[0].group.k.shape[2] == 2 * 2 and runs_of_attention[0].group.v.shape[2] == 2   # two key maps, one value
    bare = session(folders["C"]).cache.layers
    assert bare[1].aux is None and bare[6].group.ring_pages == 0                # one tap keeps no record; no chunk keeps every key


@pytest.mark.parametrize("name", list(cases.CASES))
def test_every_cutting_matches_plain(folders, name):
    folder = folders[name]
    seqs = random_tokens(cases.CASES[name]["vocab"], (5, 90, 41, 1, 64, 65, 2), seed=3)
    ref = cases.plain_logits(folder, seqs)
    sess = session(folder, max_rows=50, max_step_tokens=48)     # longer steps go through in several forward passes
    assert_close(run_whole(sess, seqs), ref, "float32", "alone and whole")
    assert_close(run_whole(sess, seqs[:3], together=True), ref[:3], "float32", "one ragged step")
    assert_close(run_tail_by_one(sess, seqs, tail=30), ref, "float32", "tail one by one")
    assert_close(run_ragged_batches(sess, seqs, batch_size=3, poison=True), ref, "float32", "ragged batches, freed pages poisoned")
    assert sess.cache.slots.n_held == 0


def test_portions_down_to_two_tokens(folders):
    seqs = random_tokens(211, (37,), seed=4)
    ref = cases.plain_logits(folders["A"], seqs)
    for portion in (2, 3, 7, 20, 21):
        sess = session(folders["A"], max_rows=portion)
        assert_close(run_whole(sess, seqs), ref, "float32", f"portions of {portion}")


def test_state_of_a_freed_slot_does_not_leak(folders):
    """A slot that held a sequence is used again: states and convolution records start from zero, not from what the last
    sequence left there."""
    sess = session(folders["D"], max_seqs=1)
    seqs = random_tokens(64, (70, 9, 3), seed=5)
    ref = cases.plain_logits(folders["D"], seqs)
    assert_close(run_whole(sess, seqs), ref, "float32", "later sequences in the first one's slot")
    assert_close(run_tail_by_one(sess, seqs, tail=8), ref, "float32", "and decoded")


def test_layer_runs_match_plain(folders):
    """The residual after every layer run (a looped layer counts each time), taken from the library's own stream."""
    cfg, tensors = plain.read_folder(folders["A"])
    tokens = random_tokens(211, (29,), seed=9)[0]
    want = []
    plain.forward(cfg, tensors, tokens, want)
    sess = session(folders["A"])
    seen = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            seen.append(stream.x + stream.pending)      # the last branch's output waits for the next norm
        block.forward = spy
    run_whole(sess, [tokens])
    assert len(seen) == len(want) == 8
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert got.dtype == torch.float32
        assert float((got - ref).abs().max()) <= 1e-4 * float(ref.abs().max()), f"layer run {i}"


def test_routers_that_cannot_choose_are_refused():
    expert = GatedMLPSpec(hidden_size=8, intermediate_size=8)
    base = dict(hidden_size=8, n_experts=6, n_identity=0, top=2, route_scale=1.0, expert=expert, scores="sigmoid")
    rt = Runtime(torch.float32, torch.device("cpu"), EmulatedOps())
    for change, what in (({"groups": 4}, "equal groups"), ({"groups": 3, "keep_groups": 4}, "kept"), ({"groups": 6, "keep_groups": 1}, "out of"),
                         ({"scores": "tanh"}, "scores"), ({"over_chosen": True}, "scores")):
        with pytest.raises(ValueError, match=what):
            build_part("ff", MoESpec(**dict(base, **change)), {}, rt)


def test_greedy_generation_through_the_entry_point(folders):
    cfg, tensors = plain.read_folder(folders["C"])
    prompts = random_tokens(97, (3, 11, 1), seed=6)
    want = plain.generate(cfg, tensors, prompts, 10)
    engine = Engine.from_session(session(folders["C"]), use_graphs=False)
    assert engine.generate_all(prompts, 10) == want
    assert engine.session.cache.slots.n_held == 0


def test_random_weights_from_the_command_line(tmp_path):
    from starter_b200.cli import main
    (tmp_path / "config.json").write_text(json.dumps(cases.CASES["D"]))
    assert main(["random-weights", "--config", str(tmp_path / "config.json"), "--seed", "3", "--out", str(tmp_path / "model")]) == 0
    sess = session(tmp_path / "model")
    assert sess.model.spec.vocab_size == 64 and len(sess.model.blocks) == 3
    seqs = random_tokens(64, (12,), seed=8)
    assert_close(run_whole(sess, seqs), cases.plain_logits(tmp_path / "model", seqs), "float32", "folder from the command line")
